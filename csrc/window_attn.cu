// Windowed attention with a distance bias over the paged cache on the CUDA cores (stack.h, WindowAttnArgs): any head
// sizes up to 512, any GQA group and page size, bf16 or fp32 storage, fp32 arithmetic throughout. It serves the 32-bit
// mode and the shapes that the tcgen05 kernels (window_attn_tcgen05.cu, paged_decode_tc.cu) do not take.
#include <algorithm>

#include "common.cuh"
#include "launch.cuh"
#include "stack.h"

namespace cb {

constexpr int WS_ROWS = cosmos::WINDOW_ATTN_SIMT_ROWS, WS_KEYS = 32, WS_THREADS = 256;

__device__ __forceinline__ float ws_get(const float* p) { return *p; }
__device__ __forceinline__ float ws_get(const bf16* p) { return __bfloat162float(*p); }
__device__ __forceinline__ void ws_put(float* p, float v) { *p = v; }
__device__ __forceinline__ void ws_put(bf16* p, float v) { *p = __float2bfloat16(v); }

__host__ __device__ inline int ws_smem_floats(int dim, int vdim) {
  return WS_ROWS * dim + WS_KEYS * (dim + 1) + WS_KEYS * vdim + WS_ROWS * vdim + WS_ROWS * (WS_KEYS + 1) + 2 * WS_ROWS;
}

// One CTA = up to 16 query rows of one head. Warp w owns the scores of rows w and w + 8 (lane = key).
template <typename T>
__global__ void __launch_bounds__(WS_THREADS)
window_attn_simt_kernel(const cosmos::WindowAttnArgs a) {
  extern __shared__ float sm[];
  const int dim = a.dim, vdim = a.vdim;
  float* qs = sm;                                  // [16][dim]
  float* ks = qs + WS_ROWS * dim;                  // [32][dim + 1]
  float* vs = ks + WS_KEYS * (dim + 1);            // [32][vdim]
  float* os = vs + WS_KEYS * vdim;                 // [16][vdim]
  float* ps = os + WS_ROWS * vdim;                 // [16][33]
  float* corr_s = ps + WS_ROWS * (WS_KEYS + 1);    // [16]
  float* l_s = corr_s + WS_ROWS;                   // [16]
  const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31;
  const int h = blockIdx.y, kvh = h / (a.H / a.G);
  int seq, row0, rows, pos0;
  if (a.tiles) {
    const int4 t = reinterpret_cast<const int4*>(a.tiles)[blockIdx.x];
    seq = t.x; row0 = t.y; rows = t.z; pos0 = t.w;
  } else {
    seq = row0 = blockIdx.x; rows = 1; pos0 = a.seq_lens[seq] - 1;
  }
  T* out = reinterpret_cast<T*>(a.out) + (long long)row0 * a.ldo + (long long)h * vdim;
  if (pos0 < 0) {   // idle slot of a decode batch
    for (int c = tid; c < vdim; c += WS_THREADS) ws_put(out + c, 0.f);
    return;
  }
  const T* q = reinterpret_cast<const T*>(a.q) + (long long)row0 * a.ldq + (long long)h * dim;
  for (int i = tid; i < WS_ROWS * dim; i += WS_THREADS) {
    const int r = i / dim, c = i - r * dim;
    qs[i] = r < rows ? ws_get(q + (long long)r * a.ldq + c) : 0.f;
  }
  for (int i = tid; i < WS_ROWS * vdim; i += WS_THREADS) os[i] = 0.f;
  const float r1 = a.r1 ? a.r1[h] : 0.f, r2 = a.r2 ? a.r2[h] : 0.f;
  float m_run[2] = {-INFINITY, -INFINITY}, l_run[2] = {0.f, 0.f};
  const int lo = max(0, pos0 - a.window + 1), hi = pos0 + rows;
  for (int k0 = lo; k0 < hi; k0 += WS_KEYS) {
    __syncthreads();
    for (int j = warp; j < WS_KEYS; j += WS_THREADS / 32) {
      const int pos = k0 + j;
      const T *kp = nullptr, *vp = nullptr;
      if (pos < hi) {
        int page = a.table[(long long)seq * a.max_pages + pos / a.page_size];
        if (!index_ok(page, a.num_pages, a.status, SITE_STACK_PAGE)) page = 0;
        const long long row = ((long long)page * a.G + kvh) * a.page_size + pos % a.page_size;
        kp = reinterpret_cast<const T*>(a.k_cache) + row * dim;
        vp = reinterpret_cast<const T*>(a.v_cache) + row * vdim;
      }
      for (int c = lane; c < dim; c += 32) ks[j * (dim + 1) + c] = kp ? ws_get(kp + c) : 0.f;
      for (int c = lane; c < vdim; c += 32) vs[j * vdim + c] = vp ? ws_get(vp + c) : 0.f;
    }
    __syncthreads();
#pragma unroll
    for (int rr = 0; rr < 2; ++rr) {
      const int r = warp + 8 * rr;
      const int dist = pos0 + r - (k0 + lane);
      const bool vis = r < rows && dist >= 0 && dist < a.window && k0 + lane < hi;
      float s = -INFINITY;
      if (vis) {
        float dot = 0.f;
        for (int c = 0; c < dim; ++c) dot = fmaf(qs[r * dim + c], ks[lane * (dim + 1) + c], dot);
        s = dot * a.scale;
        if (a.r1) s -= r1 * (a.r2 ? log1pf(r2 * (float)dist) : (float)dist);
      }
      float mx = s;
#pragma unroll
      for (int o = 16; o > 0; o >>= 1) mx = fmaxf(mx, __shfl_xor_sync(0xffffffffu, mx, o));
      const float m_new = fmaxf(m_run[rr], mx);
      const float p = vis ? expf(s - m_new) : 0.f;
      const float corr = m_run[rr] == -INFINITY ? 0.f : expf(m_run[rr] - m_new);
      float sum = p;
#pragma unroll
      for (int o = 16; o > 0; o >>= 1) sum += __shfl_xor_sync(0xffffffffu, sum, o);
      l_run[rr] = l_run[rr] * corr + sum;
      m_run[rr] = m_new;
      ps[r * (WS_KEYS + 1) + lane] = p;
      if (lane == 0) corr_s[r] = corr;
    }
    __syncthreads();
    for (int i = tid; i < WS_ROWS * vdim; i += WS_THREADS) {
      const int r = i / vdim, c = i - r * vdim;
      float acc = os[i] * corr_s[r];
#pragma unroll 8
      for (int j = 0; j < WS_KEYS; ++j) acc = fmaf(ps[r * (WS_KEYS + 1) + j], vs[j * vdim + c], acc);
      os[i] = acc;
    }
  }
  if (lane == 0) {
    l_s[warp] = l_run[0];
    l_s[warp + 8] = l_run[1];
  }
  __syncthreads();
  for (int i = tid; i < rows * vdim; i += WS_THREADS) {
    const int r = i / vdim, c = i - r * vdim;
    ws_put(out + (long long)r * a.ldo + c, os[i] / l_s[r]);
  }
}

}  // namespace cb

namespace cosmos {

template <typename T>
static void launch_simt(const WindowAttnArgs& a, int smem, cudaStream_t s) {
  static int granted = 48 * 1024;
  if (smem > granted) {
    if (cudaFuncSetAttribute(cb::window_attn_simt_kernel<T>, cudaFuncAttributeMaxDynamicSharedMemorySize, smem) != cudaSuccess)
      throw std::runtime_error("window_attn: head size too large");
    granted = smem;
  }
  cb::window_attn_simt_kernel<T><<<dim3(a.tiles ? a.n_tiles : a.n_seqs, a.H), cb::WS_THREADS, smem, s>>>(a);
}

void window_attn_simt(const WindowAttnArgs& a, cudaStream_t s) {
  if ((a.tiles ? a.n_tiles : a.n_seqs) <= 0) return;
  if (a.G < 1 || a.H % a.G != 0 || a.window < 1 || a.page_size < 1) throw std::runtime_error("window_attn: bad shape");
  if (a.tiles && a.tile_rows > cb::WS_ROWS) throw std::runtime_error("window_attn: tiles of at most 16 query rows");
  if (a.dim < 1 || a.vdim < 1 || a.dim > 512 || a.vdim > 512) throw std::runtime_error("window_attn: head sizes up to 512");
  const int smem = cb::ws_smem_floats(a.dim, a.vdim) * (int)sizeof(float);
  if (a.is_f32)
    launch_simt<float>(a, smem, s);
  else
    launch_simt<bf16>(a, smem, s);
}

}  // namespace cosmos
