// Row-wise kernels of a layer stack's step (stack.h): residual add + grouped RMS norm with the expert dispatch / combine
// folded in, the value side of the q/k/v projection, expert routing by token table, and the 32-bit grouped GEMM.
#include <algorithm>

#include "common.cuh"
#include "launch.cuh"
#include "stack.h"
#include "vec.cuh"

namespace cb {

// The common case of residual_norm_kernel (below), tuned for whole prompts: at most 4 vectors of 8 per thread, kept in
// registers (all loads of a row are issued before the first use), one or two parts of at least a warp's vectors each.
template <typename T, typename Y, int NV>
__global__ void __launch_bounds__(256)
residual_norm_row_kernel(const cosmos::ResidualNormArgs a) {
  __shared__ float part_s[2][8];
  const long long r = blockIdx.x;
  const int tid = threadIdx.x, nt = blockDim.x, warp = tid >> 5, lane = tid & 31, warps = nt >> 5;
  const int d = a.d;
  float* xr = a.x + r * d;
  float v[NV][8];
  if (a.embed) {
    long long tok = a.tokens[r];
    if (!index_ok(tok, a.vocab, a.status, SITE_STACK_TOKEN)) tok = 0;
    const T* er = reinterpret_cast<const T*>(a.embed) + tok * a.ld_embed;
#pragma unroll
    for (int i = 0; i < NV; ++i) {
      const int c = (tid + i * nt) * 8;
      if (c < d) {
        Vec<T, 8>::load(er + c, v[i]);
#pragma unroll
        for (int e = 0; e < 8; ++e) v[i][e] *= a.embed_scale;
      }
    }
  } else {
#pragma unroll
    for (int i = 0; i < NV; ++i) {
      const int c = (tid + i * nt) * 8;
      if (c < d) Vec<float, 8>::load(xr + c, v[i]);
    }
  }
  if (a.y) {
    for (int k = 0; k < a.top; ++k) {
      const long long yr = a.y_rows ? (long long)a.y_rows[r * a.top + k] : r;
      if (!index_ok(yr, a.y_n, a.status, SITE_MOE_ROW)) continue;
      const Y* src = reinterpret_cast<const Y*>(a.y) + yr * a.ldy;
      for (int ks = 0; ks < a.k_splits; ++ks, src += a.split_stride) {
#pragma unroll
        for (int i = 0; i < NV; ++i) {
          const int c = (tid + i * nt) * 8;
          if (c < d) {
            float t[8];
            Vec<Y, 8>::load(src + c, t);
#pragma unroll
            for (int e = 0; e < 8; ++e) v[i][e] = fmaf(a.weight, t[e], v[i][e]);
          }
        }
      }
    }
  }
  const int psize = d / a.groups;   // one or two parts
  float ss[2] = {0.f, 0.f};
#pragma unroll
  for (int i = 0; i < NV; ++i) {
    const int c = (tid + i * nt) * 8;
    if (c < d) {
      Vec<float, 8>::store(xr + c, v[i]);
      float s = 0.f;
#pragma unroll
      for (int e = 0; e < 8; ++e) s = fmaf(v[i][e], v[i][e], s);
      if (c < psize) ss[0] += s; else ss[1] += s;
    }
  }
  if (!a.h) return;
  ss[0] = warp_add(ss[0]);
  ss[1] = warp_add(ss[1]);
  if (lane == 0) {
    part_s[0][warp] = ss[0];
    part_s[1][warp] = ss[1];
  }
  __syncthreads();
  float rinv[2] = {0.f, 0.f};
  for (int w = 0; w < warps; ++w) {
    rinv[0] += part_s[0][w];
    rinv[1] += part_s[1][w];
  }
  rinv[0] = 1.f / sqrtf(rinv[0] / (float)psize + a.eps);
  rinv[1] = 1.f / sqrtf(rinv[1] / (float)psize + a.eps);
  const T* gamma = reinterpret_cast<const T*>(a.gamma);
  T* h = reinterpret_cast<T*>(a.h);
#pragma unroll
  for (int i = 0; i < NV; ++i) {
    const int c = (tid + i * nt) * 8;
    if (c < d) {
      float g[8];
      Vec<T, 8>::load(gamma + c, g);
      const float q = c < psize ? rinv[0] : rinv[1];
#pragma unroll
      for (int e = 0; e < 8; ++e) v[i][e] = v[i][e] * q * g[e];
    }
  }
  for (int k = 0; k < (a.h_rows ? a.h_top : 1); ++k) {
    const long long hr = a.h_rows ? (long long)a.h_rows[r * a.h_top + k] : r;
    if (!index_ok(hr, a.h_n, a.status, SITE_MOE_ROW)) continue;
#pragma unroll
    for (int i = 0; i < NV; ++i) {
      const int c = (tid + i * nt) * 8;
      if (c < d) Vec<T, 8>::store(h + hr * a.ldh + c, v[i]);
    }
  }
}

// One CTA per token row; the updated row is kept in shared memory between the sum and the norm.
template <typename T, typename Y, int VEC>
__global__ void __launch_bounds__(1024)
residual_norm_kernel(const cosmos::ResidualNormArgs a) {
  extern __shared__ __align__(16) float row_s[];   // d
  __shared__ float part_s[32];
  __shared__ float rinv_s[32];
  const long long r = blockIdx.x;
  const int tid = threadIdx.x, nt = blockDim.x, warp = tid >> 5, lane = tid & 31, warps = nt >> 5;
  const int d = a.d;
  float* xr = a.x + r * d;
  const T* er = nullptr;
  if (a.embed) {
    long long tok = a.tokens[r];
    if (!index_ok(tok, a.vocab, a.status, SITE_STACK_TOKEN)) tok = 0;
    er = reinterpret_cast<const T*>(a.embed) + tok * a.ld_embed;
  }
  const Y* y = reinterpret_cast<const Y*>(a.y);
  for (int i = tid * VEC; i < d; i += nt * VEC) {
    float v[VEC];
    if (er) {
      Vec<T, VEC>::load(er + i, v);
#pragma unroll
      for (int e = 0; e < VEC; ++e) v[e] *= a.embed_scale;
    } else {
      Vec<float, VEC>::load(xr + i, v);
    }
    if (y) {
      float s[VEC];
#pragma unroll
      for (int e = 0; e < VEC; ++e) s[e] = 0.f;
      for (int k = 0; k < a.top; ++k) {
        const long long yr = a.y_rows ? (long long)a.y_rows[r * a.top + k] : r;
        if (!index_ok(yr, a.y_n, a.status, SITE_MOE_ROW)) continue;
        const Y* src = y + yr * a.ldy + i;
#pragma unroll 4
        for (int ks = 0; ks < a.k_splits; ++ks) {
          float t[VEC];
          Vec<Y, VEC>::load(src + ks * a.split_stride, t);
#pragma unroll
          for (int e = 0; e < VEC; ++e) s[e] += t[e];
        }
      }
#pragma unroll
      for (int e = 0; e < VEC; ++e) v[e] = fmaf(a.weight, s[e], v[e]);
    }
    if (er || y) Vec<float, VEC>::store(xr + i, v);
    Vec<float, VEC>::store(row_s + i, v);
  }
  if (!a.h) return;
  __syncthreads();
  // root mean square of every part, 32 parts at a time; with fewer parts than warps several warps share one
  const int psize = d / a.groups;
  const T* gamma = reinterpret_cast<const T*>(a.gamma);
  T* h = reinterpret_cast<T*>(a.h);
  for (int g0 = 0; g0 < a.groups; g0 += 32) {
    const int ng = min(32, a.groups - g0);
    if (ng >= warps) {
      for (int g = warp; g < ng; g += warps) {
        const float* p = row_s + (g0 + g) * psize;
        float s = 0.f;
        for (int i = lane; i < psize; i += 32) s = fmaf(p[i], p[i], s);
        s = warp_add(s);
        if (lane == 0) rinv_s[g] = 1.f / sqrtf(s / (float)psize + a.eps);
      }
    } else {
      const int wpg = warps / ng, g = warp / wpg, w = warp - g * wpg;
      float s = 0.f;
      if (g < ng) {
        const float* p = row_s + (g0 + g) * psize;
        for (int i = w * 32 + lane; i < psize; i += wpg * 32) s = fmaf(p[i], p[i], s);
      }
      s = warp_add(s);
      if (lane == 0) part_s[warp] = s;
      __syncthreads();
      if (tid < ng) {
        float t = 0.f;
        for (int j = 0; j < wpg; ++j) t += part_s[tid * wpg + j];
        rinv_s[tid] = 1.f / sqrtf(t / (float)psize + a.eps);
      }
    }
    __syncthreads();
    const int i1 = (g0 + ng) * psize;
    for (int i = g0 * psize + tid * VEC; i < i1; i += nt * VEC) {   // VEC divides psize: a vector stays in its part
      float v[VEC], g[VEC];
      Vec<float, VEC>::load(row_s + i, v);
      Vec<T, VEC>::load(gamma + i, g);
      const float rinv = rinv_s[i / psize - g0];
#pragma unroll
      for (int e = 0; e < VEC; ++e) v[e] = v[e] * rinv * g[e];
      if (a.h_rows) {
        for (int k = 0; k < a.h_top; ++k) {
          const long long hr = a.h_rows[r * a.h_top + k];
          if (index_ok(hr, a.h_n, a.status, SITE_MOE_ROW)) Vec<T, VEC>::store(h + hr * a.ldh + i, v);
        }
      } else {
        Vec<T, VEC>::store(h + r * a.ldh + i, v);
      }
    }
    __syncthreads();
  }
}

// One warp per (token, head): q heads (partial sums only), k heads, v heads.
template <typename T>
__global__ void __launch_bounds__(256)
qkv_value_post_kernel(const cosmos::QkvValueArgs a) {
  constexpr int R = 16;   // head sizes up to 512
  const int lane = threadIdx.x & 31;
  const int nq = a.partial ? a.H : 0;
  const int heads = nq + 2 * a.G;
  const long long w = (long long)blockIdx.x * (blockDim.x >> 5) + (threadIdx.x >> 5);
  if (w >= a.n * heads) return;
  const long long t = w / heads;
  const int h = (int)(w - t * heads);
  const int kind = h < nq ? 0 : (h < nq + a.G ? 1 : 2);   // q, k, v
  const int hh = kind == 0 ? h : (kind == 1 ? h - nq : h - nq - a.G);
  const int size = kind == 2 ? a.vdim : a.dim;
  const int col = kind == 0 ? hh * a.dim : (kind == 1 ? (a.H + hh) * a.dim : (a.H + a.G) * a.dim + hh * a.vdim);
  float v[R];
  float ss = 0.f;
#pragma unroll
  for (int i = 0; i < R; ++i) {
    const int c = lane + 32 * i;
    v[i] = 0.f;
    if (c < size) {
      if (a.partial) {
        const float* p = a.partial + t * a.ld_partial + col + c;
        float s = 0.f;
        for (int ks = 0; ks < a.k_splits; ++ks) s += p[ks * a.split_stride];
        if (a.bias) s += Elem<T>::get(reinterpret_cast<const T*>(a.bias) + col + c);
        v[i] = s;
      } else {
        v[i] = Elem<T>::get(reinterpret_cast<const T*>(a.qkv) + t * a.ld + col + c);
      }
      ss = fmaf(v[i], v[i], ss);
    }
  }
  if (kind == 0) {
    T* dst = reinterpret_cast<T*>(a.q_out) + (t * a.H + hh) * a.dim;
#pragma unroll
    for (int i = 0; i < R; ++i)
      if (lane + 32 * i < size) Elem<T>::put(dst + lane + 32 * i, v[i]);
    return;
  }
  float rinv = 1.f;
  if (kind == 2 && a.value_norm) rinv = 1.f / sqrtf(warp_add(ss) / (float)size + a.eps);
  const long long slot = a.slots[t];
  const bool ok = index_ok(slot, a.n_slots, a.status, SITE_STACK_SLOT);
  const long long page = ok ? slot / a.page_size : 0;
  const int off = ok ? (int)(slot - page * a.page_size) : 0;
  T* dst = reinterpret_cast<T*>(kind == 1 ? a.k_cache : a.v_cache) + ((page * a.G + hh) * a.page_size + off) * (long long)size;
  const float lam = (kind == 2 && a.v_first_in) ? *a.lam : 0.f;
  const long long fo = (t * a.G + hh) * (long long)a.vdim;
#pragma unroll
  for (int i = 0; i < R; ++i) {
    const int c = lane + 32 * i;
    if (c < size) {
      float x = v[i] * rinv;
      if (kind == 2) {
        if (a.v_first_out) a.v_first_out[fo + c] = x;
        if (a.v_first_in) x = (1.f - lam) * x + lam * a.v_first_in[fo + c];
      }
      if (ok) Elem<T>::put(dst + c, x);
    }
  }
}

// The same for head sizes that are multiples of 8: `lanes` threads (a power of two that covers the larger head) share a
// head, 8 elements each, so a row moves in 16-byte pieces.
template <typename T>
__global__ void __launch_bounds__(256)
qkv_value_post_vec_kernel(const cosmos::QkvValueArgs a, int lanes) {
  const int nq = a.partial ? a.H : 0;
  const int heads = nq + 2 * a.G;
  const long long w = ((long long)blockIdx.x * blockDim.x + threadIdx.x) / lanes;
  const int sub = threadIdx.x & (lanes - 1);
  const bool live = w < a.n * heads;    // dead lanes stay for the shuffles
  const long long t = live ? w / heads : 0;
  const int h = live ? (int)(w - t * heads) : 0;
  const int kind = h < nq ? 0 : (h < nq + a.G ? 1 : 2);
  const int hh = kind == 0 ? h : (kind == 1 ? h - nq : h - nq - a.G);
  const int size = kind == 2 ? a.vdim : a.dim;
  const int col = kind == 0 ? hh * a.dim : (kind == 1 ? (a.H + hh) * a.dim : (a.H + a.G) * a.dim + hh * a.vdim);
  const int c = sub * 8;
  const bool in = live && c < size;
  float v[8] = {0.f, 0.f, 0.f, 0.f, 0.f, 0.f, 0.f, 0.f};
  if (in) {
    if (a.partial) {
      const float* p = a.partial + t * a.ld_partial + col + c;
#pragma unroll 4
      for (int ks = 0; ks < a.k_splits; ++ks) {
        float x[8];
        Vec<float, 8>::load(p + ks * a.split_stride, x);
#pragma unroll
        for (int e = 0; e < 8; ++e) v[e] += x[e];
      }
      if (a.bias) {
        float x[8];
        Vec<T, 8>::load(reinterpret_cast<const T*>(a.bias) + col + c, x);
#pragma unroll
        for (int e = 0; e < 8; ++e) v[e] += x[e];
      }
    } else {
      Vec<T, 8>::load(reinterpret_cast<const T*>(a.qkv) + t * a.ld + col + c, v);
    }
  }
  if (kind == 2 && a.value_norm) {
    float ss = 0.f;
#pragma unroll
    for (int e = 0; e < 8; ++e) ss = fmaf(v[e], v[e], ss);
    // lanes of one head share `kind`; the mask names exactly them
    const unsigned mask = (lanes == 32 ? 0xffffffffu : ((1u << lanes) - 1u)) << ((threadIdx.x & 31) & ~(lanes - 1));
    for (int o = lanes >> 1; o > 0; o >>= 1) ss += __shfl_xor_sync(mask, ss, o);
    const float rinv = 1.f / sqrtf(ss / (float)size + a.eps);
#pragma unroll
    for (int e = 0; e < 8; ++e) v[e] *= rinv;
  }
  if (!in) return;
  if (kind == 0) {
    Vec<T, 8>::store(reinterpret_cast<T*>(a.q_out) + (t * a.H + hh) * a.dim + c, v);
    return;
  }
  if (kind == 2) {
    const long long fo = (t * a.G + hh) * (long long)a.vdim + c;
    if (a.v_first_out) Vec<float, 8>::store(a.v_first_out + fo, v);
    if (a.v_first_in) {
      const float lam = *a.lam;
      float f[8];
      Vec<float, 8>::load(a.v_first_in + fo, f);
#pragma unroll
      for (int e = 0; e < 8; ++e) v[e] = (1.f - lam) * v[e] + lam * f[e];
    }
  }
  const long long slot = a.slots[t];
  if (!index_ok(slot, a.n_slots, a.status, SITE_STACK_SLOT)) return;
  const long long page = slot / a.page_size;
  const int off = (int)(slot - page * a.page_size);
  Vec<T, 8>::store(reinterpret_cast<T*>(kind == 1 ? a.k_cache : a.v_cache) +
                       ((page * a.G + hh) * a.page_size + off) * (long long)size + c, v);
}

// Counting sort of the step's (token, k) pairs by expert, one CTA per layer. The order inside an expert is arbitrary:
// the rows of a product do not depend on one another.
__global__ void __launch_bounds__(1024)
moe_route_kernel(const long long* __restrict__ tokens, long long n, int vocab, const long long* __restrict__ desc,
                 int top_max, int* __restrict__ rows, int4* __restrict__ tiles, int max_tiles, int* __restrict__ n_tiles,
                 int* status) {
  extern __shared__ int cnt[];   // [experts]: counts, then the next free row of each expert
  const int layer = blockIdx.x, tid = threadIdx.x, nt = blockDim.x;
  const int* table = reinterpret_cast<const int*>(desc[layer * 4]);
  const int E = (int)desc[layer * 4 + 1], top = (int)desc[layer * 4 + 2], tile = (int)desc[layer * 4 + 3];
  rows += (long long)layer * n * top_max;
  tiles += (long long)layer * max_tiles;
  for (int e = tid; e < E; e += nt) cnt[e] = 0;
  __syncthreads();
  const long long pairs = n * top;
  auto expert_of = [&](long long p) {
    const long long t = p / top;
    long long tok = tokens[t];
    if (!index_ok(tok, vocab, status, SITE_STACK_TOKEN)) tok = 0;
    int e = table[tok * top + (p - t * top)];
    if (!index_ok(e, E, status, SITE_MOE_EXPERT)) e = 0;
    return e;
  };
  for (long long p = tid; p < pairs; p += nt) atomicAdd(&cnt[expert_of(p)], 1);
  __syncthreads();
  if (tid < 32) {
    int row_base = 0, tile_base = 0;
    for (int e0 = 0; e0 < E; e0 += 32) {
      const int e = e0 + tid;
      const int c = e < E ? cnt[e] : 0;
      const int nti = (c + tile - 1) / tile;
      int rs = c, ts = nti;   // inclusive sums over the lanes
#pragma unroll
      for (int o = 1; o < 32; o <<= 1) {
        const int a = __shfl_up_sync(0xffffffffu, rs, o), b = __shfl_up_sync(0xffffffffu, ts, o);
        if (tid >= o) { rs += a; ts += b; }
      }
      const int r0 = row_base + rs - c, t0 = tile_base + ts - nti;
      for (int j = 0; j < nti; ++j)
        if (t0 + j < max_tiles) tiles[t0 + j] = make_int4(e, r0 + j * tile, min(tile, c - j * tile), 0);
      if (e < E) cnt[e] = r0;
      row_base += __shfl_sync(0xffffffffu, rs, 31);
      tile_base += __shfl_sync(0xffffffffu, ts, 31);
    }
    if (tid == 0) n_tiles[layer] = min(tile_base, max_tiles);
  }
  __syncthreads();
  for (long long p = tid; p < pairs; p += nt) rows[p] = atomicAdd(&cnt[expert_of(p)], 1);
}

// 128 x 64 output tile per CTA, 256 threads with 8 x 4 outputs each, K in steps of 16.
__global__ void __launch_bounds__(256)
grouped_gemm_f32_kernel(const float* __restrict__ A, long long lda, const float* __restrict__ W, long long ldw,
                        float* __restrict__ C, long long ldc, int N, int K, const int4* __restrict__ tiles,
                        const int* __restrict__ n_tiles, int gelu) {
  constexpr int TM = 128, TN = 64, TK = 16;
  __shared__ float as[TK][TM + 4];
  __shared__ float ws[TK][TN + 4];
  if ((int)blockIdx.x >= *n_tiles) return;
  const int4 t = tiles[blockIdx.x];
  const int n0 = blockIdx.y * TN, tid = threadIdx.x;
  const int rm = (tid >> 4) * 8, cn = (tid & 15) * 4;
  const float* w0 = W + (long long)t.x * N * ldw;
  float acc[8][4] = {};
  for (int k0 = 0; k0 < K; k0 += TK) {
    for (int i = tid; i < TM * TK; i += 256) {
      const int m = i / TK, k = i % TK;
      as[k][m] = (m < t.z && k0 + k < K) ? A[(long long)(t.y + m) * lda + k0 + k] : 0.f;
    }
    for (int i = tid; i < TN * TK; i += 256) {
      const int nn = i / TK, k = i % TK;
      ws[k][nn] = (n0 + nn < N && k0 + k < K) ? w0[(long long)(n0 + nn) * ldw + k0 + k] : 0.f;
    }
    __syncthreads();
#pragma unroll
    for (int k = 0; k < TK; ++k) {
      float x[8], y[4];
#pragma unroll
      for (int i = 0; i < 8; ++i) x[i] = as[k][rm + i];
#pragma unroll
      for (int j = 0; j < 4; ++j) y[j] = ws[k][cn + j];
#pragma unroll
      for (int i = 0; i < 8; ++i)
#pragma unroll
        for (int j = 0; j < 4; ++j) acc[i][j] = fmaf(x[i], y[j], acc[i][j]);
    }
    __syncthreads();
  }
#pragma unroll
  for (int i = 0; i < 8; ++i)
    if (rm + i < t.z)
#pragma unroll
      for (int j = 0; j < 4; ++j)
        if (n0 + cn + j < N)
          C[(long long)(t.y + rm + i) * ldc + n0 + cn + j] = gelu ? gelu_erf(acc[i][j]) : acc[i][j];
}

}  // namespace cb

namespace cosmos {

static bool aligned(const void* p, size_t bytes) { return (reinterpret_cast<uintptr_t>(p) % bytes) == 0; }

template <typename T, typename Y, int VEC>
static void launch_residual_norm(const ResidualNormArgs& a, int threads, cudaStream_t s) {
  const size_t smem = (size_t)a.d * sizeof(float);
  if (smem > 48 * 1024) {
    static size_t granted = 0;
    if (smem > granted) {
      if (cudaFuncSetAttribute(cb::residual_norm_kernel<T, Y, VEC>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem) !=
          cudaSuccess)
        throw std::runtime_error("residual_norm: row too long");
      granted = smem;
    }
  }
  cb::residual_norm_kernel<T, Y, VEC><<<(unsigned)a.rows, threads, smem, s>>>(a);
}

void residual_norm(const ResidualNormArgs& a, cudaStream_t s) {
  if (a.rows <= 0) return;
  if (a.groups < 1 || a.d % a.groups != 0) throw std::runtime_error("residual_norm: the width must be a multiple of the norm groups");
  const int psize = a.d / a.groups;
  const size_t te = a.is_f32 ? 4 : 2, ye = a.y_f32 ? 4 : te;
  const bool vec = psize % 4 == 0 && a.ldy % 4 == 0 && a.split_stride % 4 == 0 && a.ldh % 4 == 0 && a.ld_embed % 4 == 0 &&
                   aligned(a.x, 16) && aligned(a.y, 4 * ye) && aligned(a.h, 4 * te) && aligned(a.gamma, 4 * te) &&
                   aligned(a.embed, 4 * te);
  // whole prompts with one or two norm parts: rows in registers
  const bool vec8 = vec && psize % 8 == 0 && a.d % 8 == 0 && a.groups <= 2 && a.d <= 8192 && a.ldy % 8 == 0 &&
                    a.split_stride % 8 == 0 && a.ldh % 8 == 0 && a.ld_embed % 8 == 0 && aligned(a.y, 16) && aligned(a.h, 16) &&
                    aligned(a.gamma, 16) && aligned(a.embed, 16);
  if (vec8 && a.rows > 296 && !a.is_f32 && !a.y_f32) {
    const int vecs = a.d / 8;
    const int nv = vecs <= 256 ? 1 : vecs <= 512 ? 2 : 4;
    const int threads = std::max(32, ((vecs + nv - 1) / nv + 31) / 32 * 32);
    switch (nv) {
      case 1: cb::residual_norm_row_kernel<bf16, bf16, 1><<<(unsigned)a.rows, threads, 0, s>>>(a); break;
      case 2: cb::residual_norm_row_kernel<bf16, bf16, 2><<<(unsigned)a.rows, threads, 0, s>>>(a); break;
      default: cb::residual_norm_row_kernel<bf16, bf16, 4><<<(unsigned)a.rows, threads, 0, s>>>(a); break;
    }
    return;
  }
  // few rows (a decode step): one vector per thread, so that all of a row's loads are in flight together
  const int work = (a.d + (vec ? 4 : 1) - 1) / (vec ? 4 : 1);
  const int cap = a.rows <= 296 ? 1024 : 256;
  const int threads = std::min(cap, std::max(32, (work + 31) / 32 * 32));
  if (a.is_f32) {
    vec ? launch_residual_norm<float, float, 4>(a, threads, s) : launch_residual_norm<float, float, 1>(a, threads, s);
  } else if (a.y_f32) {
    vec ? launch_residual_norm<bf16, float, 4>(a, threads, s) : launch_residual_norm<bf16, float, 1>(a, threads, s);
  } else {
    vec ? launch_residual_norm<bf16, bf16, 4>(a, threads, s) : launch_residual_norm<bf16, bf16, 1>(a, threads, s);
  }
}

void qkv_value_post(const QkvValueArgs& a, cudaStream_t s) {
  if (a.n <= 0) return;
  if (a.dim > 512 || a.vdim > 512) throw std::runtime_error("qkv_value_post: head sizes up to 512");
  const long long warps = a.n * ((a.partial ? a.H : 0) + 2 * a.G);
  if (a.dim % 8 == 0 && a.vdim % 8 == 0 && a.dim <= 256 && a.vdim <= 256 && a.ld % 8 == 0 && a.ld_partial % 8 == 0 &&
      a.split_stride % 8 == 0 && aligned(a.qkv, 16) && aligned(a.partial, 16) && aligned(a.bias, 16) &&
      aligned(a.q_out, 16) && aligned(a.k_cache, 16) && aligned(a.v_cache, 16) && aligned(a.v_first_out, 16) &&
      aligned(a.v_first_in, 16)) {
    int lanes = 1;
    while (lanes * 8 < std::max(a.dim, a.vdim)) lanes *= 2;
    const unsigned blocks = (unsigned)((warps * lanes + 255) / 256);
    if (a.is_f32)
      cb::qkv_value_post_vec_kernel<float><<<blocks, 256, 0, s>>>(a, lanes);
    else
      cb::qkv_value_post_vec_kernel<bf16><<<blocks, 256, 0, s>>>(a, lanes);
    return;
  }
  const unsigned grid = (unsigned)((warps + 7) / 8);
  if (a.is_f32)
    cb::qkv_value_post_kernel<float><<<grid, 256, 0, s>>>(a);
  else
    cb::qkv_value_post_kernel<bf16><<<grid, 256, 0, s>>>(a);
}

void moe_route(const long long* tokens, long long n, int vocab, const long long* desc, int n_layers, int max_experts,
               int top_max, int* rows, void* tiles, int max_tiles, int* n_tiles, int* status, cudaStream_t s) {
  if (n <= 0 || n_layers <= 0) return;
  if (max_experts < 1 || max_experts > 8192) throw std::runtime_error("moe_route: 1 to 8192 experts");
  const long long pairs = n * top_max;
  const int threads = (int)std::min<long long>(1024, std::max<long long>(64, (pairs + 31) / 32 * 32));
  cb::moe_route_kernel<<<n_layers, threads, max_experts * sizeof(int), s>>>(
      tokens, n, vocab, desc, top_max, rows, reinterpret_cast<int4*>(tiles), max_tiles, n_tiles, status);
}

void grouped_gemm_f32(const float* A, long long lda, const float* W, long long ldw, float* C, long long ldc, int N, int K,
                      const void* tiles, const int* n_tiles, int max_tiles, int gelu, cudaStream_t s) {
  if (max_tiles <= 0 || N <= 0) return;
  cb::grouped_gemm_f32_kernel<<<dim3(max_tiles, (N + 63) / 64), 256, 0, s>>>(
      A, lda, W, ldw, C, ldc, N, K, reinterpret_cast<const int4*>(tiles), n_tiles, gelu);
}

}  // namespace cosmos
