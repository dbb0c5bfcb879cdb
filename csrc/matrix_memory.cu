// Matrix memory (mLSTM, stack.h) on the CUDA cores: the recurrence token by token, for decode steps, 32-bit models, short
// portions and head sizes that the chunked kernel does not take; and the per-head norm with its output gate.
//
// One CTA = one head's slice of MEMORY_SLICE value columns of one sequence. The slice of S stays in registers (a warp holds
// dim / 8 rows, a lane one column) for the whole portion; a tile of 8 tokens is staged in shared memory, the eight warps'
// partial sums of o and n . q are added once per tile. A decode step is a portion of one token: S is read and written once.
#include <algorithm>
#include <stdexcept>

#include "common.cuh"
#include "launch.cuh"
#include "stack.h"
#include "vec.cuh"

namespace cb {

constexpr int MM_VS = cosmos::MEMORY_SLICE, MM_TT = 8;
static_assert(MM_VS == 32, "a lane holds one value column");

__device__ __forceinline__ float log_sigmoid_f32(float x) { return fminf(x, 0.f) - log1pf(expf(-fabsf(x))); }

template <typename T, int DR>   // DR: rows of S per warp, dim <= 8 DR
__global__ void __launch_bounds__(256)
matrix_memory_kernel(const cosmos::MatrixMemoryArgs a) {
  constexpr int DP = 8 * DR, NL = (DR + 31) / 32;
  __shared__ float q_s[MM_TT][DP], k_s[MM_TT][DP], v_s[MM_TT][MM_VS];
  __shared__ float keep_s[MM_TT], take_s[MM_TT], em_s[MM_TT], gi_s[MM_TT], gf_s[MM_TT];
  __shared__ float red_s[MM_TT][8][MM_VS + 1];
  const int tid = threadIdx.x, rg = tid >> 5, lane = tid & 31;
  const int h = blockIdx.y, slice = blockIdx.x, v0 = slice * MM_VS;
  const Portion p = get_portion(a.rows, blockIdx.z);
  T* og = reinterpret_cast<T*>(a.o);
  const int vcol = v0 + lane;
  const bool vin = vcol < a.vdim;
  const long long slot = p.pos0 < 0 ? -1 : get_state_slot(a.rows, p.seq, a.status);
  if (slot < 0) {   // idle slot of a decode batch
    for (int t = rg; t < p.rows; t += 8)
      if (vin) Elem<T>::put(og + (long long)(p.row0 + t) * a.ldo + h * a.vdim + vcol, 0.f);
    return;
  }
  const bool start = p.pos0 == 0;
  const long long sh = slot * a.H + h;
  float* Sg = a.S + sh * a.dim * (long long)a.vdim;
  float* ng = a.n + (sh * gridDim.x + slice) * a.dim;
  float* mg = a.m + sh * gridDim.x + slice;
  float S[DR], nn[NL];
#pragma unroll
  for (int i = 0; i < DR; ++i) {
    const int r = rg * DR + i;
    S[i] = !start && r < a.dim && vin ? Sg[(long long)r * a.vdim + vcol] : 0.f;
  }
#pragma unroll
  for (int l = 0; l < NL; ++l) {
    const int i = lane + 32 * l, r = rg * DR + i;
    nn[l] = !start && i < DR && r < a.dim ? ng[r] : 0.f;
  }
  float m_run = start ? 0.f : *mg;
  for (int t0 = 0; t0 < p.rows; t0 += MM_TT) {
    const int cnt = min(MM_TT, p.rows - t0);
    for (int idx = tid; idx < cnt * DP; idx += 256) {
      const int t = idx / DP, c = idx - t * DP;
      const long long row = p.row0 + t0 + t;
      const bool in = c < a.dim;
      q_s[t][c] = in ? load_source1<T>(a.q, row, h * a.dim + c) * a.q_scale : 0.f;
      k_s[t][c] = in ? load_source1<T>(a.k, row, h * a.dim + c) : 0.f;
    }
    if (rg < cnt) v_s[rg][lane] = vin ? load_source1<T>(a.v, p.row0 + t0 + rg, h * a.vdim + vcol) : 0.f;
    if (tid < cnt) {
      const long long row = p.row0 + t0 + tid;
      gi_s[tid] = a.cap * tanhf((load_source1<float>(a.gates, row, h) + a.gate_bias[h]) / a.cap);
      gf_s[tid] = log_sigmoid_f32(a.cap * tanhf((load_source1<float>(a.gates, row, a.H + h) + a.gate_bias[a.H + h]) / a.cap));
    }
    __syncthreads();
    if (rg == 0) {   // the running maximum, token by token (every lane keeps it)
      for (int t = 0; t < cnt; ++t) {
        const float fm = gf_s[t] + m_run, m_new = fmaxf(fm, gi_s[t]);
        if (lane == 0) {
          keep_s[t] = expf(fm - m_new);
          take_s[t] = expf(gi_s[t] - m_new);
          em_s[t] = expf(-m_new);
        }
        m_run = m_new;
      }
    }
    __syncthreads();
#pragma unroll 1
    for (int t = 0; t < cnt; ++t) {
      const float keep = keep_s[t], tv = take_s[t] * v_s[t][lane], take = take_s[t];
      float o = 0.f;
#pragma unroll
      for (int i = 0; i < DR; ++i) {
        S[i] = fmaf(keep, S[i], k_s[t][rg * DR + i] * tv);
        o = fmaf(q_s[t][rg * DR + i], S[i], o);
      }
      float nq = 0.f;
#pragma unroll
      for (int l = 0; l < NL; ++l) {
        const int i = lane + 32 * l;
        if (i < DR) {
          nn[l] = fmaf(keep, nn[l], take * k_s[t][rg * DR + i]);
          nq = fmaf(nn[l], q_s[t][rg * DR + i], nq);
        }
      }
      nq = warp_add(nq);
      red_s[t][rg][lane] = o;
      if (lane == 0) red_s[t][rg][MM_VS] = nq;
    }
    __syncthreads();
    if (rg < cnt) {
      float o = 0.f, nq = 0.f;
#pragma unroll
      for (int w = 0; w < 8; ++w) {
        o += red_s[rg][w][lane];
        nq += red_s[rg][w][MM_VS];
      }
      o /= fmaxf(fabsf(nq), em_s[rg]) + 1e-6f;
      if (vin) Elem<T>::put(og + (long long)(p.row0 + t0 + rg) * a.ldo + h * a.vdim + vcol, o);
    }
    __syncthreads();
  }
#pragma unroll
  for (int i = 0; i < DR; ++i) {
    const int r = rg * DR + i;
    if (r < a.dim && vin) Sg[(long long)r * a.vdim + vcol] = S[i];
  }
#pragma unroll
  for (int l = 0; l < NL; ++l) {
    const int i = lane + 32 * l, r = rg * DR + i;
    if (i < DR && r < a.dim) ng[r] = nn[l];
  }
  if (tid == 0) *mg = m_run;
}

// One warp per (token, head).
template <typename T, int VEC>
__global__ void __launch_bounds__(256)
head_norm_gate_kernel(const cosmos::HeadNormGateArgs a) {
  const int lane = threadIdx.x & 31;
  const long long w = (long long)blockIdx.x * 8 + (threadIdx.x >> 5);
  if (w >= a.n * a.H) return;
  const long long r = w / a.H;
  const int h = (int)(w - r * a.H), c0 = h * a.vdim;
  const T* o = reinterpret_cast<const T*>(a.o) + r * a.ldo + c0;
  float ss = 0.f;
  for (int c = lane * VEC; c < a.vdim; c += 32 * VEC) {
    float v[VEC];
    Vec<T, VEC>::load(o + c, v);
#pragma unroll
    for (int e = 0; e < VEC; ++e) ss = fmaf(v[e], v[e], ss);
  }
  const float rinv = 1.f / sqrtf(warp_add(ss) / (float)a.vdim + a.eps);
  T* y = reinterpret_cast<T*>(a.y) + r * a.ldy + c0;
  for (int c = lane * VEC; c < a.vdim; c += 32 * VEC) {   // the row is read again from L1
    float v[VEC], g[VEC], wt[VEC];
    Vec<T, VEC>::load(o + c, v);
    load_source<T, VEC>(a.g, r, c0 + c, g);
    Vec<float, VEC>::load(a.w + c0 + c, wt);
#pragma unroll
    for (int e = 0; e < VEC; ++e) v[e] = v[e] * rinv * wt[e] * sigmoid_f32(g[e]);
    Vec<T, VEC>::store(y + c, v);
  }
}

}  // namespace cb

namespace cosmos {

template <typename T>
static void launch_memory(const MatrixMemoryArgs& a, cudaStream_t s) {
  const dim3 grid((a.vdim + MEMORY_SLICE - 1) / MEMORY_SLICE, a.H, a.rows.n);
  const int per = (a.dim + 7) / 8;
  if (per <= 2) cb::matrix_memory_kernel<T, 2><<<grid, 256, 0, s>>>(a);
  else if (per <= 4) cb::matrix_memory_kernel<T, 4><<<grid, 256, 0, s>>>(a);
  else if (per <= 8) cb::matrix_memory_kernel<T, 8><<<grid, 256, 0, s>>>(a);
  else if (per <= 16) cb::matrix_memory_kernel<T, 16><<<grid, 256, 0, s>>>(a);
  else if (per <= 32) cb::matrix_memory_kernel<T, 32><<<grid, 256, 0, s>>>(a);
  else cb::matrix_memory_kernel<T, 64><<<grid, 256, 0, s>>>(a);
}

void matrix_memory(const MatrixMemoryArgs& a, cudaStream_t s) {
  if (a.rows.n <= 0 || a.H <= 0) return;
  if (a.dim < 1 || a.dim > MEMORY_MAX_DIM) throw std::runtime_error("matrix_memory: key sizes up to 512");
  if (a.rows.n > 65535) throw std::runtime_error("matrix_memory: up to 65535 sequences a step");
  a.is_f32 ? launch_memory<float>(a, s) : launch_memory<bf16>(a, s);
}

void head_norm_gate(const HeadNormGateArgs& a, cudaStream_t s) {
  if (a.n <= 0) return;
  auto on = [](const void* p) { return (reinterpret_cast<uintptr_t>(p) & 15) == 0; };
  const bool vec = a.vdim % 8 == 0 && a.ldo % 8 == 0 && a.ldy % 8 == 0 && a.g.ld % 8 == 0 && a.g.split_stride % 8 == 0 && on(a.o) &&
                   on(a.y) && on(a.g.p) && on(a.w);
  const unsigned grid = (unsigned)((a.n * a.H + 7) / 8);
  if (a.is_f32)
    vec ? cb::head_norm_gate_kernel<float, 8><<<grid, 256, 0, s>>>(a) : cb::head_norm_gate_kernel<float, 1><<<grid, 256, 0, s>>>(a);
  else
    vec ? cb::head_norm_gate_kernel<bf16, 8><<<grid, 256, 0, s>>>(a) : cb::head_norm_gate_kernel<bf16, 1><<<grid, 256, 0, s>>>(a);
}

}  // namespace cosmos
