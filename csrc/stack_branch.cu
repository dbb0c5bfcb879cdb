// Row-wise kernels of parallel layers (stack.h): residual add of normed branches with the two norms that follow it, and the
// norm of queries and keys over the whole projection with the cache write.
#include <algorithm>
#include <stdexcept>

#include "common.cuh"
#include "launch.cuh"
#include "stack.h"
#include "vec.cuh"

namespace cb {

// One CTA per token row; a row's vectors stay in registers, all loads are issued before the first sum.
// PART: some source holds split-K partial sums. EMBED: rows start from the embedding.
template <typename T, int VEC, int NV, bool PART, bool EMBED>
__global__ void __launch_bounds__(NV == 1 ? 1024 : 512)
branch_norm_kernel(const cosmos::BranchNormArgs a) {
  __shared__ float2 buf_s[2][32];
  const long long r = blockIdx.x;
  const int tid = threadIdx.x, nt = blockDim.x, d = a.d;
  float* xr = a.x + r * d;
  float v[NV][VEC], b0[NV][VEC], b1[NV][VEC];
  if constexpr (EMBED) {
    long long tok = a.tokens[r];
    if (!index_ok(tok, a.vocab, a.status, SITE_STACK_TOKEN)) tok = 0;
    const T* er = reinterpret_cast<const T*>(a.embed) + tok * a.ld_embed;
    const double p = a.pos_turns ? (double)a.positions[r] : 0.0;
#pragma unroll
    for (int i = 0; i < NV; ++i) {
      const int c = (tid + i * nt) * VEC;
      if (c < d) {
        Vec<T, VEC>::load(er + c, v[i]);
#pragma unroll
        for (int e = 0; e < VEC; ++e) v[i][e] *= a.embed_scale;
        if (a.pos_turns) {
          // the angle in turns, reduced in double so that far positions keep their digits
#pragma unroll
          for (int e = 0; e < VEC; ++e) {
            double t = p * a.pos_turns[(c + e) >> 1];
            t -= rint(t);
            const float h = 2.f * (float)t;
            v[i][e] += ((c + e) & 1) ? cospif(h) : sinpif(h);
          }
        }
      }
    }
  } else {
#pragma unroll
    for (int i = 0; i < NV; ++i) {
      const int c = (tid + i * nt) * VEC;
      if (c < d) Vec<float, VEC>::load(xr + c, v[i]);
    }
  }
  if (a.n_normed > 0) {
    float s0 = 0.f, s1 = 0.f;
#pragma unroll
    for (int i = 0; i < NV; ++i) {
      const int c = (tid + i * nt) * VEC;
      if (c < d) {
        load_source<T, VEC, PART>(a.normed[0], r, c, b0[i]);
#pragma unroll
        for (int e = 0; e < VEC; ++e) s0 = fmaf(b0[i][e], b0[i][e], s0);
        if (a.n_normed > 1) {
          load_source<T, VEC, PART>(a.normed[1], r, c, b1[i]);
#pragma unroll
          for (int e = 0; e < VEC; ++e) s1 = fmaf(b1[i][e], b1[i][e], s1);
        }
      }
    }
    const float2 ss = block_add2(s0, s1, buf_s[0]);
    const float q0 = a.coef / sqrtf(ss.x / (float)d + a.eps), q1 = a.coef / sqrtf(ss.y / (float)d + a.eps);
#pragma unroll
    for (int i = 0; i < NV; ++i) {
      const int c = (tid + i * nt) * VEC;
      if (c < d) {
        float w[VEC];
        Vec<float, VEC>::load(a.normed_w[0] + c, w);
#pragma unroll
        for (int e = 0; e < VEC; ++e) v[i][e] = fmaf(b0[i][e] * q0, w[e], v[i][e]);
        if (a.n_normed > 1) {
          Vec<float, VEC>::load(a.normed_w[1] + c, w);
#pragma unroll
          for (int e = 0; e < VEC; ++e) v[i][e] = fmaf(b1[i][e] * q1, w[e], v[i][e]);
        }
      }
    }
  }
  float ss = 0.f;
#pragma unroll
  for (int i = 0; i < NV; ++i) {
    const int c = (tid + i * nt) * VEC;
    if (c < d) {
      if (a.has_plain) {
        float t[VEC];
        load_source<T, VEC, PART>(a.plain, r, c, t);
#pragma unroll
        for (int e = 0; e < VEC; ++e) v[i][e] += t[e];
      }
      if (EMBED || a.n_normed || a.has_plain) Vec<float, VEC>::store(xr + c, v[i]);
#pragma unroll
      for (int e = 0; e < VEC; ++e) ss = fmaf(v[i][e], v[i][e], ss);
    }
  }
  if (!a.h[0] && !a.h[1]) return;
  const float rinv = 1.f / sqrtf(block_add2(ss, 0.f, buf_s[1]).x / (float)d + a.eps);
#pragma unroll
  for (int i = 0; i < NV; ++i) {
    const int c = (tid + i * nt) * VEC;
    if (c < d) {
#pragma unroll
      for (int o = 0; o < 2; ++o) {
        if (!a.h[o]) continue;
        float g[VEC];
        Vec<float, VEC>::load(a.gamma[o] + c, g);
#pragma unroll
        for (int e = 0; e < VEC; ++e) g[e] = v[i][e] * rinv * (a.gamma_add + g[e]);
        Vec<T, VEC>::store(reinterpret_cast<T*>(a.h[o]) + r * a.ldh + c, g);
      }
    }
  }
}

// One CTA per token row: the whole q row and the whole k row.
template <typename T, int VEC, int NV, bool PART>
__global__ void __launch_bounds__(NV == 1 ? 1024 : 512)
qk_norm_post_kernel(const cosmos::QkNormArgs a) {
  __shared__ float2 buf_s[32];
  const long long r = blockIdx.x;
  const int tid = threadIdx.x, nt = blockDim.x;
  const int qc = a.H * a.dim, kc = a.G * a.dim;
  const long long slot = a.slots[r], pos = a.temp_every > 0 ? a.positions[r] : 0;
  float q[NV][VEC], k[NV][VEC];
  float sq = 0.f, sk = 0.f;
#pragma unroll
  for (int i = 0; i < NV; ++i) {
    const int c = (tid + i * nt) * VEC;
    if (c < qc) {
      load_source<T, VEC, PART>(a.q, r, c, q[i]);
#pragma unroll
      for (int e = 0; e < VEC; ++e) sq = fmaf(q[i][e], q[i][e], sq);
    }
    if (c < kc) {
      load_source<T, VEC, PART>(a.k, r, c, k[i]);
#pragma unroll
      for (int e = 0; e < VEC; ++e) sk = fmaf(k[i][e], k[i][e], sk);
    }
  }
  const float2 ss = block_add2(sq, sk, buf_s);
  float rq = 1.f / sqrtf(ss.x / (float)qc + a.eps);
  const float rk = 1.f / sqrtf(ss.y / (float)kc + a.eps);
  if (a.temp_every > 0) {
    const unsigned step = (unsigned)(pos + 1) / (unsigned)a.temp_every;   // positions fit 32 bits
    rq *= 1.f + a.temp_coef * logf((float)(step + 1));
  }
  const bool ok = index_ok(slot, a.n_slots, a.status, SITE_STACK_SLOT);
  const unsigned page = ok ? (unsigned)slot / (unsigned)a.page_size : 0u;
  const int off = ok ? (int)((unsigned)slot - page * (unsigned)a.page_size) : 0;
  T* qo = reinterpret_cast<T*>(a.q_out) + r * qc;
#pragma unroll
  for (int i = 0; i < NV; ++i) {
    const int c = (tid + i * nt) * VEC;
    float w[VEC];
    if (c < qc) {
      Vec<float, VEC>::load(a.wq + c, w);
#pragma unroll
      for (int e = 0; e < VEC; ++e) q[i][e] = q[i][e] * rq * w[e];
      Vec<T, VEC>::store(qo + c, q[i]);
    }
    if (c < kc && ok) {
      const int g = c / a.dim;
      const long long row = (((long long)page * a.G + g) * a.page_size + off) * (long long)a.dim + (c - g * a.dim);
      Vec<T, VEC>::store(reinterpret_cast<T*>(a.v_cache) + row, k[i]);
      Vec<float, VEC>::load(a.wk + c, w);
#pragma unroll
      for (int e = 0; e < VEC; ++e) k[i][e] = k[i][e] * rk * w[e];
      Vec<T, VEC>::store(reinterpret_cast<T*>(a.k_cache) + row, k[i]);
    }
  }
}

}  // namespace cb

namespace cosmos {

static bool on(const void* p, size_t bytes) { return (reinterpret_cast<uintptr_t>(p) % bytes) == 0; }
static bool vec8_source(const RowSource& s) { return on(s.p, 16) && s.ld % 8 == 0 && s.split_stride % 8 == 0; }

// Threads for a row of `cols` values: VEC per thread and pass, NV passes.
static int row_threads(int cols, int vec, int nv) {
  const int per = vec * nv;
  return std::max(32, ((cols + per - 1) / per + 31) / 32 * 32);
}

template <typename T, bool PART, bool EMBED>
static void launch_branch(const BranchNormArgs& a, cudaStream_t s) {
  bool vec = a.d % 8 == 0 && a.ldh % 8 == 0 && a.ld_embed % 8 == 0 && on(a.x, 16) && on(a.embed, 16);
  for (int i = 0; i < 2; ++i) vec = vec && on(a.gamma[i], 16) && on(a.h[i], 16) && on(a.normed_w[i], 16) && vec8_source(a.normed[i]);
  if (a.has_plain) vec = vec && vec8_source(a.plain);
  const unsigned rows = (unsigned)a.rows;
  if (vec && a.d <= 8192 && (a.rows <= 296 || a.d <= 1024))
    cb::branch_norm_kernel<T, 8, 1, PART, EMBED><<<rows, row_threads(a.d, 8, 1), 0, s>>>(a);
  else if (vec && a.d <= 8192)
    cb::branch_norm_kernel<T, 8, 2, PART, EMBED><<<rows, row_threads(a.d, 8, 2), 0, s>>>(a);
  else if (a.d <= 1024)
    cb::branch_norm_kernel<T, 1, 1, PART, EMBED><<<rows, row_threads(a.d, 1, 1), 0, s>>>(a);
  else if (a.d <= 16384)
    cb::branch_norm_kernel<T, 1, 32, PART, EMBED><<<rows, row_threads(a.d, 1, 32), 0, s>>>(a);
  else
    throw std::runtime_error("branch_norm: rows of up to 16384 columns");
}

void branch_norm(const BranchNormArgs& a, cudaStream_t s) {
  if (a.rows <= 0) return;
  bool part = a.has_plain && a.plain.k_splits > 0;
  for (int i = 0; i < a.n_normed; ++i) part = part || a.normed[i].k_splits > 0;
  if (a.embed) {
    if (a.n_normed || a.has_plain) throw std::runtime_error("branch_norm: the embedding starts a row");
    a.is_f32 ? launch_branch<float, false, true>(a, s) : launch_branch<bf16, false, true>(a, s);
  } else if (part) {
    a.is_f32 ? launch_branch<float, true, false>(a, s) : launch_branch<bf16, true, false>(a, s);
  } else {
    a.is_f32 ? launch_branch<float, false, false>(a, s) : launch_branch<bf16, false, false>(a, s);
  }
}

template <typename T, bool PART>
static void launch_qk(const QkNormArgs& a, cudaStream_t s) {
  const int cols = std::max(a.H, a.G) * a.dim;
  const bool vec = a.dim % 8 == 0 && vec8_source(a.q) && vec8_source(a.k) && on(a.wq, 16) && on(a.wk, 16) && on(a.q_out, 16) &&
                   on(a.k_cache, 16) && on(a.v_cache, 16);
  const unsigned rows = (unsigned)a.n;
  if (vec && cols <= 8192 && cols > 1024 && a.n > 296)
    cb::qk_norm_post_kernel<T, 8, 2, PART><<<rows, row_threads(cols, 8, 2), 0, s>>>(a);
  else if (vec && cols <= 8192)
    cb::qk_norm_post_kernel<T, 8, 1, PART><<<rows, row_threads(cols, 8, 1), 0, s>>>(a);
  else if (cols <= 1024)
    cb::qk_norm_post_kernel<T, 1, 1, PART><<<rows, row_threads(cols, 1, 1), 0, s>>>(a);
  else if (cols <= 16384)
    cb::qk_norm_post_kernel<T, 1, 32, PART><<<rows, row_threads(cols, 1, 32), 0, s>>>(a);
  else
    throw std::runtime_error("qk_norm_post: projections of up to 16384 columns");
}

void qk_norm_post(const QkNormArgs& a, cudaStream_t s) {
  if (a.n <= 0) return;
  if (a.n_slots > 0xffffffffll || a.temp_every > 0x7fffffff) throw std::runtime_error("qk_norm_post: too many cache slots");
  if (a.q.k_splits || a.k.k_splits)
    a.is_f32 ? launch_qk<float, true>(a, s) : launch_qk<bf16, true>(a, s);
  else
    a.is_f32 ? launch_qk<float, false>(a, s) : launch_qk<bf16, false>(a, s);
}

}  // namespace cosmos
