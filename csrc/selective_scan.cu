// Selective scan (stack.h): causal convolution with its state, the scan over portions of prompts, and the decode step.
//
// Scan over a portion: a CTA owns CH channels of one portion. Half of its warps scan: four lanes a channel, NS of its states per
// lane in registers for the whole portion, one exponential and two packed pairs of multiply-adds per state and token; the sums
// over a channel's four lanes are reduced for four tokens at a time (three exchanges), after which each lane holds one token's.
// The other warps feed them: they load the next tile of 32 tokens, compute softplus, dt * u and the gate silu(z) once per (token,
// channel), and write out the finished tile before the current one. The two halves meet once per tile.
#include <algorithm>
#include <stdexcept>

#include "common.cuh"
#include "launch.cuh"
#include "stack.h"
#include "vec.cuh"

namespace cb {

__device__ __forceinline__ float silu_fast(float z) { return __fdividef(z, 1.f + fast_ex2(-1.4426950408889634f * fmaxf(z, -80.f))); }

// ------------------------------------------------------------------ causal convolution
// Rows of finished values, 8 channels per thread: the loads of the next rows are in flight while one is worked on.
template <typename T, int TAPS>
__global__ void __launch_bounds__(128)
causal_conv_rows_kernel(const cosmos::CausalConvArgs a) {
  const int c = (blockIdx.x * blockDim.x + threadIdx.x) * 8;
  if (c >= a.inner) return;
  const int* tile = a.tiles + (long long)blockIdx.y * 8;
  const int seq = tile[0], row0 = tile[1], rows = tile[2], pos0 = tile[3], first = tile[4];
  const long long slot = get_state_slot(a.rows, seq, a.status);
  if (slot < 0) return;
  const T* x = reinterpret_cast<const T*>(a.x.p) + c;
  const T* st = reinterpret_cast<const T*>(a.conv_state) + slot * (TAPS - 1) * a.inner + c;
  T* u = reinterpret_cast<T*>(a.u) + c;
  constexpr int AHEAD = 8, H = TAPS > 1 ? TAPS - 1 : 1;
  Raw<T, 8> nx[AHEAD];
#pragma unroll
  for (int i = 0; i < AHEAD; ++i) nx[i].load(x + (long long)(row0 + min(i, rows - 1)) * a.x.ld);
  float hist[H][8], w[TAPS][8], bias[8];
#pragma unroll
  for (int j = 0; j < TAPS - 1; ++j) {
    const int src = row0 - (TAPS - 1) + j;
    if (src >= first) {
      Vec<T, 8>::load(x + (long long)src * a.x.ld, hist[j]);
    } else if (pos0 > 0) {
      Vec<T, 8>::load(st + (long long)(TAPS - 1 + src - first) * a.inner, hist[j]);
    } else {
#pragma unroll
      for (int e = 0; e < 8; ++e) hist[j][e] = 0.f;
    }
  }
  Vec<float, 8>::load(a.b + c, bias);
  float wr[8 * TAPS];   // the 8 channels' taps lie side by side
#pragma unroll
  for (int k = 0; k < 2 * TAPS; ++k) Vec<float, 4>::load(a.w + (long long)c * TAPS + 4 * k, *reinterpret_cast<float(*)[4]>(&wr[4 * k]));
#pragma unroll
  for (int e = 0; e < 8; ++e)
#pragma unroll
    for (int j = 0; j < TAPS; ++j) w[j][e] = wr[e * TAPS + j];
  for (int r8 = 0; r8 < rows; r8 += AHEAD) {
#pragma unroll
    for (int i = 0; i < AHEAD; ++i) {
      const int r = r8 + i;
      float v[8], s[8];
      nx[i].get(v);
      nx[i].load(x + (long long)(row0 + min(r + AHEAD, rows - 1)) * a.x.ld);
#pragma unroll
      for (int e = 0; e < 8; ++e) {
        s[e] = bias[e];
#pragma unroll
        for (int j = 0; j < TAPS - 1; ++j) s[e] = fmaf(w[j][e], hist[j][e], s[e]);
        s[e] = silu_fast(fmaf(w[TAPS - 1][e], v[e], s[e]));
#pragma unroll
        for (int j = 0; j + 1 < TAPS - 1; ++j) hist[j][e] = hist[j + 1][e];
        hist[H - 1][e] = v[e];
      }
      if (r < rows) Vec<T, 8>::store(u + (long long)(row0 + r) * a.ldu, s);
    }
  }
}

// grid (channel blocks, tiles or sequences). A decode step updates the conv state here (a thread owns its channels); portions do
// it in conv_state_kernel, because another tile of the portion may still read the old state.
template <typename T, int VEC, int TAPS>   // TAPS 0: any number up to CONV_MAX_TAPS
__global__ void __launch_bounds__(128)
causal_conv_kernel(const cosmos::CausalConvArgs a) {
  const int c = (blockIdx.x * blockDim.x + threadIdx.x) * VEC;
  if (c >= a.inner) return;
  const int taps = TAPS ? TAPS : a.taps;
  int seq, row0, rows, pos0, first;
  if (a.tiles) {
    const int* t = a.tiles + (long long)blockIdx.y * 8;
    seq = t[0]; row0 = t[1]; rows = t[2]; pos0 = t[3]; first = t[4];
  } else {
    const Portion p = get_portion(a.rows, blockIdx.y);
    seq = p.seq; row0 = p.row0; rows = 1; pos0 = p.pos0; first = p.row0;
  }
  T* u = reinterpret_cast<T*>(a.u);
  const long long slot = pos0 < 0 ? -1 : get_state_slot(a.rows, seq, a.status);
  if (slot < 0) {   // idle slot of a decode batch
    float z[VEC];
#pragma unroll
    for (int e = 0; e < VEC; ++e) z[e] = 0.f;
    for (int r = 0; r < rows; ++r) Vec<T, VEC>::store(u + (long long)(row0 + r) * a.ldu + c, z);
    return;
  }
  T* st = reinterpret_cast<T*>(a.conv_state) + slot * (taps - 1) * a.inner + c;
  constexpr int H = TAPS ? (TAPS > 1 ? TAPS - 1 : 1) : cosmos::CONV_MAX_TAPS - 1;
  float hist[H][VEC];   // inputs of the tokens before the current one, oldest first
#pragma unroll
  for (int j = 0; j < H; ++j) {
    if (j >= taps - 1) break;
    const int src = row0 - (taps - 1) + j;
    if (src >= first) {
      load_source<T, VEC>(a.x, src, c, hist[j]);
    } else if (pos0 > 0) {
      Vec<T, VEC>::load(st + (long long)(taps - 1 + src - first) * a.inner, hist[j]);
    } else {
#pragma unroll
      for (int e = 0; e < VEC; ++e) hist[j][e] = 0.f;
    }
  }
  float w[H + 1][VEC], bias[VEC];
  Vec<float, VEC>::load(a.b + c, bias);
#pragma unroll
  for (int j = 0; j < H + 1; ++j) {
    if (j >= taps) break;
#pragma unroll
    for (int e = 0; e < VEC; ++e) w[j][e] = a.w[(long long)(c + e) * taps + j];
  }
  for (int r = 0; r < rows; ++r) {
    float x[VEC], s[VEC];
    load_source<T, VEC>(a.x, row0 + r, c, x);
    if (a.x.k_splits) {   // the state keeps inputs in the element type: take the same value for the current token
#pragma unroll
      for (int e = 0; e < VEC; ++e) {
        T t;
        Elem<T>::put(&t, x[e]);
        x[e] = Elem<T>::get(&t);
      }
    }
#pragma unroll
    for (int e = 0; e < VEC; ++e) s[e] = bias[e];
#pragma unroll
    for (int j = 0; j < H; ++j) {
      if (j >= taps - 1) break;
#pragma unroll
      for (int e = 0; e < VEC; ++e) s[e] = fmaf(w[j][e], hist[j][e], s[e]);
    }
#pragma unroll
    for (int e = 0; e < VEC; ++e) {
      const float wl = TAPS ? w[TAPS ? TAPS - 1 : 0][e] : a.w[(long long)(c + e) * taps + taps - 1];
      s[e] = silu_fast(fmaf(wl, x[e], s[e]));
    }
    Vec<T, VEC>::store(u + (long long)(row0 + r) * a.ldu + c, s);
#pragma unroll
    for (int j = 0; j + 1 < H; ++j) {
      if (j + 1 >= taps - 1) break;
#pragma unroll
      for (int e = 0; e < VEC; ++e) hist[j][e] = hist[j + 1][e];
    }
    if (taps > 1) {
      if (TAPS) {
#pragma unroll
        for (int e = 0; e < VEC; ++e) hist[H - 1][e] = x[e];
      } else {
#pragma unroll
        for (int j = 0; j < H; ++j)
          if (j == taps - 2) {
#pragma unroll
            for (int e = 0; e < VEC; ++e) hist[j][e] = x[e];
          }
      }
    }
  }
  if (!a.tiles) {
#pragma unroll
    for (int j = 0; j < H; ++j) {
      if (j >= taps - 1) break;
      Vec<T, VEC>::store(st + (long long)j * a.inner, hist[j]);
    }
  }
}

// The portion's last taps - 1 inputs become the state (grid: channel blocks, portions).
template <typename T>
__global__ void __launch_bounds__(256)
conv_state_kernel(const cosmos::CausalConvArgs a) {
  const int c = blockIdx.x * blockDim.x + threadIdx.x;
  if (c >= a.inner) return;
  const Portion p = get_portion(a.rows, blockIdx.y);
  const long long slot = get_state_slot(a.rows, p.seq, a.status);
  if (slot < 0 || p.rows <= 0) return;
  const int keep = a.taps - 1;
  T* st = reinterpret_cast<T*>(a.conv_state) + slot * keep * a.inner + c;
  for (int j = 0; j < keep; ++j) {   // ascending: an old entry is read before it is overwritten
    const int i = p.rows - keep + j;
    float x = 0.f;
    if (i >= 0)
      x = load_source1<T>(a.x, p.row0 + i, c);
    else if (p.pos0 > 0)
      x = Elem<T>::get(st + (long long)(p.rows + j) * a.inner);
    Elem<T>::put(st + (long long)j * a.inner, x);
  }
}

// ------------------------------------------------------------------ scan
// log(1 + e^x) for the step sizes: max(x, 0) + log(1 + e) with e = e^-|x|, and log(1 + e) = 2 atanh(s), s = e / (2 + e) <= 1/3,
// by the series of atanh, which keeps the digits of a small e.
__device__ __forceinline__ float softplus_f32(float x) {
  const float e = fast_ex2(-1.4426950408889634f * fabsf(x));
  const float s = __fdividef(e, 2.f + e), q = s * s;
  float r = fmaf(q, 1.f / 13.f, 1.f / 11.f);
  r = fmaf(q, r, 1.f / 9.f);
  r = fmaf(q, r, 1.f / 7.f);
  r = fmaf(q, r, 1.f / 5.f);
  r = fmaf(q, r, 1.f / 3.f);
  r = fmaf(q, r, 1.f);
  return fmaf(2.f * s, r, fmaxf(x, 0.f));
}

__device__ __forceinline__ uint64_t pack2(float lo, float hi) {
  uint64_t r;
  asm("mov.b64 %0, {%1, %2};" : "=l"(r) : "f"(lo), "f"(hi));
  return r;
}
__device__ __forceinline__ float2 unpack2(uint64_t v) {
  float2 r;
  asm("mov.b64 {%0, %1}, %2;" : "=f"(r.x), "=f"(r.y) : "l"(v));
  return r;
}
__device__ __forceinline__ uint64_t mul2(uint64_t a, uint64_t b) {
  uint64_t r;
  asm("mul.rn.f32x2 %0, %1, %2;" : "=l"(r) : "l"(a), "l"(b));
  return r;
}
__device__ __forceinline__ uint64_t fma2(uint64_t a, uint64_t b, uint64_t c) {
  uint64_t r;
  asm("fma.rn.f32x2 %0, %1, %2, %3;" : "=l"(r) : "l"(a), "l"(b), "l"(c));
  return r;
}

// NP pairs in storage form from shared memory (8-byte aligned) as fp32 pairs.
template <int NP>
__device__ __forceinline__ void load_pairs(const float* p, uint64_t (&v)[NP]) {
  if constexpr (NP % 2 == 0) {
#pragma unroll
    for (int i = 0; i < NP; i += 2) {
      const ulonglong2 x = *reinterpret_cast<const ulonglong2*>(p + 2 * i);
      v[i] = x.x; v[i + 1] = x.y;
    }
  } else {
#pragma unroll
    for (int i = 0; i < NP; ++i) v[i] = *reinterpret_cast<const unsigned long long*>(p + 2 * i);
  }
}
template <int NP>
__device__ __forceinline__ void load_pairs(const bf16* p, uint64_t (&v)[NP]) {
  uint32_t w[NP];
  if constexpr (NP % 4 == 0) {
#pragma unroll
    for (int i = 0; i < NP; i += 4) {
      const uint4 x = *reinterpret_cast<const uint4*>(p + 2 * i);
      w[i] = x.x; w[i + 1] = x.y; w[i + 2] = x.z; w[i + 3] = x.w;
    }
  } else {
#pragma unroll
    for (int i = 0; i < NP; i += 2) {
      const uint2 x = *reinterpret_cast<const uint2*>(p + 2 * i);
      w[i] = x.x; w[i + 1] = x.y;
    }
  }
#pragma unroll
  for (int i = 0; i < NP; ++i) v[i] = pack2(bf16lo(w[i]), bf16hi(w[i]));
}

constexpr int SC_TT = 32;   // tokens per tile

// The two halves of the CTA meet here from different places in the code.
template <int N>
__device__ __forceinline__ void tile_barrier() {
  asm volatile("barrier.sync 1, %0;" ::"n"(N) : "memory");
}

// Row strides are such that the four lanes of a channel, which finish four different tokens, meet different banks.
template <typename T, int NS, int CH>
struct ScanSmem {
  float2 du[2][SC_TT][CH];                   // dt, dt * u
  float2 uz[2][SC_TT][CH + 4];               // u, silu(z)
  float y[2][SC_TT][CH + 8];                 // finished output
  __align__(16) T bc[2][SC_TT][4][2 * NS];   // NS values of B, then of C, for each of a channel's four lanes
};

// FAST: finished, aligned rows and N = 4 NS, loaded a tile ahead; otherwise rows are loaded when their tile is made.
template <typename T, int NS, int CH, bool FAST>
__global__ void __launch_bounds__(8 * CH)
selective_scan_kernel(const cosmos::SelectiveScanArgs a) {
  constexpr int NT = 4 * CH, NP = NS / 2, Q = CH / 4, ROWS = SC_TT * Q / NT;   // threads of a half; a feeder loads ROWS x 4 values
  static_assert(NS % 2 == 0 && NT % 32 == 0 && ROWS * NT == SC_TT * Q, "tile shape");
  extern __shared__ __align__(16) uint8_t sm_raw[];
  using Smem = ScanSmem<T, NS, CH>;
  Smem& sm = *reinterpret_cast<Smem*>(sm_raw);
  const Portion p = get_portion(a.rows, blockIdx.y);
  if (p.rows <= 0) return;
  const long long slot = get_state_slot(a.rows, p.seq, a.status);
  if (slot < 0) return;
  const int c0 = blockIdx.x * CH, N = a.state;
  const int n_tiles = (p.rows + SC_TT - 1) / SC_TT;
  if (threadIdx.x < NT) {
    // ---------------- scan
    const int tid = threadIdx.x, ch = tid >> 2, lane4 = tid & 3, c = c0 + ch;
    const bool live = c < a.inner;
    uint64_t S[NP], a2[NP];
    float* sp = a.S + (slot * a.inner + c) * (long long)N + lane4 * NS;
    const float* ap = a.a2 + (long long)c * N + lane4 * NS;
#pragma unroll
    for (int i = 0; i < NP; ++i) {
      const bool i0 = live && lane4 * NS + 2 * i < N, i1 = live && lane4 * NS + 2 * i + 1 < N;
      S[i] = pack2(i0 && p.pos0 > 0 ? sp[2 * i] : 0.f, i1 && p.pos0 > 0 ? sp[2 * i + 1] : 0.f);
      a2[i] = pack2(i0 ? ap[2 * i] : 0.f, i1 ? ap[2 * i + 1] : 0.f);
    }
    const float D = live ? a.D[c] : 0.f;
    for (int k = 0; k < n_tiles; ++k) {
      const int b = k & 1;
      tile_barrier<8 * CH>();   // tile k is in place
      // the next four tokens' rows are read before the current four's output is stored
      float2 du[4];
      uint64_t BC[4][2 * NP];
      auto rows = [&](int t4) {
#pragma unroll
        for (int j = 0; j < 4; ++j) {
          du[j] = sm.du[b][t4 + j][ch];
          load_pairs<2 * NP>(&sm.bc[b][t4 + j][lane4][0], BC[j]);
        }
      };
      rows(0);
#pragma unroll 2
      for (int t4 = 0; t4 < SC_TT; t4 += 4) {
        const float2 v = sm.uz[b][t4 + lane4][ch];
        float acc[4];
#pragma unroll
        for (int j = 0; j < 4; ++j) {
          const uint64_t dt2 = pack2(du[j].x, du[j].x), x2 = pack2(du[j].y, du[j].y);
          uint64_t s = 0ull;
#pragma unroll
          for (int i = 0; i < NP; ++i) {
            const float2 e = unpack2(mul2(dt2, a2[i]));
            S[i] = fma2(pack2(fast_ex2(e.x), fast_ex2(e.y)), S[i], mul2(x2, BC[j][i]));
            s = fma2(S[i], BC[j][NP + i], s);
          }
          const float2 r = unpack2(s);
          acc[j] = r.x + r.y;
        }
        rows(min(t4 + 4, SC_TT - 4));
        // four sums over four lanes, one left on each lane: lane l ends with token t4 + l
        const float x0 = (lane4 & 1) ? acc[0] : acc[1], x1 = (lane4 & 1) ? acc[2] : acc[3];
        const float g0 = __shfl_xor_sync(0xffffffffu, x0, 1), g1 = __shfl_xor_sync(0xffffffffu, x1, 1);
        const float h0 = ((lane4 & 1) ? acc[1] : acc[0]) + g0, h1 = ((lane4 & 1) ? acc[3] : acc[2]) + g1;
        const float g2 = __shfl_xor_sync(0xffffffffu, (lane4 & 2) ? h0 : h1, 2);
        const float y = ((lane4 & 2) ? h1 : h0) + g2;
        sm.y[b][t4 + lane4][ch] = fmaf(D, v.x, y) * v.y;
      }
    }
    tile_barrier<8 * CH>();     // the last tile is finished
#pragma unroll
    for (int i = 0; i < NP; ++i) {
      const float2 v = unpack2(S[i]);
      if (live && lane4 * NS + 2 * i < N) sp[2 * i] = v.x;
      if (live && lane4 * NS + 2 * i + 1 < N) sp[2 * i + 1] = v.y;
    }
    return;
  }
  // ---------------- feed
  const int tid = threadIdx.x - NT;
  constexpr int STEP = NT / Q;
  const int lt = tid / Q, lq = (tid % Q) * 4, lc = c0 + lq;   // tokens lt + r * STEP, channels lc .. lc + 3
  float bias[4];
#pragma unroll
  for (int e = 0; e < 4; ++e) bias[e] = lc + e < a.inner ? a.dt_bias[lc + e] : 0.f;
  const T* ug = reinterpret_cast<const T*>(a.u);
  T* yg = reinterpret_cast<T*>(a.y);
  const bool vec_y = FAST || (a.inner % 4 == 0 && a.ldy % 4 == 0 && (reinterpret_cast<uintptr_t>(a.y) & 15) == 0);
  constexpr int NBC = (SC_TT * 2 * NS + NT - 1) / NT;   // B / C groups of four that a thread loads
  Raw<T, 4> ru[FAST ? ROWS : 1], rd[FAST ? ROWS : 1], rz[FAST ? ROWS : 1], rbc[FAST ? NBC : 1];
  auto fetch = [&](int t0) {   // rows beyond the portion: its last one again
    if constexpr (FAST) {
      const int cc = min(lc, a.inner - 4);
#pragma unroll
      for (int r = 0; r < ROWS; ++r) {
        const long long row = p.row0 + min(t0 + lt + r * STEP, p.rows - 1);
        ru[r].load(ug + row * a.ldu + cc);
        rd[r].load(reinterpret_cast<const T*>(a.dt.p) + row * a.dt.ld + cc);
        rz[r].load(reinterpret_cast<const T*>(a.z.p) + row * a.z.ld + cc);
      }
#pragma unroll
      for (int k = 0; k < NBC; ++k) {
        const int idx = min(tid + k * NT, SC_TT * 2 * NS - 1);
        const int tt = idx / (2 * NS), w = idx - tt * 2 * NS;
        rbc[k].load(reinterpret_cast<const T*>(a.bc.p) + (p.row0 + min(t0 + tt, p.rows - 1)) * a.bc.ld + 4 * w);
      }
    }
  };
  auto put = [&](int t0, int b) {
#pragma unroll
    for (int r = 0; r < ROWS; ++r) {
      const int t = lt + r * STEP;
      const bool in = t0 + t < p.rows;
      float u4[4], d4[4], z4[4];
      if constexpr (FAST) {
        ru[r].get(u4); rd[r].get(d4); rz[r].get(z4);
      } else {
#pragma unroll
        for (int e = 0; e < 4; ++e) {
          const bool have = in && lc + e < a.inner;
          const long long row = p.row0 + t0 + t;
          u4[e] = have ? Elem<T>::get(ug + row * a.ldu + lc + e) : 0.f;
          d4[e] = have ? load_source1<T>(a.dt, row, lc + e) : 0.f;
          z4[e] = have ? load_source1<T>(a.z, row, lc + e) : 0.f;
        }
      }
      float d[4], z[4];
#pragma unroll
      for (int e = 0; e < 4; ++e) {
        d[e] = in ? softplus_f32(d4[e] + bias[e]) : 0.f;   // tokens beyond the portion leave the state alone (dt = 0)
        z[e] = silu_fast(z4[e]);
      }
      // pieces of two channels; every second group of four threads starts with its upper piece, so that eight threads' 16-byte
      // stores meet all banks
      const bool up = (tid >> 2) & 1;
#pragma unroll
      for (int k = 0; k < 2; ++k) {
        const int e = (k == 0) == up ? 2 : 0;
        const float da = e ? d[2] : d[0], db = e ? d[3] : d[1], ua = e ? u4[2] : u4[0], ub = e ? u4[3] : u4[1];
        *reinterpret_cast<float4*>(&sm.du[b][t][lq + e]) = make_float4(da, da * ua, db, db * ub);
        *reinterpret_cast<float4*>(&sm.uz[b][t][lq + e]) = make_float4(ua, e ? z[2] : z[0], ub, e ? z[3] : z[1]);
      }
    }
    if constexpr (FAST) {
#pragma unroll
      for (int k = 0; k < NBC; ++k) {
        const int idx = tid + k * NT;
        if (idx >= SC_TT * 2 * NS) break;
        const int tt = idx / (2 * NS), w = idx - tt * 2 * NS, half = w / NS, n = (w - half * NS) * 4;
        float v[4];
        rbc[k].get(v);
#pragma unroll
        for (int e = 0; e < 4; e += 2) {
          T* dst = &sm.bc[b][tt][(n + e) / NS][half * NS + (n + e) % NS];
          Elem<T>::put(dst, v[e]);
          Elem<T>::put(dst + 1, v[e + 1]);
        }
      }
    } else {
#pragma unroll 1
      for (int idx = tid; idx < SC_TT * 8 * NS; idx += NT) {
        const int tt = idx / (8 * NS), w = idx - tt * 8 * NS, half = w / (4 * NS), n = w - half * 4 * NS;
        Elem<T>::put(&sm.bc[b][tt][n / NS][half * NS + n % NS],
                     t0 + tt < p.rows && n < N ? load_source1<T>(a.bc, p.row0 + t0 + tt, half * N + n) : 0.f);
      }
    }
  };
  auto flush = [&](int t0, int b) {
#pragma unroll
    for (int r = 0; r < ROWS; ++r) {
      const int t = lt + r * STEP;
      if (t0 + t >= p.rows) continue;
      T* dst = yg + (long long)(p.row0 + t0 + t) * a.ldy + lc;
      float o[4];
      Vec<float, 4>::load(&sm.y[b][t][lq], o);
      if (vec_y) {
        if (lc < a.inner) Vec<T, 4>::store(dst, o);
      } else {
#pragma unroll
        for (int e = 0; e < 4; ++e)
          if (lc + e < a.inner) Elem<T>::put(dst + e, o[e]);
      }
    }
  };
  fetch(0);
  put(0, 0);
  fetch(SC_TT);
  for (int k = 0; k < n_tiles; ++k) {
    tile_barrier<8 * CH>();   // the scan takes tile k; tile k - 1 is finished
    if (k > 0) flush((k - 1) * SC_TT, (k - 1) & 1);
    if (k + 1 < n_tiles) {
      put((k + 1) * SC_TT, (k + 1) & 1);
      fetch((k + 2) * SC_TT);
    }
  }
  tile_barrier<8 * CH>();
  flush((n_tiles - 1) * SC_TT, (n_tiles - 1) & 1);
}

// One token per sequence: four lanes a channel, the state read and written once.
template <typename T, int NS>
__global__ void __launch_bounds__(256)
selective_step_kernel(const cosmos::SelectiveScanArgs a) {
  const Portion p = get_portion(a.rows, blockIdx.y);
  const int lane4 = threadIdx.x & 3, c = (blockIdx.x * blockDim.x + threadIdx.x) >> 2, N = a.state;
  if (c >= a.inner) return;   // whole groups of four lanes
  T* y = reinterpret_cast<T*>(a.y) + (long long)p.row0 * a.ldy + c;
  const long long slot = p.pos0 < 0 ? -1 : get_state_slot(a.rows, p.seq, a.status);
  if (slot < 0) {
    if (lane4 == 0) Elem<T>::put(y, 0.f);
    return;
  }
  float* sp = a.S + (slot * a.inner + c) * (long long)N + lane4 * NS;
  const float* ap = a.a2 + (long long)c * N + lane4 * NS;
  float S[NS], a2[NS];
  const bool full = NS % 4 == 0 && N == 4 * NS;
  if (full) {
#pragma unroll
    for (int i = 0; i < NS; i += 4) {
      if constexpr (NS % 4 == 0) {
        Vec<float, 4>::load(ap + i, *reinterpret_cast<float(*)[4]>(&a2[i]));
        if (p.pos0 > 0) Vec<float, 4>::load(sp + i, *reinterpret_cast<float(*)[4]>(&S[i]));
      }
    }
  } else {
#pragma unroll
    for (int i = 0; i < NS; ++i) {
      const bool in = lane4 * NS + i < N;
      a2[i] = in ? ap[i] : 0.f;
      S[i] = in ? sp[i] : 0.f;
    }
  }
  if (p.pos0 == 0) {
#pragma unroll
    for (int i = 0; i < NS; ++i) S[i] = 0.f;
  }
  const float u = Elem<T>::get(reinterpret_cast<const T*>(a.u) + (long long)p.row0 * a.ldu + c);
  const float dt = softplus_f32(load_source1<T>(a.dt, p.row0, c) + a.dt_bias[c]);
  float s = 0.f;
#pragma unroll
  for (int i = 0; i < NS; ++i) {
    const int n = lane4 * NS + i;
    const bool in = n < N;
    const float B = in ? load_source1<T>(a.bc, p.row0, n) : 0.f, C = in ? load_source1<T>(a.bc, p.row0, N + n) : 0.f;
    S[i] = fmaf(fast_ex2(dt * a2[i]), S[i], dt * u * B);
    s = fmaf(S[i], C, s);
  }
  const unsigned mask = 0xfu << ((threadIdx.x & 31) & ~3);
  s += __shfl_xor_sync(mask, s, 1);
  s += __shfl_xor_sync(mask, s, 2);
  if (full) {
#pragma unroll
    for (int i = 0; i < NS; i += 4)
      if constexpr (NS % 4 == 0) Vec<float, 4>::store(sp + i, *reinterpret_cast<float(*)[4]>(&S[i]));
  } else {
#pragma unroll
    for (int i = 0; i < NS; ++i)
      if (lane4 * NS + i < N) sp[i] = S[i];
  }
  if (lane4 == 0) Elem<T>::put(y, fmaf(a.D[c], u, s) * silu_f32(load_source1<T>(a.z, p.row0, c)));
}

// Columns [inner, y_cols) of y: the product behind reads whole 16-byte pieces.
template <typename T>
__global__ void zero_cols_kernel(T* y, long long ldy, int c0, int cols, long long n) {
  const long long i = (long long)blockIdx.x * blockDim.x + threadIdx.x;
  if (i < n * cols) Elem<T>::put(y + i / cols * ldy + c0 + i % cols, 0.f);
}

}  // namespace cb

namespace cosmos {

template <typename T>
static void launch_conv(const CausalConvArgs& a, cudaStream_t s) {
  auto on = [](const void* p) { return (reinterpret_cast<uintptr_t>(p) & 15) == 0; };
  const bool vec = a.inner % 8 == 0 && a.x.ld % 8 == 0 && a.x.split_stride % 8 == 0 && a.ldu % 8 == 0 && on(a.x.p) && on(a.u) &&
                   on(a.conv_state) && on(a.b) && on(a.w);
  const int v = vec && a.taps <= 4 ? 8 : 1;
  const int per = (a.inner + v - 1) / v, threads = std::min(128, (per + 31) / 32 * 32);
  const dim3 grid((per + threads - 1) / threads, a.tiles ? a.n_tiles : a.rows.n);
  if (v == 8 && a.tiles && a.x.k_splits == 0) {
    switch (a.taps) {
      case 1: cb::causal_conv_rows_kernel<T, 1><<<grid, threads, 0, s>>>(a); break;
      case 2: cb::causal_conv_rows_kernel<T, 2><<<grid, threads, 0, s>>>(a); break;
      case 3: cb::causal_conv_rows_kernel<T, 3><<<grid, threads, 0, s>>>(a); break;
      default: cb::causal_conv_rows_kernel<T, 4><<<grid, threads, 0, s>>>(a); break;
    }
  } else if (v == 8) {
    switch (a.taps) {
      case 1: cb::causal_conv_kernel<T, 8, 1><<<grid, threads, 0, s>>>(a); break;
      case 2: cb::causal_conv_kernel<T, 8, 2><<<grid, threads, 0, s>>>(a); break;
      case 3: cb::causal_conv_kernel<T, 8, 3><<<grid, threads, 0, s>>>(a); break;
      default: cb::causal_conv_kernel<T, 8, 4><<<grid, threads, 0, s>>>(a); break;
    }
  } else {
    cb::causal_conv_kernel<T, 1, 0><<<grid, threads, 0, s>>>(a);
  }
  if (a.tiles && a.taps > 1)
    cb::conv_state_kernel<T><<<dim3((a.inner + 255) / 256, a.rows.n), 256, 0, s>>>(a);
}

void causal_conv(const CausalConvArgs& a, cudaStream_t s) {
  if (a.rows.n <= 0 || (a.tiles && a.n_tiles <= 0)) return;
  if (a.taps < 1 || a.taps > CONV_MAX_TAPS) throw std::runtime_error("causal_conv: 1 to 16 taps");
  a.is_f32 ? launch_conv<float>(a, s) : launch_conv<bf16>(a, s);
}

template <typename T, int NS, int CH, bool FAST>
static void launch_scan_ch(const SelectiveScanArgs& a, cudaStream_t s) {
  constexpr int smem = (int)sizeof(cb::ScanSmem<T, NS, CH>);
  static bool granted = false;
  if (!granted && smem > 48 * 1024) {
    if (cudaFuncSetAttribute(cb::selective_scan_kernel<T, NS, CH, FAST>, cudaFuncAttributeMaxDynamicSharedMemorySize, smem) != cudaSuccess)
      throw std::runtime_error("selective_scan: shared memory not available");
    granted = true;
  }
  cb::selective_scan_kernel<T, NS, CH, FAST><<<dim3((a.inner + CH - 1) / CH, a.rows.n), 8 * CH, smem, s>>>(a);
}

template <typename T, int NS>
static void launch_scan_ns(const SelectiveScanArgs& a, cudaStream_t s) {
  if (!a.rows.portions) {
    cb::selective_step_kernel<T, NS><<<dim3((a.inner + 63) / 64, a.rows.n), 256, 0, s>>>(a);
    return;
  }
  auto on = [](const RowSource& r) { return (reinterpret_cast<uintptr_t>(r.p) & 15) == 0 && r.ld % 4 == 0 && r.k_splits == 0; };
  const bool fast = a.inner % 4 == 0 && a.state == 4 * NS && on(a.dt) && on(a.z) && on(a.bc) && a.ldu % 4 == 0 && a.ldy % 4 == 0 &&
                    (reinterpret_cast<uintptr_t>(a.u) & 15) == 0 && (reinterpret_cast<uintptr_t>(a.y) & 15) == 0;
  if constexpr (NS <= 16) {
    if (fast) {
      // about two CTAs of 32 channels per SM; fewer channels a CTA while that leaves SMs idle
      const long long ctas = (long long)((a.inner + 31) / 32) * a.rows.n;
      if constexpr (sizeof(T) == 2) {
        if (ctas >= 200) return launch_scan_ch<T, NS, 32, true>(a, s);
      }
      return launch_scan_ch<T, NS, 16, true>(a, s);
    }
  }
  launch_scan_ch<T, NS, 16, false>(a, s);
}

template <typename T>
static void launch_scan(const SelectiveScanArgs& a, cudaStream_t s) {
  const int per = (a.state + 3) / 4;
  if (per <= 2) launch_scan_ns<T, 2>(a, s);
  else if (per <= 4) launch_scan_ns<T, 4>(a, s);
  else if (per <= 6) launch_scan_ns<T, 6>(a, s);
  else if (per <= 8) launch_scan_ns<T, 8>(a, s);
  else if (per <= 16) launch_scan_ns<T, 16>(a, s);
  else launch_scan_ns<T, 32>(a, s);
}

void selective_scan(const SelectiveScanArgs& a, cudaStream_t s) {
  if (a.rows.n <= 0 || a.inner <= 0) return;
  if (a.state < 1 || a.state > SCAN_MAX_STATE) throw std::runtime_error("selective_scan: 1 to 128 states a channel");
  a.is_f32 ? launch_scan<float>(a, s) : launch_scan<bf16>(a, s);
}

void zero_cols(void* y, long long ldy, int c0, int c1, long long n, bool is_f32, cudaStream_t s) {
  const int cols = c1 - c0;
  if (cols <= 0 || n <= 0) return;
  const unsigned grid = (unsigned)((n * cols + 255) / 256);
  if (is_f32)
    cb::zero_cols_kernel<float><<<grid, 256, 0, s>>>((float*)y, ldy, c0, cols, n);
  else
    cb::zero_cols_kernel<bf16><<<grid, 256, 0, s>>>((bf16*)y, ldy, c0, cols, n);
}

}  // namespace cosmos
