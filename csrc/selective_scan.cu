// Selective scan (stack.h): causal convolution with its state, the scan over portions of prompts, and the decode step.
//
// Scan over a portion: a CTA owns CH channels of one portion, four lanes a channel, NS of its states per lane in registers for
// the whole portion. Tokens come in tiles of 16: the next tile's rows are loaded into registers while the current one is
// worked on, and softplus, dt * u and the gate silu(z) are computed once per (token, channel) on the way to shared memory.
// What is left per (token, channel, state) is one exponential and four multiply-adds; the sums over a channel's four lanes
// are reduced for four tokens at a time (three exchanges), after which each lane finishes one token.
#include <algorithm>
#include <stdexcept>

#include "common.cuh"
#include "launch.cuh"
#include "stack.h"
#include "vec.cuh"

namespace cb {

// ------------------------------------------------------------------ causal convolution
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
      s[e] = silu_f32(fmaf(wl, x[e], s[e]));
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
__device__ __forceinline__ float softplus_f32(float x) { return fmaxf(x, 0.f) + log1pf(expf(-fabsf(x))); }

constexpr int SC_TT = 16;   // tokens per tile

template <typename T, int NS, int CH>
__global__ void __launch_bounds__(4 * CH)
selective_scan_kernel(const cosmos::SelectiveScanArgs a) {
  constexpr int NT = 4 * CH, Q = CH / 4;   // threads; groups of four channels
  static_assert(NT == SC_TT * Q, "a thread loads four channels of one token");
  __shared__ float2 du_s[2][SC_TT][CH];            // dt, dt * u
  __shared__ float u_s[2][SC_TT][CH];
  __shared__ float z_s[2][SC_TT][CH];              // gate, then the finished output
  __shared__ float bc_s[2][SC_TT][2][4][NS];       // B | C by lane
  const int tid = threadIdx.x, ch = tid >> 2, lane4 = tid & 3;
  const Portion p = get_portion(a.rows, blockIdx.y);
  if (p.rows <= 0) return;
  const long long slot = get_state_slot(a.rows, p.seq, a.status);
  if (slot < 0) return;
  const int c0 = blockIdx.x * CH, c = c0 + ch, N = a.state;
  const bool live = c < a.inner;
  float S[NS], a2[NS];
  float* sp = a.S + (slot * a.inner + c) * (long long)N + lane4 * NS;
#pragma unroll
  for (int i = 0; i < NS; ++i) {
    const bool in = live && lane4 * NS + i < N;
    S[i] = in && p.pos0 > 0 ? sp[i] : 0.f;
    a2[i] = in ? a.a2[(long long)c * N + lane4 * NS + i] : 0.f;
  }
  const float D = live ? a.D[c] : 0.f;
  // loader: token lt, channels lc .. lc + 3 of the tile
  const int lt = tid / Q, lq = (tid % Q) * 4, lc = c0 + lq;
  float ru[4], rd[4], rz[4], bias[4];
#pragma unroll
  for (int e = 0; e < 4; ++e) bias[e] = lc + e < a.inner ? a.dt_bias[lc + e] : 0.f;
  constexpr int NBC = (SC_TT * 8 * NS + NT - 1) / NT;   // B / C values a thread loads
  float rbc[NBC];
  const T* ug = reinterpret_cast<const T*>(a.u);
  const bool vec = a.inner % 4 == 0 && a.ldu % 4 == 0 && a.dt.ld % 4 == 0 && a.z.ld % 4 == 0 && a.dt.split_stride % 4 == 0 &&
                   a.z.split_stride % 4 == 0 && (reinterpret_cast<uintptr_t>(a.u) & 15) == 0 &&
                   (reinterpret_cast<uintptr_t>(a.dt.p) & 15) == 0 && (reinterpret_cast<uintptr_t>(a.z.p) & 15) == 0;
  auto fetch = [&](int t0) {
    const int t = t0 + lt;
    const long long row = p.row0 + t;
    if (t < p.rows && vec && lc < a.inner) {
      Vec<T, 4>::load(ug + row * a.ldu + lc, ru);
      load_source<T, 4>(a.dt, row, lc, rd);
      load_source<T, 4>(a.z, row, lc, rz);
    } else {
#pragma unroll
      for (int e = 0; e < 4; ++e) {
        const bool in = t < p.rows && lc + e < a.inner;
        ru[e] = in ? Elem<T>::get(ug + row * a.ldu + lc + e) : 0.f;
        rd[e] = in ? load_source1<T>(a.dt, row, lc + e) : 0.f;
        rz[e] = in ? load_source1<T>(a.z, row, lc + e) : 0.f;
      }
    }
#pragma unroll
    for (int k = 0; k < NBC; ++k) {
      const int idx = tid + k * NT;
      const int tt = idx / (8 * NS), w = idx - tt * 8 * NS, half = w / (4 * NS), n = w - half * 4 * NS;
      rbc[k] = idx < SC_TT * 8 * NS && t0 + tt < p.rows && n < N ? load_source1<T>(a.bc, p.row0 + t0 + tt, half * N + n) : 0.f;
    }
  };
  auto put = [&](int t0, int b) {
    const bool in = t0 + lt < p.rows;
#pragma unroll
    for (int e = 0; e < 4; ++e) {
      const float dt = in ? softplus_f32(rd[e] + bias[e]) : 0.f;   // tokens beyond the portion leave the state alone
      du_s[b][lt][lq + e] = make_float2(dt, dt * ru[e]);
      u_s[b][lt][lq + e] = ru[e];
      z_s[b][lt][lq + e] = silu_f32(rz[e]);
    }
#pragma unroll
    for (int k = 0; k < NBC; ++k) {
      const int idx = tid + k * NT;
      if (idx < SC_TT * 8 * NS) (&bc_s[b][0][0][0][0])[idx] = rbc[k];
    }
  };
  T* yg = reinterpret_cast<T*>(a.y);
  const bool vec_y = a.inner % 4 == 0 && a.ldy % 4 == 0 && (reinterpret_cast<uintptr_t>(a.y) & 15) == 0;
  fetch(0);
  put(0, 0);
  __syncthreads();
  int b = 0;
  for (int t0 = 0; t0 < p.rows; t0 += SC_TT, b ^= 1) {
    const bool more = t0 + SC_TT < p.rows;
    if (more) fetch(t0 + SC_TT);
#pragma unroll 1
    for (int t4 = 0; t4 < SC_TT; t4 += 4) {
      float acc[4];
#pragma unroll
      for (int j = 0; j < 4; ++j) {
        const float2 du = du_s[b][t4 + j][ch];
        const float* B = bc_s[b][t4 + j][0][lane4];
        const float* C = bc_s[b][t4 + j][1][lane4];
        float s = 0.f;
#pragma unroll
        for (int i = 0; i < NS; ++i) {
          S[i] = fmaf(fast_ex2(du.x * a2[i]), S[i], du.y * B[i]);
          s = fmaf(S[i], C[i], s);
        }
        acc[j] = s;
      }
      // four sums over four lanes, one left on each lane: lane l ends with token t4 + l
      const float x0 = (lane4 & 1) ? acc[0] : acc[1], x1 = (lane4 & 1) ? acc[2] : acc[3];
      const float g0 = __shfl_xor_sync(0xffffffffu, x0, 1), g1 = __shfl_xor_sync(0xffffffffu, x1, 1);
      const float h0 = ((lane4 & 1) ? acc[1] : acc[0]) + g0, h1 = ((lane4 & 1) ? acc[3] : acc[2]) + g1;
      const float g2 = __shfl_xor_sync(0xffffffffu, (lane4 & 2) ? h0 : h1, 2);
      const float y = ((lane4 & 2) ? h1 : h0) + g2;
      const int t = t4 + lane4;
      z_s[b][t][ch] *= fmaf(D, u_s[b][t][ch], y);
    }
    if (more) put(t0 + SC_TT, b ^ 1);
    __syncthreads();
    if (t0 + lt < p.rows) {
      T* dst = yg + (long long)(p.row0 + t0 + lt) * a.ldy + lc;
      if (vec_y) {
        float o[4];
#pragma unroll
        for (int e = 0; e < 4; ++e) o[e] = z_s[b][lt][lq + e];
        if (lc < a.inner) Vec<T, 4>::store(dst, o);
      } else {
#pragma unroll
        for (int e = 0; e < 4; ++e)
          if (lc + e < a.inner) Elem<T>::put(dst + e, z_s[b][lt][lq + e]);
      }
    }
  }
#pragma unroll
  for (int i = 0; i < NS; ++i)
    if (live && lane4 * NS + i < N) sp[i] = S[i];
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
                   on(a.conv_state) && on(a.b);
  const int v = vec && a.taps <= 4 ? 8 : 1;
  const int per = (a.inner + v - 1) / v, threads = std::min(128, (per + 31) / 32 * 32);
  const dim3 grid((per + threads - 1) / threads, a.tiles ? a.n_tiles : a.rows.n);
  if (v == 8) {
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

template <typename T, int NS>
static void launch_scan_ns(const SelectiveScanArgs& a, cudaStream_t s) {
  if (!a.rows.portions) {
    cb::selective_step_kernel<T, NS><<<dim3((a.inner + 63) / 64, a.rows.n), 256, 0, s>>>(a);
  } else if ((long long)(a.inner + 31) / 32 * a.rows.n >= 148) {
    cb::selective_scan_kernel<T, NS, 32><<<dim3((a.inner + 31) / 32, a.rows.n), 128, 0, s>>>(a);
  } else {   // few channels: more, smaller CTAs
    cb::selective_scan_kernel<T, NS, 8><<<dim3((a.inner + 7) / 8, a.rows.n), 32, 0, s>>>(a);
  }
}

template <typename T>
static void launch_scan(const SelectiveScanArgs& a, cudaStream_t s) {
  const int per = (a.state + 3) / 4;
  if (per <= 1) launch_scan_ns<T, 1>(a, s);
  else if (per <= 2) launch_scan_ns<T, 2>(a, s);
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
