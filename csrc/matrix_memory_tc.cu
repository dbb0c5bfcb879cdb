// Matrix memory (mLSTM, stack.h) over portions of prompts on tcgen05 tensor cores, in chunks of 128 tokens.
//
// With F_t the sum of a chunk's log forget gates up to t, a_s = i_s - F_s and M_t = max(m, max_{s <= t} a_s), the running maximum
// is m_t = F_t + M_t, and a chunk that starts from (S, n, m) gives
//     o_t   = sum_{s <= t} e^(a_s - M_t) (q_t . k_s) v_s + e^(m - M_t) S^T q_t           (n . q likewise, with 1 for v)
//     S_end = e^(m - M_C) S + sum_s e^(a_s - M_C) k_s v_s^T,     m_end = F_C + M_C.
// One CTA = one head's slice of 32 value columns of one sequence; it walks over the portion's chunks. Four products per chunk:
//     scores  = Q K^T                       [128 tokens x 128 tokens]
//     inter   = Q [S | n]                   [128 tokens x 80]: the state as a bf16 high and a bf16 low part, so that reading it
//                                           costs no digits that matter
//     state^T = state^T e^(m - M_C) + [w V | w]^T K   [value rows x dim], accumulated in tensor memory in fp32 for the portion
//     intra   = P [V | 1]                   [128 tokens x 48], P = scores e^(a_s - M_t) from tensor memory
// The normaliser n is one more row of the state (a column of ones beside V), with the weights split into two bf16 parts.
// Roles: 8 warps of elementwise work (state rescale and operand, V operands, P, output), one TMA warp (Q and K tiles, 128-byte
// swizzle), one MMA issuer, one warp that runs the gates' sums and maxima a chunk ahead. Every wait is bounded.
#include <algorithm>
#include <cmath>
#include <stdexcept>

#include "common.cuh"
#include "launch.cuh"
#include "stack.h"
#include "vec.cuh"

namespace cb {

constexpr int MT_C = 128, MT_VS = cosmos::MEMORY_SLICE, MT_WORK = 256, MT_THREADS = MT_WORK + 96;
constexpr int MT_TILE = MT_C * 128;                 // 128 rows x 64 columns bf16
constexpr int MT_BS_ROWS = 80;                      // 32 values high | n (3 rows, padded to 16) | 32 values low
constexpr int MT_BS_BLOCK = MT_BS_ROWS * 128;
constexpr int MT_N_COL = 32, MT_LO = 48, MT_PV_N = 48;
// tensor memory columns
constexpr uint32_t MT_T_STATE = 0, MT_T_SCORE = 256, MT_T_INTER = 384, MT_T_INTRA = 464;
static_assert(MT_VS == 32, "value rows fill one quarter of the tensor-memory lanes");

template <int DIM>
struct MtSmem {
  static constexpr int KB = DIM / 64, HALVES = DIM > 128 ? 2 : 1, HB = KB / HALVES;   // 64-column blocks; halves of K
  static constexpr int Q = 0, K = KB * MT_TILE, BS = 2 * KB * MT_TILE, VP = BS + KB * MT_BS_BLOCK, VA = VP + 2 * MT_TILE, GATES = VA + MT_TILE;
  // the elementwise warps share the state's columns: with 128 columns or more, value rows appear twice (tensor-memory lanes 0 and
  // 64), so that twice as many warps can reach them
  static constexpr int PARTS = DIM >= 128 ? 4 : 2, COLS = DIM / PARTS;
  static constexpr int GATE_BUF = (5 * MT_C + 4) * 4;   // a2, M2, c, floor, w | keep
  static constexpr int BAR = GATES + 2 * GATE_BUF;
  static constexpr int USED = BAR + 256 + 1024;
  static constexpr int BYTES = USED < 120 * 1024 ? 120 * 1024 : USED;   // one CTA per SM: each takes all of the tensor memory
};
static_assert(MtSmem<256>::VP % 1024 == 0 && MtSmem<128>::VP % 1024 == 0 && MtSmem<64>::VP % 1024 == 0 && MtSmem<64>::BAR % 16 == 0 &&
                  MtSmem<256>::BYTES <= 232448, "matrix memory shared memory");

// barriers; K comes and goes in halves of 128 columns (KF, KE), gates in two buffers
enum : int { MB_QF, MB_QE, MB_KF, MB_KE = MB_KF + 2, MB_GF = MB_KE + 2, MB_GE = MB_GF + 2, MB_XF = MB_GE + 2, MB_SF, MB_PF, MB_OF, MB_COUNT };

__device__ __forceinline__ void mt_ld16(uint32_t taddr, uint32_t (&v)[16]) {
  asm volatile(
      "tcgen05.ld.sync.aligned.32x32b.x16.b32 "
      "{%0, %1, %2, %3, %4, %5, %6, %7, %8, %9, %10, %11, %12, %13, %14, %15}, [%16];"
      : "=r"(v[0]), "=r"(v[1]), "=r"(v[2]), "=r"(v[3]), "=r"(v[4]), "=r"(v[5]), "=r"(v[6]), "=r"(v[7]), "=r"(v[8]), "=r"(v[9]),
        "=r"(v[10]), "=r"(v[11]), "=r"(v[12]), "=r"(v[13]), "=r"(v[14]), "=r"(v[15])
      : "r"(taddr)
      : "memory");
}

// Brings a tile of a tensor map into L2.
__device__ __forceinline__ void mt_prefetch(const CUtensorMap* m, int x, int y) {
  asm volatile("cp.async.bulk.prefetch.tensor.2d.L2.global.tile [%0, {%1, %2}];" ::"l"(reinterpret_cast<uint64_t>(m)), "r"(x), "r"(y)
               : "memory");
}

// 16-byte piece `chunk` of row `row` in a tile of 128-byte rows with the 128-byte swizzle.
__device__ __forceinline__ uint4* mt_piece(uint8_t* tile, int row, int chunk) {
  return reinterpret_cast<uint4*>(tile + row * 128 + ((chunk ^ (row & 7)) << 4));
}
__device__ __forceinline__ float mt_round(float x) { return __bfloat162float(__float2bfloat16(x)); }

struct MtParams {
  cosmos::RowSource gates;
  const bf16* v;
  long long ldv;
  int H, vdim;
  float cap, log2_scale, scale;
  const float* gate_bias;
  float* S;
  float* n;
  float* m;
  bf16* o;
  long long ldo;
  cosmos::StepRows rows;
  int* status;
};

template <int DIM>
__global__ void __launch_bounds__(MT_THREADS, 1)
matrix_memory_tc_kernel(const __grid_constant__ CUtensorMap tmQ, const __grid_constant__ CUtensorMap tmK, const MtParams p) {
  using L = MtSmem<DIM>;
  constexpr int KB = L::KB, HB = L::HB, HALVES = L::HALVES;
  extern __shared__ uint8_t smem_raw[];
  const uint32_t base = (smem_u32(smem_raw) + 1023u) & ~1023u;
  uint8_t* gen = smem_raw + (base - smem_u32(smem_raw));
  auto B = [&](int i) { return base + L::BAR + 8u * i; };
  volatile uint32_t* tmem_slot = reinterpret_cast<volatile uint32_t*>(gen + L::BAR + 8 * MB_COUNT);
  volatile int* abort_flag = reinterpret_cast<volatile int*>(gen + L::BAR + 8 * MB_COUNT + 8);
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const int slice = blockIdx.x, h = blockIdx.y, v0 = slice * MT_VS;
  const Portion pt = get_portion(p.rows, blockIdx.z);
  const long long slot = pt.rows > 0 ? get_state_slot(p.rows, pt.seq, p.status) : -1;
  if (slot < 0) return;   // the whole CTA, before any set-up
  const int n_chunks = (pt.rows + MT_C - 1) / MT_C;
  const bool start = pt.pos0 == 0;
  const long long sh = slot * p.H + h;
  float* Sg = p.S + sh * DIM * (long long)p.vdim + v0;
  float* ng = p.n + (sh * gridDim.x + slice) * DIM;
  float* mg = p.m + sh * gridDim.x + slice;

  if (threadIdx.x == 0) {
    for (int i = 0; i < MB_COUNT; ++i) {
      const bool work = i == MB_GE || i == MB_GE + 1 || i == MB_XF || i == MB_PF;
      mbar_init(B(i), work ? MT_WORK : 1);
    }
    *abort_flag = 0;
    fence_barrier_init();
    prefetch_tmap(&tmQ);
    prefetch_tmap(&tmK);
  }
  if (warp == 9) {
    tmem_alloc(base + L::BAR + 8 * MB_COUNT, 512);
    tmem_relinquish();
  }
  // operand tiles start as zeros: padding rows and columns stay zero for good
  for (int i = threadIdx.x; i < (L::GATES - L::BS) / 16; i += MT_THREADS) reinterpret_cast<uint4*>(gen + L::BS)[i] = make_uint4(0, 0, 0, 0);
  fence_proxy_async();
  tc_fence_before();
  __syncthreads();
  tc_fence_after();
  const uint32_t tmem = *tmem_slot;
  auto gate_buf = [&](int j) { return reinterpret_cast<float*>(gen + L::GATES + (j & 1) * L::GATE_BUF); };

  if (warp == 8) {
    // ---------------- TMA: Q and K tiles of a chunk
    if (lane == 0) {
      int issued_q = 0, issued_k[HALVES] = {};
      // a tile is waited for with nothing else to do, so it has to come from L2: the slices of a head share the blocks of the
      // chunk after the next
      auto ahead = [&](int j) {
        if (j >= n_chunks) return;
        const int x = h * DIM + (slice % KB) * 64, row = pt.row0 + j * MT_C;
        mt_prefetch(&tmK, x, row);
        mt_prefetch(&tmQ, x, row);
      };
      ahead(1);
      for (int j = 0; j < n_chunks; ++j) {
        const int row = pt.row0 + j * MT_C;
        ahead(j + 2);
        if (j > 0 && !mbar_wait(B(MB_QE), (j - 1) & 1, abort_flag, p.status, ST_TIMEOUT_TMA)) break;
        mbar_arrive_expect_tx(B(MB_QF), KB * MT_TILE);
        for (int b = 0; b < KB; ++b) tma_load_2d(base + L::Q + b * MT_TILE, &tmQ, B(MB_QF), h * DIM + b * 64, row);
        ++issued_q;
        bool ok = true;
        for (int f = 0; f < HALVES && ok; ++f) {
          if (j > 0) ok = mbar_wait(B(MB_KE + f), (j - 1) & 1, abort_flag, p.status, ST_TIMEOUT_TMA);
          if (!ok) break;
          mbar_arrive_expect_tx(B(MB_KF + f), HB * MT_TILE);
          for (int b = f * HB; b < (f + 1) * HB; ++b) tma_load_2d(base + L::K + b * MT_TILE, &tmK, B(MB_KF + f), h * DIM + b * 64, row);
          ++issued_k[f];
        }
        if (!ok) break;
      }
      // copies in flight end before the CTA does, also when a wait gave up
      volatile int no_abort = 0;
      if (issued_q > 0) mbar_wait(B(MB_QF), (issued_q - 1) & 1, &no_abort, nullptr, 0);
      for (int f = 0; f < HALVES; ++f)
        if (issued_k[f] > 0) mbar_wait(B(MB_KF + f), (issued_k[f] - 1) & 1, &no_abort, nullptr, 0);
    }
  } else if (warp == 9) {
    // ---------------- MMA issuer (unrolled: descriptor arithmetic between two products would cost more than a product)
    if (lane == 0) {
      const uint64_t q_desc = make_smem_desc_sw128(base + L::Q, 16, 1024), k_desc = make_smem_desc_sw128(base + L::K, 16, 1024);
      const uint64_t bs_desc = make_smem_desc_sw128(base + L::BS, 16, 1024);
      const uint64_t kt_desc = make_smem_desc_sw128(base + L::K, MT_TILE, 1024);
      const uint64_t vp_desc = make_smem_desc_sw128(base + L::VP, MT_TILE, 1024);   // value rows 0..63, and again
      const uint64_t va_desc = make_smem_desc_sw128(base + L::VA, MT_TILE, 1024);
      constexpr uint32_t id_s = make_idesc_bf16(128, 128, 0, 0), id_i = make_idesc_bf16(128, MT_BS_ROWS, 0, 0),
                         id_u = make_idesc_bf16(128, HB * 64, 1, 1), id_p = make_idesc_bf16(128, MT_PV_N, 0, 1);
      auto wait = [&](int b, int phase) { return mbar_wait(B(b), phase & 1, abort_flag, p.status, ST_TIMEOUT_MMA); };
      for (int j = 0; j < n_chunks; ++j) {
        // the inter-chunk product first: it needs no K, whose tile is still on its way
        bool ok = wait(MB_QF, j) && wait(MB_XF, j);
        if (!ok) break;
        tc_fence_after();
#pragma unroll
        for (int kk = 0; kk < DIM / 16; ++kk)
          mma_ss(tmem + MT_T_INTER, q_desc + (uint64_t)((kk >> 2) * (MT_TILE >> 4) + 2 * (kk & 3)),
                 bs_desc + (uint64_t)((kk >> 2) * (MT_BS_BLOCK >> 4) + 2 * (kk & 3)), id_i, kk > 0);
#pragma unroll
        for (int f = 0; f < HALVES; ++f) {
          ok = ok && wait(MB_KF + f, j);
          if (!ok) break;
          tc_fence_after();
#pragma unroll
          for (int kk = f * HB * 4; kk < (f + 1) * HB * 4; ++kk) {
            const uint64_t off = (uint64_t)((kk >> 2) * (MT_TILE >> 4) + 2 * (kk & 3));
            mma_ss(tmem + MT_T_SCORE, q_desc + off, k_desc + off, id_s, kk > 0);
          }
        }
        if (!ok) break;
        tc_commit(B(MB_SF));
        tc_commit(B(MB_QE));
#pragma unroll
        for (int f = 0; f < HALVES; ++f) {
#pragma unroll
          for (int kk = 0; kk < MT_C / 16; ++kk)
            mma_ss(tmem + MT_T_STATE + f * HB * 64, vp_desc + (uint64_t)(kk * (2048 >> 4)),
                   kt_desc + (uint64_t)(f * HB * (MT_TILE >> 4) + kk * (2048 >> 4)), id_u, 1u);
          tc_commit(B(MB_KE + f));
        }
        if (!wait(MB_PF, j)) break;
        tc_fence_after();
#pragma unroll
        for (int kk = 0; kk < MT_C / 16; ++kk)
          mma_ts(tmem + MT_T_INTRA, tmem + MT_T_SCORE + (kk >> 2) * 64 + (kk & 3) * 8, va_desc + (uint64_t)(kk * (2048 >> 4)), id_p, kk > 0);
        tc_commit(B(MB_OF));
      }
    }
  } else if (warp == 10) {
    // ---------------- gates: sums and maxima of a chunk, a chunk ahead; four tokens a lane
    const float bi = p.gate_bias[h], bf = p.gate_bias[p.H + h];
    float m_prev = start ? 0.f : *mg;
    bool ok = true;
    float ni[4], nf[4];   // the next chunk's rows, on their way
    const float* gp = reinterpret_cast<const float*>(p.gates.p) + h;
    auto fetch = [&](int j) {
      const int left = pt.rows - j * MT_C;
      if (left <= 0) return;
      const float* r[4];
#pragma unroll
      for (int e = 0; e < 4; ++e) {
        r[e] = gp + (pt.row0 + j * MT_C + min(lane * 4 + e, left - 1)) * p.gates.ld;
        ni[e] = r[e][0];
        nf[e] = r[e][p.H];
      }
      for (int k = 1; k < p.gates.k_splits; ++k) {
        float x[8];
#pragma unroll
        for (int e = 0; e < 4; ++e) {
          x[e] = r[e][k * p.gates.split_stride];
          x[4 + e] = r[e][k * p.gates.split_stride + p.H];
        }
#pragma unroll
        for (int e = 0; e < 4; ++e) {
          ni[e] += x[e];
          nf[e] += x[4 + e];
        }
      }
    };
    fetch(0);
    for (int j = 0; j < n_chunks; ++j) {
      const int cnt = min(MT_C, pt.rows - j * MT_C);
      float gi[4], gf[4];
#pragma unroll
      for (int e = 0; e < 4; ++e) {
        gi[e] = ni[e];
        gf[e] = nf[e];
      }
      fetch(j + 1);
      float F[4], a[4], sum = 0.f;
#pragma unroll
      for (int e = 0; e < 4; ++e) {
        const bool in = lane * 4 + e < cnt;
        const float x = p.cap * tanhf((gf[e] + bf) / p.cap);
        sum += in ? fminf(x, 0.f) - log1pf(expf(-fabsf(x))) : 0.f;
        F[e] = sum;
        a[e] = in ? p.cap * tanhf((gi[e] + bi) / p.cap) : -INFINITY;
      }
      float inc = sum;
#pragma unroll
      for (int o = 1; o < 32; o <<= 1) {
        const float t = __shfl_up_sync(0xffffffffu, inc, o);
        if (lane >= o) inc += t;
      }
      const float before = inc - sum, total = __shfl_sync(0xffffffffu, inc, 31);
      float mx = -INFINITY, M[4];
#pragma unroll
      for (int e = 0; e < 4; ++e) {
        F[e] += before;
        a[e] -= F[e];
        mx = fmaxf(mx, a[e]);
        M[e] = mx;
      }
      float run = mx;
#pragma unroll
      for (int o = 1; o < 32; o <<= 1) {
        const float t = __shfl_up_sync(0xffffffffu, run, o);
        if (lane >= o) run = fmaxf(run, t);
      }
      float prior = __shfl_up_sync(0xffffffffu, run, 1);
      prior = lane == 0 ? m_prev : fmaxf(prior, m_prev);
      const float M_end = fmaxf(m_prev, __shfl_sync(0xffffffffu, run, 31));
      int good = 1;
      if (j > 1 && lane == 0) good = mbar_wait(B(MB_GE + (j & 1)), ((j >> 1) - 1) & 1, abort_flag, p.status, ST_TIMEOUT_EPI) ? 1 : 0;
      ok = __shfl_sync(0xffffffffu, good, 0) != 0;
      if (!ok) break;
      float* g = gate_buf(j);
      constexpr float LOG2E = 1.4426950408889634f;
#pragma unroll
      for (int e = 0; e < 4; ++e) {
        const int t = lane * 4 + e;
        M[e] = fmaxf(M[e], prior);
        g[t] = a[e] * LOG2E;
        g[MT_C + t] = M[e] * LOG2E - p.log2_scale;               // the query scale rides along
        g[2 * MT_C + t] = expf(m_prev - M[e]) * p.scale;
        g[3 * MT_C + t] = expf(-(F[e] + M[e]));
        g[4 * MT_C + t] = expf(a[e] - M_end);
      }
      if (lane == 0) g[5 * MT_C] = expf(m_prev - M_end);
      m_prev = total + M_end;
      __syncwarp();
      if (lane == 0) mbar_arrive(B(MB_GF + (j & 1)));
    }
    if (ok && lane == 0) *mg = m_prev;
  } else {
    // ---------------- elementwise work: token row t = TMEM lane; warps w and w + 4 share rows and split columns
    const int wg = warp >> 2, quad = warp & 3, t = quad * 32 + lane;
    const uint32_t lane_addr = tmem + (uint32_t(quad * 32) << 16);
    const int vt = threadIdx.x >> 1, vh = threadIdx.x & 1;       // V operands: token, half of the columns
    const bf16* vsrc = p.v + (long long)pt.row0 * p.ldv + (long long)h * p.vdim + v0 + vh * 16;
    uint4 vr[2];
    auto fetch_v = [&](int j) {
      const int r = j * MT_C + vt;
      vr[0] = vr[1] = make_uint4(0, 0, 0, 0);
      if (r < pt.rows) {
        const uint4* s = reinterpret_cast<const uint4*>(vsrc + (long long)r * p.ldv);
        vr[0] = s[0];
        vr[1] = s[1];
      }
    };
    auto wait = [&](int b, int phase) {   // for the whole warp: all lanes go on, or none
      const bool r = mbar_wait(B(b), phase & 1, abort_flag, p.status, ST_TIMEOUT_SOFTMAX);
      return __all_sync(0xffffffffu, r) != 0;
    };
    // The state as operand, then rescaled in place, for chunk j: value rows on even quarters of the lanes, n on lanes 0 and 1 of
    // odd ones; this warp's columns only.
    const bool even = (quad & 1) == 0, holds = L::PARTS == 4 || quad < 2;
    const int col0 = (L::PARTS == 4 ? wg * 2 + (quad >> 1) : wg) * L::COLS;
    auto convert = [&](int j) {
      if (holds) {
        const float keep = gate_buf(j)[5 * MT_C];
#pragma unroll 1
        for (int c0 = col0; c0 < col0 + L::COLS; c0 += 32) {
          uint32_t s[32];
          if (j == 0) {
#pragma unroll
            for (int i = 0; i < 32; ++i) {
              float x = 0.f;
              if (!start && even) x = Sg[(long long)(c0 + i) * p.vdim + lane];
              if (!start && !even && lane == 0) x = ng[c0 + i];
              s[i] = __float_as_uint(x);
            }
          } else {
            tmem_ld32(lane_addr + MT_T_STATE + c0, s);
            tmem_wait_ld();
          }
          uint8_t* block = gen + L::BS + (c0 >> 6) * MT_BS_BLOCK;
          const int row_hi = even ? lane : MT_N_COL + 2 * lane;       // n: rows 32 (high), 33 (low), 34 (the low weights' sum)
          const int row_lo = even ? MT_LO + lane : MT_N_COL + 1;
#pragma unroll
          for (int q = 0; q < 4; ++q) {
            uint32_t hi[4], lo[4];
#pragma unroll
            for (int e = 0; e < 4; ++e) {
              const float x = __uint_as_float(s[8 * q + 2 * e]), y = __uint_as_float(s[8 * q + 2 * e + 1]);
              hi[e] = pack_bf16(x, y);
              lo[e] = pack_bf16(x - bf16lo(hi[e]), y - bf16hi(hi[e]));
            }
            const int chunk = ((c0 & 63) >> 3) + q;
            if (even || lane < 2) *mt_piece(block, row_hi, chunk) = make_uint4(hi[0], hi[1], hi[2], hi[3]);
            if (even || lane == 0) *mt_piece(block, row_lo, chunk) = make_uint4(lo[0], lo[1], lo[2], lo[3]);
          }
#pragma unroll
          for (int i = 0; i < 32; ++i) s[i] = __float_as_uint(__uint_as_float(s[i]) * keep);
          __syncwarp();
          tmem_st32(lane_addr + MT_T_STATE + c0, s);
        }
        tmem_wait_st();
      }
    };
    // V operands of chunk j, [V | 1] and [w V | w], then everything that the chunk's products read is in place.
    auto operands = [&](int j) {
      const float w = gate_buf(j)[4 * MT_C + vt];
      uint8_t *va = gen + L::VA, *vp = gen + L::VP, *vp2 = vp + MT_TILE;
#pragma unroll
      for (int q = 0; q < 2; ++q) {
        *mt_piece(va, vt, vh * 2 + q) = vr[q];
        const uint32_t in[4] = {vr[q].x, vr[q].y, vr[q].z, vr[q].w};
        uint32_t o[4];
#pragma unroll
        for (int e = 0; e < 4; ++e) o[e] = pack_bf16(w * bf16lo(in[e]), w * bf16hi(in[e]));
        *mt_piece(vp, vt, vh * 2 + q) = make_uint4(o[0], o[1], o[2], o[3]);
        if (L::PARTS == 4) *mt_piece(vp2, vt, vh * 2 + q) = make_uint4(o[0], o[1], o[2], o[3]);
      }
      if (vh == 0) {
        *mt_piece(va, vt, 4) = make_uint4(pack_bf16(j * MT_C + vt < pt.rows ? 1.f : 0.f, 0.f), 0u, 0u, 0u);
        const float hi = mt_round(w);
        *mt_piece(vp, vt, 4) = make_uint4(pack_bf16(hi, w - hi), 0u, 0u, 0u);
        if (L::PARTS == 4) *mt_piece(vp2, vt, 4) = make_uint4(pack_bf16(hi, w - hi), 0u, 0u, 0u);
      }
      fence_proxy_async();
      tc_fence_before();
      mbar_arrive(B(MB_XF));
      if (j + 1 < n_chunks) fetch_v(j + 1);
    };
    fetch_v(0);
    bool ok = wait(MB_GF, 0);
    if (ok) {
      convert(0);
      operands(0);
    }
    for (int j = 0; j < n_chunks && ok; ++j) {
      const int cnt = min(MT_C, pt.rows - j * MT_C);
      const bool more = j + 1 < n_chunks;
      const float* g = gate_buf(j);
      // ---- P = scores e^(a_s - M_t), causal; this half's 64 columns in two blocks of 32
      const float M2 = g[MT_C + t], c_t = g[2 * MT_C + t], floor_t = g[3 * MT_C + t];
      ok = wait(MB_SF, j);
      if (!ok) break;
      tc_fence_after();
      uint32_t pk[32];
#pragma unroll
      for (int b = 0; b < 2; ++b) {
        const int blk = wg * 2 + b;
        if (blk > quad) {         // above the diagonal
#pragma unroll
          for (int i = 0; i < 16; ++i) pk[b * 16 + i] = 0u;
          continue;
        }
        uint32_t s[32];
        tmem_ld32(lane_addr + MT_T_SCORE + blk * 32, s);
        tmem_wait_ld();
        const float4* ga = reinterpret_cast<const float4*>(g + blk * 32);
        const int last = blk == quad ? lane : 31;
#pragma unroll
        for (int i = 0; i < 8; ++i) {
          const float4 a = ga[i];
          const float x0 = 4 * i <= last ? __uint_as_float(s[4 * i]) * fast_ex2(a.x - M2) : 0.f;
          const float x1 = 4 * i + 1 <= last ? __uint_as_float(s[4 * i + 1]) * fast_ex2(a.y - M2) : 0.f;
          const float x2 = 4 * i + 2 <= last ? __uint_as_float(s[4 * i + 2]) * fast_ex2(a.z - M2) : 0.f;
          const float x3 = 4 * i + 3 <= last ? __uint_as_float(s[4 * i + 3]) * fast_ex2(a.w - M2) : 0.f;
          pk[b * 16 + 2 * i] = pack_bf16(x0, x1);
          pk[b * 16 + 2 * i + 1] = pack_bf16(x2, x3);
        }
      }
      __syncwarp();
      tmem_st32(lane_addr + MT_T_SCORE + wg * 64, pk);
      tmem_wait_st();
      tc_fence_before();
      mbar_arrive(B(MB_PF));
      mbar_arrive(B(MB_GE + (j & 1)));
      // ---- the state after this chunk as the next one's operand, beside the last product
      if (more) {
        ok = wait(MB_GF + ((j + 1) & 1), (j + 1) >> 1) && wait(MB_KE + HALVES - 1, j);
        if (!ok) break;
        tc_fence_after();
        convert(j + 1);
      }
      // ---- output: this half's 16 value columns
      ok = wait(MB_OF, j);
      if (!ok) break;
      tc_fence_after();
      uint32_t hi[16], lo[16], in[16], nn[16], ni[16];
      mt_ld16(lane_addr + MT_T_INTER + wg * 16, hi);
      mt_ld16(lane_addr + MT_T_INTER + MT_LO + wg * 16, lo);
      mt_ld16(lane_addr + MT_T_INTER + MT_N_COL, nn);
      mt_ld16(lane_addr + MT_T_INTRA + wg * 16, in);
      mt_ld16(lane_addr + MT_T_INTRA + MT_N_COL, ni);
      tmem_wait_ld();
      if (more) operands(j + 1);
      auto f = [](uint32_t u) { return __uint_as_float(u); };
      const float nq = fmaf(c_t, f(nn[0]) + (f(nn[1]) + f(nn[2])), f(ni[0]));
      const float inv = 1.f / (fmaxf(fabsf(nq), floor_t) + 1e-6f);
      if (t < cnt) {
        uint32_t o[8];
#pragma unroll
        for (int i = 0; i < 8; ++i)
          o[i] = pack_bf16(fmaf(c_t, f(hi[2 * i]) + f(lo[2 * i]), f(in[2 * i])) * inv,
                           fmaf(c_t, f(hi[2 * i + 1]) + f(lo[2 * i + 1]), f(in[2 * i + 1])) * inv);
        uint4* dst = reinterpret_cast<uint4*>(p.o + (long long)(pt.row0 + j * MT_C + t) * p.ldo + (long long)h * p.vdim + v0 + wg * 16);
        dst[0] = make_uint4(o[0], o[1], o[2], o[3]);
        dst[1] = make_uint4(o[4], o[5], o[6], o[7]);
      }
      __syncwarp();
    }
    // ---- the state back to memory
    if (ok && holds) {
#pragma unroll 1
      for (int c0 = col0; c0 < col0 + L::COLS; c0 += 32) {
        uint32_t s[32];
        tmem_ld32(lane_addr + MT_T_STATE + c0, s);
        tmem_wait_ld();
#pragma unroll
        for (int i = 0; i < 32; ++i) {
          const float x = __uint_as_float(s[i]), other = __shfl_down_sync(0xffffffffu, x, 1);
          if (even) Sg[(long long)(c0 + i) * p.vdim + lane] = x;
          if (!even && lane == 0) ng[c0 + i] = x + other;
        }
        __syncwarp();
      }
    }
  }
  __syncwarp();
  tc_fence_before();
  __syncthreads();
  if (warp == 9) {
    __syncwarp();
    tc_fence_after();
    tmem_dealloc(tmem, 512);
  }
}

}  // namespace cb

namespace cosmos {

bool matrix_memory_tc_supported(const MatrixMemoryArgs& a) {
  auto on = [](const RowSource& s) { return s.k_splits == 0 && (reinterpret_cast<uintptr_t>(s.p) & 15) == 0 && s.ld % 8 == 0; };
  return !a.is_f32 && a.rows.portions && (a.dim == 64 || a.dim == 128 || a.dim == 256) && a.vdim % MEMORY_SLICE == 0 && on(a.q) && on(a.k) &&
         on(a.v) && a.ldo % 8 == 0 && (reinterpret_cast<uintptr_t>(a.o) & 15) == 0;
}

template <int DIM>
static void launch_tc(const MatrixMemoryArgs& a, cudaStream_t s) {
  constexpr int smem = cb::MtSmem<DIM>::BYTES;
  static bool configured = false;
  if (!configured) {
    if (cudaFuncSetAttribute(cb::matrix_memory_tc_kernel<DIM>, cudaFuncAttributeMaxDynamicSharedMemorySize, smem) != cudaSuccess)
      throw std::runtime_error("matrix_memory: shared memory not available");
    configured = true;
  }
  const uint64_t dims[2] = {(uint64_t)a.H * DIM, (uint64_t)a.n_rows};
  const uint32_t box[2] = {64, cb::MT_C};
  const uint64_t sq[1] = {(uint64_t)a.q.ld * 2}, sk[1] = {(uint64_t)a.k.ld * 2};
  const CUtensorMap tq = cbh::make_tmap_bf16(a.q.p, 2, dims, sq, box, true), tk = cbh::make_tmap_bf16(a.k.p, 2, dims, sk, box, true);
  cb::MtParams p{};
  p.gates = a.gates;
  p.v = reinterpret_cast<const bf16*>(a.v.p); p.ldv = a.v.ld;
  p.H = a.H; p.vdim = a.vdim; p.cap = a.cap; p.scale = a.q_scale; p.log2_scale = std::log2(a.q_scale);
  p.gate_bias = a.gate_bias; p.S = a.S; p.n = a.n; p.m = a.m;
  p.o = reinterpret_cast<bf16*>(a.o); p.ldo = a.ldo;
  p.rows = a.rows; p.status = a.status;
  cb::matrix_memory_tc_kernel<DIM><<<dim3(a.vdim / MEMORY_SLICE, a.H, a.rows.n), cb::MT_THREADS, smem, s>>>(tq, tk, p);
}

void matrix_memory_tc(const MatrixMemoryArgs& a, cudaStream_t s) {
  switch (a.dim) {
    case 64: launch_tc<64>(a, s); break;
    case 128: launch_tc<128>(a, s); break;
    default: launch_tc<256>(a, s); break;
  }
}

}  // namespace cosmos
