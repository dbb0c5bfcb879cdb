// Windowed attention with a distance bias for portions of prompts (stack.h, WindowAttnArgs) on tcgen05 tensor cores.
//
// The structure is that of attn_tcgen05.cu (one CTA = 256 query rows of one head as two 128-row tiles, S = Q K^T and
// O += P V with accumulators in tensor memory, one query row per softmax thread, lazy rescale). What differs:
//   * K and V come straight from the paged cache: one TMA box (page_size rows x 64 columns) per page, tensor and half, so
//     a portion sees the tokens of earlier portions and its own through one path, and nothing is gathered beforehand.
//   * Query tiles are listed by the host (sequence, first row, rows, position), so one launch serves portions of several
//     sequences. Only the key blocks inside [first row's window, last row] are visited, and each 128-row tile skips those
//     of them that lie outside its own rows' range.
//   * Mask and bias are one table. Within a 128 x 128 block the distance i - j takes 255 values, so the softmax warps of a
//     tile compute bias[i - j] once per block (at most two logarithms per thread), with -inf outside the window and above the
//     diagonal, and add it with the FMA that scales the scores. A row's entries are consecutive; four copies of the table,
//     each shifted by one entry, let every thread read four at a time with aligned 16-byte loads. The copies start 8 words
//     apart modulo the 32 banks, so the eight lanes of a 16-byte load phase hit different banks. Half of a row's entries
//     are read before the scores are waited for (the table needs no score), which takes those loads off the chain
//     scores -> softmax -> next product that bounds the kernel.
//   * Head sizes up to 128 that are multiples of 8: the copies zero-fill the columns beyond the head size, products run
//     over the 16-column steps that hold data.
#include "common.cuh"
#include "launch.cuh"
#include "stack.h"

namespace cb {

constexpr int WA_THREADS = 384;
constexpr int WA_TILE_BYTES = 128 * 128 * 2;
constexpr int WA_HALF = WA_TILE_BYTES / 2;
constexpr int WA_NSLOT = 4;
constexpr int WA_TAB = 264;                    // words per table copy: 256 entries + pad, = 8 modulo 32
constexpr int WA_TAB_BYTES = 4 * WA_TAB * 4;   // four shifted copies
constexpr int WA_OFF_TAB = (2 + WA_NSLOT) * WA_TILE_BYTES;
constexpr int WA_OFF_BAR = WA_OFF_TAB + 4 * WA_TAB_BYTES;   // [tile][parity]
constexpr int WA_SMEM = WA_OFF_BAR + 256 + 1024;
static_assert(WA_TAB % 32 == 8 && WA_TAB_BYTES % 16 == 0 && WA_SMEM <= 232448, "window attention shared memory");

struct WinAttnParams {
  const int4* tiles;
  const int* table;
  int max_pages, num_pages, page_size;
  int group, kdim, vdim, window;
  float scale_log2;
  const float* r1;
  const float* r2;
  bf16* out;
  long long ldo;
  int* status;
};

__device__ __forceinline__ float wa_ex2(float x) {
  float y;
  asm("ex2.approx.ftz.f32 %0, %1;" : "=f"(y) : "f"(x));
  return y;
}
__device__ __forceinline__ float wa_max3(float a, float b, float c) {
  float d;
  asm("max.f32 %0, %1, %2, %3;" : "=f"(d) : "f"(a), "f"(b), "f"(c));
  return d;
}
__device__ __forceinline__ uint64_t wa_pack(float lo, float hi) {
  uint64_t r;
  asm("mov.b64 %0, {%1, %2};" : "=l"(r) : "f"(lo), "f"(hi));
  return r;
}
__device__ __forceinline__ void wa_unpack(uint64_t v, float& lo, float& hi) {
  asm("mov.b64 {%0, %1}, %2;" : "=f"(lo), "=f"(hi) : "l"(v));
}
__device__ __forceinline__ uint64_t wa_fma2(uint64_t a, uint64_t b, uint64_t c) {
  uint64_t r;
  asm("fma.rn.f32x2 %0, %1, %2, %3;" : "=l"(r) : "l"(a), "l"(b), "l"(c));
  return r;
}
__device__ __forceinline__ uint64_t wa_add2(uint64_t a, uint64_t b) {
  uint64_t r;
  asm("add.rn.f32x2 %0, %1, %2;" : "=l"(r) : "l"(a), "l"(b));
  return r;
}

__global__ void __launch_bounds__(WA_THREADS, 1)
window_attn_prefill_kernel(const __grid_constant__ CUtensorMap tmQ, const __grid_constant__ CUtensorMap tmK,
                           const __grid_constant__ CUtensorMap tmV, const WinAttnParams p) {
  extern __shared__ uint8_t smem_raw[];
  const uint32_t base = (smem_u32(smem_raw) + 1023u) & ~1023u;
  uint8_t* gen = smem_raw + (base - smem_u32(smem_raw));
  const uint32_t q_smem = base, kv_smem = base + 2 * WA_TILE_BYTES, bar = base + WA_OFF_BAR;
  const uint32_t q_full = bar;
  auto kv_full = [&](int s) { return bar + 8u * (1 + s); };
  auto kv_empty = [&](int s) { return bar + 8u * (1 + WA_NSLOT + s); };
  auto s_full = [&](int t) { return bar + 8u * (1 + 2 * WA_NSLOT + t); };
  auto p_full = [&](int t, int h) { return bar + 8u * (3 + 2 * WA_NSLOT + 2 * t + h); };
  auto o_final = [&](int t) { return bar + 8u * (7 + 2 * WA_NSLOT + t); };
  constexpr int NBAR = 9 + 2 * WA_NSLOT;
  const uint32_t tmem_slot = bar + 8u * NBAR;
  volatile uint32_t* tmem_slot_ptr = reinterpret_cast<volatile uint32_t*>(gen + WA_OFF_BAR + 8 * NBAR);
  volatile int* abort_flag = reinterpret_cast<volatile int*>(gen + WA_OFF_BAR + 8 * NBAR + 8);

  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const int4 tile = p.tiles[blockIdx.x];
  const int seq = tile.x, row0 = tile.y, n_rows = tile.z, pos0 = tile.w;
  const int head = blockIdx.y, kvh = head / p.group;
  // key blocks: from the page that holds the first row's oldest key to the last row
  const int kv0 = max(0, pos0 - p.window + 1) / p.page_size * p.page_size;
  const int kv_end = pos0 + n_rows;
  const int n_blocks = (kv_end - kv0 + 127) / 128;
  // blocks [jl, jh) of each tile: from its first row's oldest key to its last row (none for a tile without rows)
  int jl[2], jh[2];
#pragma unroll
  for (int t = 0; t < 2; ++t) {
    const int first = pos0 + t * 128, last = min(first + 127, kv_end - 1);
    jl[t] = (max(0, first - p.window + 1) - kv0) >> 7;
    jh[t] = last >= first ? ((last - kv0) >> 7) + 1 : jl[t];
  }
  const int k_halves = p.kdim > 64 ? 2 : 1, v_halves = p.vdim > 64 ? 2 : 1;

  if (threadIdx.x == 0) {
    mbar_init(q_full, 1);
    for (int s = 0; s < WA_NSLOT; ++s) {
      mbar_init(kv_full(s), 1);
      mbar_init(kv_empty(s), 1);
    }
    for (int t = 0; t < 2; ++t) {
      mbar_init(s_full(t), 1);
      mbar_init(p_full(t, 0), 128);
      mbar_init(p_full(t, 1), 128);
      mbar_init(o_final(t), 1);
    }
    *abort_flag = 0;
    fence_barrier_init();
    prefetch_tmap(&tmQ);
    prefetch_tmap(&tmK);
    prefetch_tmap(&tmV);
  }
  if (warp == 1) {
    tmem_alloc(tmem_slot, 512);
    tmem_relinquish();
  }
  tc_fence_before();
  __syncthreads();
  tc_fence_after();
  const uint32_t tmem_base = *tmem_slot_ptr;   // S0 | S1 | O0 | O1, 128 columns each

  static_assert(128 * 56 + 256 * 224 <= WA_THREADS * 168, "setmaxnreg split exceeds the CTA's registers");
  if (warp < 4) {
    asm volatile("setmaxnreg.dec.sync.aligned.u32 56;");
    if (warp == 0) {
      // ---------------- TMA producer warp: lane 0 waits and arms, the lanes share a block's page copies
      if (lane == 0) {
        mbar_arrive_expect_tx(q_full, 2 * k_halves * WA_HALF);
        for (int t = 0; t < 2; ++t)
          for (int h = 0; h < k_halves; ++h)
            tma_load_3d(q_smem + t * WA_TILE_BYTES + h * WA_HALF, &tmQ, q_full, h * 64, head, row0 + t * 128);
      }
      const int pages = 128 / p.page_size;
      int issued = 0;
      bool ok = true;
      for (int i = 0; i < 2 * n_blocks; ++i) {
        const int s = i % WA_NSLOT;
        int good = 1;
        if (lane == 0) good = mbar_wait(kv_empty(s), ((i / WA_NSLOT) & 1) ^ 1, abort_flag, p.status, ST_TIMEOUT_TMA) ? 1 : 0;
        good = __shfl_sync(0xffffffffu, good, 0);
        if (!good) {
          ok = false;
          break;
        }
        const bool is_v = i & 1;
        const int halves = is_v ? v_halves : k_halves;
        if (lane == 0) mbar_arrive_expect_tx(kv_full(s), halves * WA_HALF);
        __syncwarp();
        for (int op = lane; op < pages * halves; op += 32) {
          const int pg = op / halves, h = op - pg * halves;
          const int tok = kv0 + (i >> 1) * 128 + pg * p.page_size;
          int page = p.num_pages;   // beyond the last key: an out-of-range page is zero-filled
          if (tok < kv_end) {
            page = p.table[(long long)seq * p.max_pages + tok / p.page_size];
            if (!index_ok(page, p.num_pages, p.status, SITE_STACK_PAGE)) page = p.num_pages;
          }
          tma_load_4d(kv_smem + s * WA_TILE_BYTES + h * WA_HALF + uint32_t(pg * p.page_size) * 128u, is_v ? &tmV : &tmK,
                      kv_full(s), h * 64, 0, kvh, page);
        }
        issued = i + 1;
      }
      if (!ok && lane == 0) {
        volatile int no_abort = 0;
        mbar_wait(q_full, 0, &no_abort, nullptr, 0);
        const int first = issued > WA_NSLOT ? issued - WA_NSLOT : 0;
        for (int i = first; i < issued; ++i)
          mbar_wait(kv_full(i % WA_NSLOT), (i / WA_NSLOT) & 1, &no_abort, nullptr, 0);
      }
    } else if (warp == 1) {
      // ---------------- MMA issuer: the warp walks the schedule, one elected lane issues
      const bool issuer = elect_one();
      auto wait_all = [&](uint32_t b, uint32_t phase) {
        return __all_sync(0xffffffffu, mbar_wait(b, phase, abort_flag, p.status, ST_TIMEOUT_MMA)) != 0;
      };
      constexpr uint32_t idesc_qk = make_idesc_bf16(128, 128, 0, 0);
      const uint32_t idesc_pv = make_idesc_bf16(128, (p.vdim + 15) / 16 * 16, 0, 1);
      const int k_steps = (p.kdim + 15) / 16;
      const uint64_t q_desc0 = make_smem_desc_sw128(q_smem, 16, 1024);
      const uint64_t k_desc0 = make_smem_desc_sw128(kv_smem, 16, 1024);
      const uint64_t v_desc0 = make_smem_desc_sw128(kv_smem, WA_HALF, 1024);
      auto issue_qk = [&](int t, int slot) {
        if (!issuer) return;
        const uint64_t a0 = q_desc0 + uint64_t(t * (WA_TILE_BYTES >> 4));
        const uint64_t b0 = k_desc0 + uint64_t(slot * (WA_TILE_BYTES >> 4));
        for (int kk = 0; kk < k_steps; ++kk) {
          const uint32_t off = (kk >> 2) * (WA_HALF >> 4) + 2 * (kk & 3);
          mma_ss(tmem_base + t * 128, a0 + off, b0 + off, idesc_qk, kk > 0 ? 1u : 0u);
        }
      };
      auto commit = [&](uint32_t b) {
        if (issuer) tc_commit(b);
      };
      auto issue_pv = [&](int t, int slot, bool acc, int half) {
        if (!issuer) return;
        const uint64_t b0 = v_desc0 + uint64_t(slot * (WA_TILE_BYTES >> 4));
#pragma unroll
        for (int k4 = 0; k4 < 4; ++k4) {
          const int kk = half * 4 + k4;
          mma_ts(tmem_base + 256 + t * 128, tmem_base + t * 128 + kk * 8, b0 + uint64_t(kk * (2048 >> 4)), idesc_pv,
                 (acc || kk > 0) ? 1u : 0u);
        }
      };
      bool ok = wait_all(q_full, 0);
      if (ok) ok = wait_all(kv_full(0), 0);
      if (ok) {
        tc_fence_after();
#pragma unroll
        for (int t = 0; t < 2; ++t)
          if (jl[t] == 0 && jh[t] > 0) {
            issue_qk(t, 0);
            commit(s_full(t));
          }
        commit(kv_empty(0));
        __syncwarp();
      }
      for (int j = 0; j < n_blocks && ok; ++j) {
        const int iv = 2 * j + 1, ik = 2 * j + 2;
        const int sv = iv % WA_NSLOT, sk = ik % WA_NSLOT;
        const bool more = j + 1 < n_blocks;
        ok = wait_all(kv_full(sv), (iv / WA_NSLOT) & 1);
        if (ok && more) ok = wait_all(kv_full(sk), (ik / WA_NSLOT) & 1);
        if (!ok) break;
#pragma unroll 1
        for (int t = 0; t < 2; ++t) {
          const int lo = t ? jl[1] : jl[0], hi = t ? jh[1] : jh[0];
          if (j >= lo && j < hi) {
            ok = wait_all(p_full(t, 0), (j - lo) & 1);
            if (!ok) break;
            tc_fence_after();
            issue_pv(t, sv, j > lo, 0);
            ok = wait_all(p_full(t, 1), (j - lo) & 1);
            if (!ok) break;
            tc_fence_after();
            issue_pv(t, sv, j > lo, 1);
            if (j + 1 == hi) commit(o_final(t));
          }
          if (j + 1 >= lo && j + 1 < hi) {
            issue_qk(t, sk);
            commit(s_full(t));
          }
          __syncwarp();
        }
        if (!ok) break;
        commit(kv_empty(sv));
        if (more) commit(kv_empty(sk));
        __syncwarp();
      }
    }
  } else {
    asm volatile("setmaxnreg.inc.sync.aligned.u32 224;");
    // ---------------- softmax + epilogue, one query row per thread
    const int t = (warp - 4) >> 2;
    const int quad = warp & 3;
    const int row = quad * 32 + lane;
    const uint32_t lane_addr = tmem_base + (uint32_t(quad * 32) << 16);
    const uint32_t s_addr = lane_addr + t * 128;
    const uint32_t o_addr = lane_addr + 256 + t * 128;
    const float sl2 = p.scale_log2;
    const bool linear = p.r2 == nullptr;   // scores are in base 2
    const float r1 = p.r1 ? p.r1[head] * (linear ? 1.4426950408889634f : 1.f) : 0.f, r2 = linear ? 0.f : p.r2[head];
    // table entry u = column - row + 127 stands for the distance d0 - (u - 127), d0 = distance of (row 0, column 0)
    const int shift = (127 - row) & 3;
    float* tab_t = reinterpret_cast<float*>(gen + WA_OFF_TAB + t * 2 * WA_TAB_BYTES);
    float m_used = -1e30f, l = 0.f;
    bool ok = true;
    const int lo = t ? jl[1] : jl[0], hi = t ? jh[1] : jh[0];
    for (int j = lo; j < hi; ++j) {
      float* tab = tab_t + (j & 1) * (4 * WA_TAB);
      const int d0 = pos0 + t * 128 - (kv0 + j * 128);
#pragma unroll
      for (int e = 0; e < 2; ++e) {
        const int u = row + 128 * e;
        const int dist = d0 - (u - 127);
        const float b = (dist >= 0 && dist < p.window) ? -r1 * (linear ? (float)dist : __log2f(fmaf(r2, (float)dist, 1.f))) : -INFINITY;
#pragma unroll
        for (int c = 0; c < 4; ++c)
          if (u >= c) tab[c * WA_TAB + u - c] = b;   // copy c: entry i holds table entry i + c
      }
      // the table of block j is complete; the buffer it overwrites at j + 2 has been read by every thread by then. A
      // thread that has given up on a wait keeps meeting the others here, so that nobody is left behind.
      asm volatile("bar.sync %0, 128;" ::"r"(1 + t) : "memory");
      const float4* brow = reinterpret_cast<const float4*>(tab + shift * WA_TAB + (127 - row - shift));
      float4 bias[16];
#pragma unroll
      for (int c = 0; c < 16; ++c) bias[c] = brow[c];
      if (!ok || !mbar_wait(s_full(t), (j - lo) & 1, abort_flag, p.status, ST_TIMEOUT_SOFTMAX)) {
        ok = false;
        continue;
      }
      tc_fence_after();
      uint32_t s[128];
      tmem_ld32(s_addr, *reinterpret_cast<uint32_t(*)[32]>(&s[0]));
      tmem_ld32(s_addr + 32, *reinterpret_cast<uint32_t(*)[32]>(&s[32]));
      tmem_ld32(s_addr + 64, *reinterpret_cast<uint32_t(*)[32]>(&s[64]));
      tmem_ld32(s_addr + 96, *reinterpret_cast<uint32_t(*)[32]>(&s[96]));
      tmem_wait_ld();
      // s = score * scale * log2(e) - bias, masked entries -inf; running maximum in eight chains
      const uint64_t sl2_2 = wa_pack(sl2, sl2);
      float mx8[8];
#pragma unroll
      for (int c = 0; c < 128; c += 4) {
        const float4 b = c < 64 ? bias[(c >> 2) & 15] : brow[c >> 2];
        float x0, x1, x2, x3;
        wa_unpack(wa_fma2(wa_pack(__uint_as_float(s[c]), __uint_as_float(s[c + 1])), sl2_2, wa_pack(b.x, b.y)), x0, x1);
        wa_unpack(wa_fma2(wa_pack(__uint_as_float(s[c + 2]), __uint_as_float(s[c + 3])), sl2_2, wa_pack(b.z, b.w)), x2, x3);
        s[c] = __float_as_uint(x0); s[c + 1] = __float_as_uint(x1);
        s[c + 2] = __float_as_uint(x2); s[c + 3] = __float_as_uint(x3);
      }
#pragma unroll
      for (int e = 0; e < 8; ++e) mx8[e] = __uint_as_float(s[e]);
#pragma unroll
      for (int i = 8; i < 128; i += 16)
#pragma unroll
        for (int e = 0; e < 8; ++e) mx8[e] = i + 8 + e < 128 ? wa_max3(mx8[e], __uint_as_float(s[i + e]), __uint_as_float(s[(i + 8 + e) & 127]))
                                                             : fmaxf(mx8[e], __uint_as_float(s[i + e]));
      const float mx = wa_max3(wa_max3(mx8[0], mx8[1], mx8[2]), wa_max3(mx8[3], mx8[4], mx8[5]), fmaxf(mx8[6], mx8[7]));
      const float m_new = fmaxf(m_used, mx);
      if (j == lo) {
        m_used = m_new;
      } else {
        const bool need = m_new > m_used + 8.f;
        if (__any_sync(0xffffffffu, need)) {
          const float sc = need ? wa_ex2(m_used - m_new) : 1.f;
#pragma unroll 1
          for (int c = 0; c < p.vdim; c += 32) {
            uint32_t o[32];
            tmem_ld32(o_addr + c, o);
            tmem_wait_ld();
#pragma unroll
            for (int i = 0; i < 32; ++i) o[i] = __float_as_uint(__uint_as_float(o[i]) * sc);
            tmem_st32(o_addr + c, o);
          }
          tmem_wait_st();
          l *= sc;
          if (need) m_used = m_new;
        }
      }
      const uint64_t negm_2 = wa_pack(-m_used, -m_used);
      uint64_t ls2[4] = {0ull, 0ull, 0ull, 0ull};
#pragma unroll
      for (int half = 0; half < 2; ++half) {
        uint32_t pk[32];
#pragma unroll
        for (int i = 0; i < 32; ++i) {
          const int e = half * 64 + 2 * i;
          float p0, p1;
          wa_unpack(wa_add2(wa_pack(__uint_as_float(s[e]), __uint_as_float(s[e + 1])), negm_2), p0, p1);
          p0 = wa_ex2(p0);
          p1 = wa_ex2(p1);
          ls2[i & 3] = wa_add2(ls2[i & 3], wa_pack(p0, p1));
          pk[i] = pack_bf16(p0, p1);
        }
        tmem_st32(s_addr + half * 32, pk);
        tmem_wait_st();
        tc_fence_before();
        mbar_arrive(p_full(t, half));
      }
      float a0, a1, b0, b1;
      wa_unpack(wa_add2(ls2[0], ls2[1]), a0, a1);
      wa_unpack(wa_add2(ls2[2], ls2[3]), b0, b1);
      l += (a0 + a1) + (b0 + b1);
    }
    if (ok && hi > lo) ok = mbar_wait(o_final(t), 0, abort_flag, p.status, ST_TIMEOUT_SOFTMAX);
    if (ok && hi > lo) {
      tc_fence_after();
      const float inv = l > 0.f ? 1.f / l : 0.f;
      const int qr = t * 128 + row;
      bf16* dst = p.out + (long long)(row0 + qr) * p.ldo + (long long)head * p.vdim;
#pragma unroll 1
      for (int c = 0; c < p.vdim; c += 32) {
        uint32_t o[32];
        tmem_ld32(o_addr + c, o);
        tmem_wait_ld();
        if (qr < n_rows) {
#pragma unroll
          for (int q = 0; q < 4; ++q) {
            if (c + q * 8 < p.vdim) {
              uint4 v;
              v.x = pack_bf16(__uint_as_float(o[q * 8 + 0]) * inv, __uint_as_float(o[q * 8 + 1]) * inv);
              v.y = pack_bf16(__uint_as_float(o[q * 8 + 2]) * inv, __uint_as_float(o[q * 8 + 3]) * inv);
              v.z = pack_bf16(__uint_as_float(o[q * 8 + 4]) * inv, __uint_as_float(o[q * 8 + 5]) * inv);
              v.w = pack_bf16(__uint_as_float(o[q * 8 + 6]) * inv, __uint_as_float(o[q * 8 + 7]) * inv);
              reinterpret_cast<uint4*>(dst + c)[q] = v;
            }
          }
        }
      }
    }
  }

  // ---------------- common tail
  tc_fence_before();
  __syncthreads();
  if (warp == 1) {
    __syncwarp();
    tc_fence_after();
    tmem_dealloc(tmem_base, 512);
  }
}

}  // namespace cb

namespace cosmos {

bool window_attn_tc_supported(const WindowAttnArgs& a) {
  const int ps = a.page_size;
  return !a.is_f32 && a.num_pages > 0 && a.G > 0 && a.H % a.G == 0 && a.dim % 8 == 0 && a.vdim % 8 == 0 && a.dim >= 8 &&
         a.vdim >= 8 && a.dim <= 128 && a.vdim <= 128 && a.ldq % 8 == 0 &&
         (ps == 8 || ps == 16 || ps == 32 || ps == 64 || ps == 128);
}

static CUtensorMap page_map(const void* cache, int num_pages, int G, int page_size, int dim) {
  const uint64_t dims[4] = {(uint64_t)dim, (uint64_t)page_size, (uint64_t)G, (uint64_t)num_pages};
  const uint64_t row = (uint64_t)dim * 2;
  const uint64_t strides[3] = {row, row * page_size, row * page_size * G};
  const uint32_t box[4] = {64, (uint32_t)page_size, 1, 1};
  return cbh::make_tmap_bf16(cache, 4, dims, strides, box, true);
}

void window_attn_prefill_tc(const WindowAttnArgs& a, cudaStream_t s) {
  if (a.n_tiles <= 0) return;
  if (!window_attn_tc_supported(a) || a.window < 1 || a.tile_rows > WINDOW_ATTN_TC_ROWS || a.ldo % 8 != 0)
    throw std::runtime_error("window_attn_prefill_tc: unsupported shape");
  static bool configured = false;
  if (!configured) {
    if (cudaFuncSetAttribute(cb::window_attn_prefill_kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, cb::WA_SMEM) != cudaSuccess)
      throw std::runtime_error("window_attn_prefill_tc: shared memory not available");
    configured = true;
  }
  const uint64_t qd[3] = {(uint64_t)a.dim, (uint64_t)a.H, (uint64_t)a.n_rows};
  const uint64_t qs[2] = {(uint64_t)a.dim * 2, (uint64_t)a.ldq * 2};
  const uint32_t qb[3] = {64, 1, 128};
  const CUtensorMap tq = cbh::make_tmap_bf16(a.q, 3, qd, qs, qb, true);
  const CUtensorMap tk = page_map(a.k_cache, a.num_pages, a.G, a.page_size, a.dim);
  const CUtensorMap tv = page_map(a.v_cache, a.num_pages, a.G, a.page_size, a.vdim);
  cb::WinAttnParams p{};
  p.tiles = reinterpret_cast<const int4*>(a.tiles);
  p.table = a.table; p.max_pages = a.max_pages; p.num_pages = a.num_pages; p.page_size = a.page_size;
  p.group = a.H / a.G; p.kdim = a.dim; p.vdim = a.vdim; p.window = a.window;
  p.scale_log2 = a.scale * 1.4426950408889634f;
  p.r1 = a.r1; p.r2 = a.r2;
  p.out = reinterpret_cast<bf16*>(a.out); p.ldo = a.ldo;
  p.status = a.status;
  cb::window_attn_prefill_kernel<<<dim3(a.n_tiles, a.H), cb::WA_THREADS, cb::WA_SMEM, s>>>(tq, tk, tv, p);
}

}  // namespace cosmos
