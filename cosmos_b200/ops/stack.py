"""Ops of the config-declared decoder stacks (models/stack.py): CUDA tensors (bf16 or fp32) run the kernels of
csrc/stack_step.cu, stack_branch.cu, selective_scan.cu, matrix_memory*.cu, window_attn*.cu, paged_decode_tc.cu and the
tile-map mode of gemm_tcgen05.cu; CPU tensors run the plain PyTorch definitions below. Scores, softmax weights, norms,
recurrent states with all that enters them, and the residual stream are 32-bit in both element types."""
from __future__ import annotations

from dataclasses import dataclass
from typing import List, Optional, Sequence, Tuple

import torch
import torch.nn.functional as F

from . import _k, load_extension

NO_WINDOW = 1 << 30
TC_TILE_ROWS, SIMT_TILE_ROWS = 256, 16   # query rows per tile of the tensor-core / CUDA-core attention kernels


def _cuda(t: torch.Tensor) -> bool:
    if not t.is_cuda:
        return False
    if not load_extension():
        raise RuntimeError("cosmos_b200 kernel library is not available on this GPU host; run `python -m cosmos_b200.ops._build`")
    return True


def pad8(n: int) -> int:
    """Row lengths are padded to 16 bytes of bf16, which the TMA copies of the GEMM need."""
    return (n + 7) // 8 * 8


# --------------------------------------------------------------------------- residual stream + grouped RMS norm
def grouped_rmsnorm_ref(x: torch.Tensor, gamma: torch.Tensor, groups: int, eps: float) -> torch.Tensor:
    p = x.float().reshape(*x.shape[:-1], groups, -1)
    p = p / torch.sqrt(p.pow(2).mean(-1, keepdim=True) + eps)
    return p.reshape(x.shape) * gamma.float()


def residual_norm_(x: torch.Tensor, gamma: Optional[torch.Tensor], groups: int, eps: float, h: Optional[torch.Tensor] = None,
                   h_rows: Optional[torch.Tensor] = None, y: Optional[torch.Tensor] = None,
                   y_rows: Optional[torch.Tensor] = None, weight: float = 1.0, embed: Optional[torch.Tensor] = None,
                   tokens: Optional[torch.Tensor] = None, embed_scale: float = 1.0) -> None:
    """One pass over the fp32 residual stream x [n, d], in place: x = embed[tokens] * embed_scale (if given), x += weight *
    the sum of its rows of y (`y_rows` [n * top], else row i; a 3-D fp32 y holds split-K partial sums), and
    h = grouped RMS norm(x) * gamma, stored at row i or at the rows h_rows [n * top] (expert dispatch)."""
    if _cuda(x):
        _k().residual_norm_(x, embed, tokens, float(embed_scale), y, y_rows, float(weight), gamma, int(groups), float(eps),
                            h, h_rows)
        return
    n, d = x.shape
    if embed is not None:
        x.copy_(embed[tokens].float() * embed_scale)
    if y is not None:
        yy = (y.sum(0) if y.dim() == 3 else y).float()[:, :d]
        x += weight * (yy[:n] if y_rows is None else yy[y_rows.long()].reshape(n, -1, d).sum(1))
    if h is not None:
        v = grouped_rmsnorm_ref(x, gamma, groups, eps).to(h.dtype)
        if h_rows is None:
            h[:n, :d] = v
        else:
            h[h_rows.long(), :d] = v.repeat_interleave(h_rows.numel() // n, dim=0)


# --------------------------------------------------------------------------- q / k / v
def qkv_value_post(qkv: torch.Tensor, bias: Optional[torch.Tensor], heads: int, kv_heads: int, eps: float, value_norm: bool,
                   slots: torch.Tensor, k_cache: torch.Tensor, v_cache: torch.Tensor,
                   v_first_out: Optional[torch.Tensor] = None, v_first_in: Optional[torch.Tensor] = None,
                   lam: Optional[torch.Tensor] = None) -> torch.Tensor:
    """Keys and values of n tokens into their cache rows, values normed per head and mixed with the values `v_first_in`
    [n, kv_heads, vdim] of an earlier layer; `v_first_out` receives this layer's. qkv: finished rows [n, >= cols], or fp32
    split-K partial sums [splits, n, >= cols] to which `bias` is added here. Returns q [n, heads, dim]."""
    dim, vdim = k_cache.shape[3], v_cache.shape[3]
    if _cuda(qkv):
        q = _k().qkv_value_post(qkv, bias if qkv.dim() == 3 else None, heads, kv_heads, float(eps), value_norm, slots,
                                k_cache, v_cache, v_first_out, v_first_in, lam)
        return q if qkv.dim() == 3 else qkv[:, :heads * dim].unflatten(1, (heads, dim))
    n, qc, kc = qkv.shape[-2], heads * dim, kv_heads * dim
    rows = qkv
    if qkv.dim() == 3:
        rows = qkv.sum(0) + (0 if bias is None else bias.float())
    q = rows[:, :qc].reshape(n, heads, dim).to(k_cache.dtype)
    k = rows[:, qc:qc + kc].reshape(n, kv_heads, dim)
    v = rows[:, qc + kc:qc + kc + kv_heads * vdim].reshape(n, kv_heads, vdim).float()
    if value_norm:
        v = v / torch.sqrt(v.pow(2).mean(-1, keepdim=True) + eps)
    if v_first_out is not None:
        v_first_out.copy_(v.reshape(v_first_out.shape))
    if v_first_in is not None:
        v = (1.0 - lam) * v + lam * v_first_in.reshape(v.shape)
    page, off = slots // k_cache.shape[2], slots % k_cache.shape[2]
    k_cache[page, :, off] = k.to(k_cache.dtype)
    v_cache[page, :, off] = v.to(v_cache.dtype)
    return q


# --------------------------------------------------------------------------- windowed attention over the paged cache
def attn_tile_rows(heads: int, kv_heads: int, dim: int, vdim: int, page_size: int, dtype, device) -> int:
    """Query rows per tile of the portion kernel that takes this shape."""
    if torch.device(device).type == "cuda" and dtype == torch.bfloat16 and load_extension():
        if torch.ops.cosmos_b200.window_attn_tc_supported(heads, kv_heads, dim, vdim, page_size)[0]:
            return TC_TILE_ROWS
    return SIMT_TILE_ROWS


def make_tiles(portions: Sequence[Tuple[int, int, int, int]], tile_rows: int) -> List[Tuple[int, int, int, int]]:
    """portions: (sequence, first row, rows, position of the first row) -> the same cut into tiles."""
    out = []
    for seq, row0, n, pos0 in portions:
        for o in range(0, n, tile_rows):
            out.append((seq, row0 + o, min(tile_rows, n - o), pos0 + o))
    return out


def window_attn(q: torch.Tensor, k_cache: torch.Tensor, v_cache: torch.Tensor, table: torch.Tensor, scale: float,
                window: Optional[int], r1: Optional[torch.Tensor] = None, r2: Optional[torch.Tensor] = None,
                tiles: Optional[torch.Tensor] = None, tile_rows: int = 0, seq_lens: Optional[torch.Tensor] = None,
                max_len: Optional[int] = None, impl: int = 0) -> torch.Tensor:
    """Attention of the new tokens q [n, H, dim] over the paged cache (their own keys included): the query at position i sees
    keys 0 <= i - j < window with score scale * q.k - r1 ln(1 + r2 (i - j)), or - r1 (i - j) without r2. Portions: `tiles` int32 [t, 4] (sequence, first
    row, rows, position). Decode step: `seq_lens` [n] (lengths with the new token; 0 = idle slot, output 0). Returns
    [n, H * vdim]. `max_len`: host-known bound of seq_lens. impl 1 forces the CUDA-core kernel."""
    w = NO_WINDOW if window is None else int(window)
    if _cuda(q):
        splits = 1
        if tiles is None and impl == 0:
            page = k_cache.shape[2]
            span = min(table.shape[1] * page if max_len is None else max_len, w + page - 1)
            splits = int(torch.ops.cosmos_b200.window_attn_decode_splits(q.shape[0], k_cache.shape[1], span))
        return _k().window_attn(q, k_cache, v_cache, table, seq_lens, tiles, tile_rows, float(scale), w, r1, r2, splits, impl)
    n, heads, _ = q.shape
    g, page, vdim = k_cache.shape[1], k_cache.shape[2], v_cache.shape[3]
    out = torch.zeros(n, heads, vdim, dtype=torch.float32, device=q.device)
    rows = tiles.tolist() if tiles is not None else [(b, b, 1, int(l) - 1) for b, l in enumerate(seq_lens.tolist())]
    for seq, row0, cnt, pos0 in rows:
        if pos0 < 0:
            continue
        lo, hi = max(0, pos0 - w + 1), pos0 + cnt
        j = torch.arange(lo, hi, device=q.device)
        pg = table[seq, j // page].long()
        k = k_cache[pg, :, j % page].float().repeat_interleave(heads // g, dim=1)
        v = v_cache[pg, :, j % page].float().repeat_interleave(heads // g, dim=1)
        dist = torch.arange(pos0, hi, device=q.device)[:, None] - j[None]
        s = torch.einsum("rhd,khd->hrk", q[row0:row0 + cnt].float(), k) * scale
        if r1 is not None:
            far = dist.clamp(min=0).float()[None]
            s = s - r1[:, None, None] * (far if r2 is None else torch.log1p(r2[:, None, None] * far))
        s = s.masked_fill((dist < 0) | (dist >= w), float("-inf"))
        out[row0:row0 + cnt] = torch.einsum("hrk,khd->rhd", torch.softmax(s, dim=-1), v)
    return out.reshape(n, -1).to(q.dtype)


# --------------------------------------------------------------------------- table-routed experts
@dataclass
class Routing:
    """Expert order of a step for every layer with experts: `rows[i]` [n * top] places of the (token, k) pairs, `tiles[i]` the
    layer's m-tiles (expert, first row, rows), `n_tiles[i]` how many."""
    rows: List[torch.Tensor]
    tiles: List[torch.Tensor]
    n_tiles: List[torch.Tensor]
    tile_m: List[int]


def pick_tile_m(n: int, top: int, experts: int, dtype, device) -> int:
    """256-row tiles (CTA pairs) once an expert sees enough rows to fill them."""
    if torch.device(device).type != "cuda" or dtype != torch.bfloat16:
        return 128
    return 256 if n * top >= 192 * experts else 128


def moe_route(tokens: torch.Tensor, vocab: int, tables: Sequence[torch.Tensor], experts: Sequence[int], tile_m: Sequence[int],
              desc: Optional[torch.Tensor] = None) -> Routing:
    """The experts depend on the token ids alone, so one launch routes all layers of a step. `desc`: device descriptors
    (`route_desc`) of these tables and tile sizes."""
    n = tokens.shape[0]
    tops = [t.shape[1] for t in tables]
    if _cuda(tokens):
        top_max = max(tops)
        bound = max(min(n * tp, n * tp // tm + e) for tp, e, tm in zip(tops, experts, tile_m))
        rows, tiles, cnt = _k().moe_route(tokens, vocab, desc, max(experts), top_max, max(1, bound))
        return Routing([rows[i, :n * tp] for i, tp in enumerate(tops)],
                       [tiles[i, :max(1, min(n * tp, n * tp // tm + e))] for i, (tp, e, tm) in enumerate(zip(tops, experts, tile_m))],
                       [cnt[i:i + 1] for i in range(len(tables))], list(tile_m))
    out = Routing([], [], [], list(tile_m))
    for table, e, tm in zip(tables, experts, tile_m):
        ex = table[tokens].reshape(-1).long()
        order = torch.argsort(ex, stable=True)
        rows = torch.empty_like(ex)
        rows[order] = torch.arange(ex.numel(), device=ex.device)
        tl, start = [], 0
        for i, c in enumerate(torch.bincount(ex, minlength=e).tolist()):
            tl += [(i, start + o, min(tm, c - o), 0) for o in range(0, c, tm)]
            start += c
        out.rows.append(rows.to(torch.int32))
        out.tiles.append(torch.tensor(tl, dtype=torch.int32).reshape(-1, 4))
        out.n_tiles.append(torch.tensor([len(tl)], dtype=torch.int32))
    return out


def route_desc(tables: Sequence[torch.Tensor], experts: Sequence[int], tile_m: Sequence[int]) -> torch.Tensor:
    return torch.tensor([[t.data_ptr(), e, t.shape[1], m] for t, e, m in zip(tables, experts, tile_m)], dtype=torch.int64,
                        device=tables[0].device)


def expert_splits(n: int, top: int, experts: int, tile_m: int, n_cols: int, k: int) -> int:
    """Split-K count of an expert product: fill the 148 SMs when few experts are hit (a small decode batch)."""
    units = min(n * top, n * top // tile_m + experts) * ((n_cols + 255) // 256)
    kb = (k + 63) // 64
    if units >= 148 or kb < 8:
        return 1
    return max(1, min(148 // units, kb // 4, 16))


def grouped_gemm(a: torch.Tensor, w: torch.Tensor, tiles: torch.Tensor, n_tiles: torch.Tensor, tile_m: int, gelu: bool = False,
                 k_splits: int = 1, partial: bool = False) -> torch.Tensor:
    """a [R, K] rows sorted by expert, w [E, N, K] -> [R, N] with each row times its expert's weights (then exact gelu), or
    fp32 split-K partial sums [splits, R, N] with `partial` (bf16 on CUDA only)."""
    if _cuda(a):
        return _k().grouped_gemm(a, w, tiles, n_tiles, tile_m, gelu, k_splits, partial)
    out = torch.zeros(a.shape[0], w.shape[1], dtype=torch.float32, device=a.device)
    for e, r0, cnt, _ in tiles[:int(n_tiles)].tolist():
        out[r0:r0 + cnt] = a[r0:r0 + cnt].float() @ w[e].float().t()
    out = F.gelu(out) if gelu else out
    return out.to(a.dtype)


def gemm_partial(a: torch.Tensor, w: torch.Tensor) -> torch.Tensor:
    """bf16 a [M, K] w [N, K]^T as fp32 partial sums [splits, M, N] for a consumer kernel that adds them up (CUDA)."""
    return _k().gemm_partial(a, w)


# --------------------------------------------------------------------------- parallel layers
def sinusoid_turns(width: int, device) -> torch.Tensor:
    """Turns per position of the sinusoid's frequencies, fp64 [(width + 1) // 2]: entries 2i and 2i + 1 share one."""
    i = torch.arange((width + 1) // 2, dtype=torch.float64)
    return (10000.0 ** (-2.0 * i / width) / (2.0 * torch.pi)).to(device)


def _rows(t: torch.Tensor) -> torch.Tensor:
    """Finished rows of a source (split-K partial sums added up), fp32."""
    return (t.sum(0) if t.dim() == 3 else t).float()


def branch_norm_(x: torch.Tensor, eps: float, dtype, normed: Sequence[Tuple[torch.Tensor, torch.Tensor]] = (), coef: float = 1.0,
                 plain: Optional[torch.Tensor] = None, gammas: Sequence[Optional[torch.Tensor]] = (), gamma_add: float = 0.0,
                 hs: Sequence[Optional[torch.Tensor]] = (), embed: Optional[torch.Tensor] = None, tokens: Optional[torch.Tensor] = None,
                 embed_scale: float = 1.0, pos_turns: Optional[torch.Tensor] = None, positions: Optional[torch.Tensor] = None) -> None:
    """One pass over the fp32 residual stream x [n, d], in place: x = embed[tokens] * embed_scale + sinusoid(positions) (if
    given), x += coef * sum of y / rms(y) * w over the branches (y, w) in `normed` (up to two) + plain, and for each of up to
    two outputs hs[i] = x / rms(x) * (gamma_add + gammas[i]). Branches and `plain` are rows [n, >= d] or fp32 partial sums
    [splits, n, >= d]; weights are fp32."""
    gammas, hs = list(gammas) + [None] * (2 - len(gammas)), list(hs) + [None] * (2 - len(hs))
    if _cuda(x):
        _k().branch_norm_(x, embed, tokens, float(embed_scale), pos_turns, positions, [y for y, _ in normed], [w for _, w in normed],
                          float(coef), plain, gammas[0], gammas[1], float(gamma_add), float(eps), hs[0], hs[1], dtype == torch.float32)
        return
    n, d = x.shape
    if embed is not None:
        x.copy_(embed[tokens].float() * embed_scale)
        if pos_turns is not None:
            ang = positions.double()[:, None] * pos_turns[None] * (2.0 * torch.pi)
            x += torch.stack([ang.sin(), ang.cos()], dim=-1).reshape(n, -1)[:, :d].float()
    for y, w in normed:
        x += coef * grouped_rmsnorm_ref(_rows(y)[:, :d], w, 1, eps)
    if plain is not None:
        x += _rows(plain)[:, :d]
    for g, h in zip(gammas, hs):
        if h is not None:
            h[:n, :d] = grouped_rmsnorm_ref(x, gamma_add + g, 1, eps).to(h.dtype)


def qk_norm_post(q: torch.Tensor, k: torch.Tensor, heads: int, kv_heads: int, wq: torch.Tensor, wk: torch.Tensor, eps: float,
                 q_temp: Optional[Tuple[float, int]], positions: torch.Tensor, slots: torch.Tensor, k_cache: torch.Tensor,
                 v_cache: torch.Tensor) -> torch.Tensor:
    """Projected queries [n, >= heads * dim] and keys [n, >= kv_heads * dim] (or partial sums): both RMS-normed over all heads at
    once, queries times 1 + coef ln(floor((p + 1) / every) + 1); normed keys go to their cache rows, the projected ones to the
    value cache. Returns q [n, heads, dim]."""
    coef, every = q_temp if q_temp is not None else (0.0, 0)
    if _cuda(q):
        return _k().qk_norm_post(q, k, heads, kv_heads, wq, wk, float(eps), float(coef), int(every), positions, slots, k_cache, v_cache)
    n, dim = slots.shape[0], k_cache.shape[3]
    qr, kr = _rows(q)[:, :heads * dim], _rows(k)[:, :kv_heads * dim]
    qn = grouped_rmsnorm_ref(qr, wq, 1, eps)
    if every > 0:
        qn = qn * (1.0 + coef * torch.log((positions + 1).div(every, rounding_mode="floor").float() + 1.0))[:, None]
    page, off = slots // k_cache.shape[2], slots % k_cache.shape[2]
    k_cache[page, :, off] = grouped_rmsnorm_ref(kr, wk, 1, eps).reshape(n, kv_heads, dim).to(k_cache.dtype)
    v_cache[page, :, off] = kr.reshape(n, kv_heads, dim).to(v_cache.dtype)
    return qn.reshape(n, heads, dim).to(k_cache.dtype)


# --------------------------------------------------------------------------- rows of recurrent layers
CONV_TILE_ROWS = 32
MEMORY_SLICE = 32   # value columns per copy of a memory's normaliser state


@dataclass
class StepRows:
    """The tokens of a step as recurrent layers see them: `portions` int32 [p, 4] (sequence, first row, rows, position) with
    `conv_tiles` int32 [t, 8] (sequence, first row, rows, the portion's position and first row), or `lens` int32 [n] of a decode
    step (one row per sequence, at position lens - 1; 0 = idle, the state is left alone). `state_slots` int32 [sequences]: where
    a sequence's state lives. A sequence at position 0 starts from a zero state whatever its slot holds."""
    state_slots: torch.Tensor
    portions: Optional[torch.Tensor] = None
    conv_tiles: Optional[torch.Tensor] = None
    lens: Optional[torch.Tensor] = None

    def host(self) -> List[Tuple[int, int, int, int]]:
        """(state slot, first row, rows, position) of every portion with a token (CPU definitions)."""
        rows = self.portions.tolist() if self.portions is not None else [(b, b, 1, int(l) - 1) for b, l in enumerate(self.lens.tolist())]
        return [(int(self.state_slots[s]), r0, n, p) for s, r0, n, p in rows if p >= 0]


def make_conv_tiles(portions: Sequence[Tuple[int, int, int, int]]) -> List[Tuple[int, ...]]:
    return [(seq, row0 + o, min(CONV_TILE_ROWS, n - o), pos0, row0, 0, 0, 0)
            for seq, row0, n, pos0 in portions for o in range(0, n, CONV_TILE_ROWS)]


# --------------------------------------------------------------------------- selective scan
def causal_conv(x: torch.Tensor, w: torch.Tensor, b: torch.Tensor, conv_state: torch.Tensor, rows: StepRows, n: int) -> torch.Tensor:
    """u[t] = silu(b + sum_j w[:, j] x[t - (taps - 1 - j)]) over rows x [n, >= inner] (or partial sums); conv_state [slots, taps - 1,
    inner] gives the inputs before a portion and takes its last ones. Returns [n, inner]."""
    if _cuda(x):
        return _k().causal_conv(x, w, b, conv_state, rows.state_slots, rows.portions, rows.conv_tiles, rows.lens, n)
    inner, taps = w.shape
    xr = _rows(x)[:, :inner].to(conv_state.dtype).float()
    u = torch.zeros(n, inner)
    for slot, r0, cnt, pos in rows.host():
        before = conv_state[slot].float() if pos > 0 else torch.zeros(taps - 1, inner)
        seq = torch.cat([before, xr[r0:r0 + cnt]])
        acc = b + sum(w[:, j] * seq[j:j + cnt] for j in range(taps))
        u[r0:r0 + cnt] = acc * torch.sigmoid(acc)
        conv_state[slot] = seq[seq.shape[0] - (taps - 1):].to(conv_state.dtype)
    return u.to(conv_state.dtype)


def scan_decay(a_log: torch.Tensor) -> torch.Tensor:
    """A log2(e) with A = -exp(A_log), fp32: the decay of a step is 2^(dt * this)."""
    return (-torch.exp(a_log.double()) / torch.log(torch.tensor(2.0, dtype=torch.float64))).float()


def selective_scan(u: torch.Tensor, dt: torch.Tensor, z: torch.Tensor, bc: torch.Tensor, dt_bias: torch.Tensor, a2: torch.Tensor,
                   d: torch.Tensor, state: torch.Tensor, rows: StepRows, y: torch.Tensor, y_cols: int) -> None:
    """S[c, s] <- 2^(dt_c a2[c, s]) S[c, s] + dt_c u_c B_s; y_c = (sum_s S[c, s] C_s + D_c u_c) silu(z_c), with
    dt = softplus(dt + dt_bias). bc holds B, then C. `state` [slots, inner, states] fp32. Writes columns [0, inner) of y and
    zeros up to y_cols."""
    if _cuda(u):
        _k().selective_scan(u, dt, z, bc, dt_bias, a2, d, state, y, y_cols, rows.state_slots, rows.portions, rows.lens)
        return
    inner, ns = a2.shape
    ur, zr = u.float(), _rows(z)[:, :inner]
    step = F.softplus(_rows(dt)[:, :inner] + dt_bias, threshold=1e9)
    b, c = _rows(bc)[:, :ns], _rows(bc)[:, ns:2 * ns]
    y[:, :y_cols] = 0
    for slot, r0, cnt, pos in rows.host():
        s = state[slot] if pos > 0 else torch.zeros(inner, ns)
        for t in range(r0, r0 + cnt):
            s = torch.exp2(step[t][:, None] * a2) * s + (step[t] * ur[t])[:, None] * b[t][None]
            out = s @ c[t] + d * ur[t]
            y[t, :inner] = (out * zr[t] * torch.sigmoid(zr[t])).to(y.dtype)
        state[slot] = s


# --------------------------------------------------------------------------- matrix memory
def memory_slices(vdim: int) -> int:
    return (vdim + MEMORY_SLICE - 1) // MEMORY_SLICE


def matrix_memory(q: torch.Tensor, k: torch.Tensor, v: torch.Tensor, gates: torch.Tensor, gate_bias: torch.Tensor, cap: float,
                  state: torch.Tensor, norm: torch.Tensor, peak: torch.Tensor, rows: StepRows, n: int, dtype, impl: int = 0) -> torch.Tensor:
    """mLSTM over rows q, k [n, >= H dim], v [n, >= H vdim] (or partial sums) and fp32 gate rows [n, >= 2 H] (input gates, then
    forget gates): log gates i = cap tanh(. / cap), f = logsigmoid(cap tanh(. / cap)), running maximum m = max(f + m, i) from 0,
    S = exp(f + m' - m) S + exp(i - m) k v^T, n likewise, o = S^T q / (max(|n . q|, exp(-m)) + 1e-6), q over sqrt(dim).
    state [slots, H, dim, vdim], norm [slots, H, slices, dim], peak [slots, H, slices] fp32. Returns [n, H * vdim]. impl 1 forces the CUDA-core kernel."""
    heads, dim, vdim = state.shape[1:]
    if _cuda(q):
        return _k().matrix_memory(q, k, v, gates, gate_bias, dim ** -0.5, float(cap), state, norm, peak, rows.state_slots, rows.portions,
                                  rows.lens, n, dtype == torch.float32, impl)
    qr = _rows(q)[:, :heads * dim].reshape(n, heads, dim) * dim ** -0.5
    kr, vr = _rows(k)[:, :heads * dim].reshape(n, heads, dim), _rows(v)[:, :heads * vdim].reshape(n, heads, vdim)
    g = cap * torch.tanh((_rows(gates)[:, :2 * heads] + gate_bias) / cap)
    gi, gf = g[:, :heads], F.logsigmoid(g[:, heads:])
    out = torch.zeros(n, heads, vdim)
    for slot, r0, cnt, pos in rows.host():
        s, z, m = (state[slot], norm[slot, :, 0], peak[slot, :, 0]) if pos > 0 else (torch.zeros(heads, dim, vdim),
                                                                                   torch.zeros(heads, dim), torch.zeros(heads))
        for t in range(r0, r0 + cnt):
            m_new = torch.maximum(gf[t] + m, gi[t])
            keep, take = torch.exp(gf[t] + m - m_new)[:, None], torch.exp(gi[t] - m_new)[:, None]
            s = keep[..., None] * s + (take * kr[t])[..., None] * vr[t][:, None]
            z, m = keep * z + take * kr[t], m_new
            den = torch.maximum((z * qr[t]).sum(-1).abs(), torch.exp(-m)) + 1e-6
            out[t] = torch.einsum("hdv,hd->hv", s, qr[t]) / den[:, None]
        state[slot], norm[slot], peak[slot] = s, z[:, None].expand_as(norm[slot]), m[:, None].expand_as(peak[slot])
    return out.reshape(n, -1).to(dtype)


def head_norm_gate(o: torch.Tensor, g: torch.Tensor, w: torch.Tensor, heads: int, eps: float) -> torch.Tensor:
    """o [n, heads * size]: every head divided by its root mean square, times w, times sigmoid(g)."""
    if _cuda(o):
        return _k().head_norm_gate(o, g, w, heads, float(eps))
    return (grouped_rmsnorm_ref(o, w, heads, eps) * torch.sigmoid(_rows(g)[:, :o.shape[1]])).to(o.dtype)
