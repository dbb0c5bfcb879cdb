"""Ops of the config-declared decoder stacks (models/stack.py): CUDA tensors (bf16 or fp32) run the kernels of
csrc/stack_step.cu, csrc/window_attn*.cu, csrc/paged_decode_tc.cu and the tile-map mode of csrc/gemm_tcgen05.cu; CPU
tensors run the plain PyTorch definitions below. Scores, softmax weights, norms and the residual stream are 32-bit in
both element types."""
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
    keys 0 <= i - j < window with score scale * q.k - r1 ln(1 + r2 (i - j)). Portions: `tiles` int32 [t, 4] (sequence, first
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
            s = s - r1[:, None, None] * torch.log1p(r2[:, None, None] * dist.clamp(min=0).float()[None])
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
