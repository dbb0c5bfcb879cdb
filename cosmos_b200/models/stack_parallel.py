"""Layers of decoder stacks in parallel order (config.StackConfig, order "parallel"): x += mixer(norm1 x) + ff(norm2 x). The
mixer is a selective scan, or attention and a matrix memory side by side; the feed-forward is a dense SwiGLU or none.

Launches per layer on CUDA bf16 (plus a split-K reduction where the framework's skinny GEMMs need one):
  scan     in GEMM -> convolution -> x GEMM -> dt GEMM -> scan + gate -> gate / up GEMM (SwiGLU) -> one GEMM over [W_o | W_down]
  branches q/k/memory GEMM (+ a small fp32 one for the memory's gates) -> q/k norm + cache write -> paged attention -> W_o;
           memory -> head norm + gate -> W_o; gate / up GEMM (SwiGLU) -> W_down
and one pass over the residual stream at the end: branch norms, sum, and both norms of the next layer. The scan and the
SwiGLU product write side by side into one buffer, so that their two output projections are one product whose sum needs no
pass of its own. For a few rows (decode) the products leave split-K partial sums that the kernel behind each reduces."""
from __future__ import annotations

from typing import Dict, List, Optional, Tuple

import torch
import torch.nn as nn

from .. import ops
from ..config import AttentionSpec, DenseSpec, MatrixMemorySpec, ParallelSpec, SelectiveScanSpec, StackConfig, StackLayerSpec
from ..ops import stack as sops
from ..ops.stack import pad8

F32 = torch.float32
Named = List[Tuple[str, torch.Tensor]]


def param(shape, dtype, device) -> nn.Parameter:
    return nn.Parameter(torch.zeros(shape, dtype=dtype, device=device), requires_grad=False)


def split_k(n: int, w: torch.Tensor) -> bool:
    """Whether a product of n rows is skinny enough that the GEMM splits K (and a consumer can reduce the sums)."""
    return (w.is_cuda and w.dtype == torch.bfloat16 and ops.load_extension()
            and torch.ops.cosmos_b200.gemm_pick_k_splits(n, w.shape[0], w.shape[1], ops.EPI_PLAIN) > 1)


def product(a: torch.Tensor, w: torch.Tensor) -> torch.Tensor:
    """a w^T as rows, or as fp32 partial sums for a few rows."""
    return sops.gemm_partial(a, w) if split_k(a.shape[0], w) else ops.gemm(a, w)


class ScanMixer(nn.Module):
    """Selective scan; its output projection is part of the layer's combined one."""

    def __init__(self, spec: SelectiveScanSpec, d: int, eps: float, dtype, device):
        super().__init__()
        self.spec, self.d = spec, d
        c, c8, r8 = spec.inner, pad8(spec.inner), pad8(spec.dt_rank)
        self.cols = c8                                     # columns of the combined output product
        self.w_in = param((2 * c8, pad8(d)), dtype, device)
        self.w_x = param((r8 + pad8(2 * spec.state), c8), dtype, device)
        self.w_dt = param((c8, r8), dtype, device)
        self.conv_w, self.conv_b = param((c, spec.conv), F32, device), param((c,), F32, device)
        self.dt_bias, self.skip = param((c,), F32, device), param((c,), F32, device)
        self.a_log = param((c, spec.state), F32, device)
        self.register_buffer("a2", torch.zeros(c, spec.state, dtype=F32, device=device), persistent=False)

    def finish(self) -> None:
        self.a2.copy_(sops.scan_decay(self.a_log))

    def views(self, w_o: torch.Tensor) -> Named:
        m, c, c8, r8 = self.spec, self.spec.inner, pad8(self.spec.inner), pad8(self.spec.dt_rank)
        return [("in", (self.w_in[:c, :self.d], self.w_in[c8:c8 + c, :self.d])), ("conv", self.conv_w), ("conv.b", self.conv_b),
                ("x", (self.w_x[:m.dt_rank, :c], self.w_x[r8:r8 + 2 * m.state, :c])), ("dt", self.w_dt[:c, :m.dt_rank]),
                ("dt.b", self.dt_bias), ("A_log", self.a_log), ("D", self.skip), ("o", w_o[:self.d, :c])]

    def state_shapes(self, dtype) -> Dict[str, Tuple]:
        m = self.spec
        return {"conv": ((m.conv - 1, m.inner), dtype), "S": ((m.inner, m.state), F32)}

    def forward(self, h: torch.Tensor, batch, state: Dict[str, torch.Tensor], y: torch.Tensor) -> None:
        """Scan of the normed rows h [n, d] into columns [0, self.cols) of y."""
        m, n = self.spec, h.shape[0]
        c, c8, r8 = m.inner, pad8(m.inner), pad8(m.dt_rank)
        xz = product(h, self.w_in[:, :self.d])
        u = sops.causal_conv(xz[..., :c], self.conv_w, self.conv_b, state["conv"], batch.rows, n)
        dbc = ops.gemm(u, self.w_x[:, :c])
        dt = ops.gemm(dbc[:, :m.dt_rank], self.w_dt[:, :m.dt_rank])
        sops.selective_scan(u, dt, xz[..., c8:], dbc[:, r8:], self.dt_bias, self.a2, self.skip, state["S"], batch.rows, y, self.cols)


class BranchMixer(nn.Module):
    """Attention (left) and a matrix memory (right) on the same input; all their input projections are rows of one matrix."""

    def __init__(self, spec: ParallelSpec, d: int, eps: float, dtype, device):
        super().__init__()
        self.spec, self.d, self.eps, self.dtype = spec, d, eps, dtype
        a, r = spec.left, spec.right
        if not (a.qk_norm and a.key_values) or a.distance_bias or a.value_norm or a.value_mix or a.qkv_bias:
            raise ValueError("attention beside a matrix memory takes normed queries and keys that serve as values")
        self.at: Dict[str, int] = {}
        row = 0
        for name, size in (("lq", a.heads * a.dim), ("lk", a.kv_heads * a.dim), ("q", r.heads * r.dim), ("k", r.heads * r.dim),
                           ("v", r.heads * r.vdim), ("g", r.heads * r.vdim), ("gates", 2 * r.heads)):
            self.at[name] = row
            row += pad8(size)
        self.rows = row
        self.w_in = param((row, pad8(d)), dtype, device)
        self.lo, self.ro = a.heads * a.vdim, r.heads * r.vdim
        self.w_left = param((pad8(d), pad8(self.lo)), dtype, device)
        self.w_right = param((pad8(d), pad8(self.ro)), dtype, device)
        self.q_norm, self.k_norm = param((a.heads * a.dim,), F32, device), param((a.kv_heads * a.dim,), F32, device)
        self.gate_bias, self.norm = param((2 * r.heads,), F32, device), param((self.ro,), F32, device)
        self.left_out, self.right_out = param((d,), F32, device), param((d,), F32, device)
        slopes = 2.0 ** (-8.0 * torch.arange(1, a.heads + 1, dtype=torch.float64) / a.heads) if a.linear_bias else torch.empty(0)
        self.register_buffer("slopes", slopes.to(dtype=F32, device=device), persistent=False)

    def finish(self) -> None:
        pass

    def views(self, w_o: Optional[torch.Tensor]) -> Named:
        a, r, d = self.spec.left, self.spec.right, self.d

        def rows(name: str, size: int, skip: int = 0) -> torch.Tensor:
            return self.w_in[self.at[name] + skip:self.at[name] + skip + size, :d]

        return [("left.q", rows("lq", a.heads * a.dim)), ("left.k", rows("lk", a.kv_heads * a.dim)), ("left.q.norm", self.q_norm),
                ("left.k.norm", self.k_norm), ("left.o", self.w_left[:d, :self.lo]), ("right.q", rows("q", r.heads * r.dim)),
                ("right.k", rows("k", r.heads * r.dim)), ("right.v", rows("v", self.ro)), ("right.g", rows("g", self.ro)),
                ("right.o", self.w_right[:d, :self.ro]), ("right.norm", self.norm), ("right.i", rows("gates", r.heads)),
                ("right.i.b", self.gate_bias[:r.heads]), ("right.f", rows("gates", r.heads, r.heads)),
                ("right.f.b", self.gate_bias[r.heads:]), ("left.out", self.left_out), ("right.out", self.right_out)]

    def state_shapes(self, dtype) -> Dict[str, Tuple]:
        r = self.spec.right
        s = sops.memory_slices(r.vdim)
        return {"S": ((r.heads, r.dim, r.vdim), F32), "n": ((r.heads, s, r.dim), F32), "m": ((r.heads, s), F32)}

    def forward(self, h: torch.Tensor, batch, k_cache: torch.Tensor, v_cache: torch.Tensor, state: Dict[str, torch.Tensor],
                tile_rows: int) -> List[Tuple[torch.Tensor, torch.Tensor]]:
        """The two outputs before their norms, with the norms' weights."""
        a, r, n, at = self.spec.left, self.spec.right, h.shape[0], self.at
        w = self.w_in[:, :self.d]
        if split_k(n, w):
            p = sops.gemm_partial(h, w)
            gates = p[..., at["gates"]:]
        else:   # the memory's gates stay in 32-bit
            p, wg = ops.gemm(h, w[:at["gates"]]), w[at["gates"]:]
            gates = sops.gemm_partial(h, wg) if h.is_cuda and self.dtype == torch.bfloat16 else ops.gemm(h.float(), wg.float())
        q = sops.qk_norm_post(p[..., at["lq"]:], p[..., at["lk"]:], a.heads, a.kv_heads, self.q_norm, self.k_norm, self.eps, a.q_temp,
                              batch.positions, batch.slots, k_cache, v_cache)
        o = sops.window_attn(q, k_cache, v_cache, batch.table, a.scale, a.window, self.slopes if a.linear_bias else None, None,
                             None if batch.tiles is None else batch.tiles[tile_rows], tile_rows, batch.lens, batch.max_len)
        left = product(o, self.w_left[:, :self.lo])
        o = sops.matrix_memory(p[..., at["q"]:], p[..., at["k"]:], p[..., at["v"]:], gates, self.gate_bias, r.gate_cap, state["S"],
                               state["n"], state["m"], batch.rows, n, self.dtype)
        y = sops.head_norm_gate(o, p[..., at["g"]:], self.norm, r.heads, self.eps)
        return [(left, self.left_out), (product(y, self.w_right[:, :self.ro]), self.right_out)]


class ParallelLayer(nn.Module):
    """Norms, mixer and feed-forward of one layer. Rows and row lengths of the matrices are padded with zeros to multiples of 8
    elements, which the GEMM's copies need."""

    def __init__(self, cfg: StackConfig, spec: StackLayerSpec, dtype, device):
        super().__init__()
        self.spec, self.d, self.dtype = spec, cfg.d_model, dtype
        d8, f = pad8(cfg.d_model), spec.mlp
        self.scan = isinstance(spec.mixer, SelectiveScanSpec)
        self.norm1 = param((cfg.d_model,), F32, device)
        self.mixer = (ScanMixer if self.scan else BranchMixer)(spec.mixer, cfg.d_model, cfg.norm_eps, dtype, device)
        self.ff_at = self.mixer.cols if self.scan else 0      # where the feed-forward's columns of the output product begin
        cols = self.ff_at + (pad8(f.ff) if f is not None else 0)
        self.w_out = param((d8, cols), dtype, device) if cols else None
        self.norm2 = self.w_gate_up = None
        if f is not None:
            self.norm2 = param((cfg.d_model,), F32, device)
            self.w_gate_up = param((2 * pad8(f.ff), d8), dtype, device)

    def finish(self) -> None:
        """Values derived from the weights (after loading or drawing them)."""
        self.mixer.finish()

    def checkpoint_views(self, prefix: str) -> Dict[str, object]:
        """Checkpoint tensor name -> the part of this layer's storage that holds it (a tuple: parts stacked along the rows)."""
        out: Dict[str, object] = {prefix + "norm1": self.norm1}
        out.update({f"{prefix}mix.{k}": v for k, v in self.mixer.views(self.w_out)})
        if self.norm2 is not None:
            ff, f8 = self.spec.mlp.ff, pad8(self.spec.mlp.ff)
            out[prefix + "norm2"] = self.norm2
            out[prefix + "mlp.gate"], out[prefix + "mlp.up"] = self.w_gate_up[:ff, :self.d], self.w_gate_up[f8:f8 + ff, :self.d]
            out[prefix + "mlp.down"] = self.w_out[:self.d, self.ff_at:self.ff_at + ff]
        return out

    def forward(self, h1: torch.Tensor, h2: Optional[torch.Tensor], batch, cache, li: int, tile_rows: int):
        """Normed rows -> (branches with their norm weights, plain sum) for the residual stream."""
        n = h1.shape[0]
        act = None
        if self.w_out is not None:
            act = torch.empty(n, self.w_out.shape[1], dtype=self.dtype, device=h1.device)
        branches = []
        if self.scan:
            self.mixer(h1, batch, cache.state[li], act)
        else:
            branches = self.mixer(h1, batch, cache.k[li], cache.v[li], cache.state[li], tile_rows)
        if h2 is not None:
            ops.gemm(h2, self.w_gate_up[:, :self.d], epi=ops.EPI_SWIGLU, out=act[:, self.ff_at:])
        return branches, None if act is None else product(act, self.w_out)
