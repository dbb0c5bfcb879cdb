"""Decoder-only language models whose layers are declared one by one in their configuration (config.StackConfig): each
layer names its attention mechanisms (window, distance bias, value norm, value mixing, biases) and its feed-forward
(table-routed experts or none). The residual stream is fp32; matrix products run in the model's dtype.

`StackModel.forward_step` is the one forward pass of such a model: it runs the tokens that a step brings (portions of
prompts of several sequences, or one new token of every decode slot) against the paged cache. Prefill, decoding and the
trace runner all go through it. Launches per layer on CUDA bf16:
  q/k/v GEMM (+ bias) -> value norm + mixing + cache write -> paged windowed attention -> out-projection GEMM
  -> residual add + norm + dispatch into expert order -> up GEMM (+ gelu) -> down GEMM -> combine + residual add + norm
(layers in serial order; those in parallel order, with recurrent mixers, are in stack_parallel.py). For a few rows (decode) the GEMMs split K and leave fp32 partial sums that the kernel behind each of them reduces. The
experts depend on the token ids alone, so one launch at the start of the step routes every layer.
"""
from __future__ import annotations

from dataclasses import dataclass
from pathlib import Path
from typing import Dict, List, Optional, Tuple

import torch
import torch.nn as nn

from .. import ops
from ..config import MODEL_REGISTRY, AttentionSpec, StackConfig, StackLayerSpec, get_model_config, stack_config_from_dir
from ..ops import stack as sops
from ..ops.stack import StepRows, pad8
from .stack_parallel import ParallelLayer, split_k
from .stack_parallel import param as _param


@dataclass
class StepBatch:
    """The tokens of one step, in row order, and where they go. Portions: `tiles` [t, 4] int32 lists the query tiles.
    Decode: `lens` [n] int32 holds every slot's length including its new token (0 = idle slot). `rows`: the same for
    recurrent layers."""
    tokens: torch.Tensor                 # [n] int64
    slots: torch.Tensor                  # [n] int64 cache slots (page * page_size + offset)
    table: torch.Tensor                  # [sequences, max_pages] int32
    tiles: Optional[Dict[int, torch.Tensor]] = None   # query tiles by rows per tile
    lens: Optional[torch.Tensor] = None
    max_len: Optional[int] = None        # host-known bound of `lens`
    positions: Optional[torch.Tensor] = None          # [n] int64
    rows: Optional[StepRows] = None


class StackLayer(nn.Module):
    """Weights of one layer. Rows and row lengths of the matrices are padded with zeros to multiples of 8 elements, which
    the GEMM's copies need; the products never read the padding columns and the padding rows give zeros."""

    def __init__(self, cfg: StackConfig, spec: StackLayerSpec, dtype, device):
        super().__init__()
        self.spec = spec
        d, d8, m = cfg.d_model, pad8(cfg.d_model), spec.mixer
        self.d = d
        self.norm1 = _param((d,), dtype, device)
        self.w_qkv = _param((pad8(m.qkv_cols), d8), dtype, device)
        self.b_qkv = _param((pad8(m.qkv_cols),), dtype, device) if m.qkv_bias else None
        self.o_cols = m.heads * m.vdim
        self.w_o = _param((d8, pad8(self.o_cols)), dtype, device)
        if m.distance_bias:
            self.r1 = _param((m.heads,), torch.float32, device)
            self.r2 = _param((m.heads,), torch.float32, device)
        else:
            self.r1 = self.r2 = None
        self.vmix = _param((), torch.float32, device) if m.value_mix else None
        f = spec.mlp
        if f is not None:
            self.norm2 = _param((d,), dtype, device)
            self.w_up = _param((f.experts, pad8(f.ff), d8), dtype, device)
            self.w_down = _param((f.experts, d8, pad8(f.ff)), dtype, device)
            self.table = nn.Parameter(torch.zeros(cfg.vocab_size, f.top, dtype=torch.int32, device=device),
                                      requires_grad=False)

    def checkpoint_views(self, prefix: str) -> Dict[str, torch.Tensor]:
        """Checkpoint tensor name -> the part of this layer's storage that holds it."""
        m, d, out = self.spec.mixer, self.d, {}
        out[prefix + "norm1"] = self.norm1
        row = 0
        for name, rows in (("q", m.heads * m.dim), ("k", m.kv_heads * m.dim), ("v", m.kv_heads * m.vdim)):
            out[f"{prefix}mix.{name}"] = self.w_qkv[row:row + rows, :d]
            if self.b_qkv is not None:
                out[f"{prefix}mix.{name}.b"] = self.b_qkv[row:row + rows]
            row += rows
        if self.vmix is not None:
            out[prefix + "mix.vmix"] = self.vmix
        if self.r1 is not None:
            out[prefix + "mix.r1"], out[prefix + "mix.r2"] = self.r1, self.r2
        out[prefix + "mix.o"] = self.w_o[:d, :self.o_cols]
        f = self.spec.mlp
        if f is not None:
            out[prefix + "norm2"] = self.norm2
            for e in range(f.experts):
                out[f"{prefix}mlp.e{e}.up"] = self.w_up[e, :f.ff, :d]
                out[f"{prefix}mlp.e{e}.down"] = self.w_down[e, :d, :f.ff]
            out[prefix + "mlp.table"] = self.table
        return out


class StackModel(nn.Module):
    def __init__(self, cfg: StackConfig, dtype=torch.bfloat16, device="cpu"):
        super().__init__()
        self.cfg, self.dtype = cfg, dtype
        d8, v8 = pad8(cfg.d_model), pad8(cfg.vocab_size)
        self.parallel = cfg.order == "parallel"
        # a tied head is the embedding table itself, stored with the padding that the head's product needs
        self.w_head = _param((v8, d8), dtype, device)
        self.embed = self.w_head[:cfg.vocab_size, :cfg.d_model] if cfg.tied_head else _param((cfg.vocab_size, cfg.d_model), dtype, device)
        kind = ParallelLayer if self.parallel else StackLayer
        own = {i: kind(cfg, s, dtype, device) for i, s in enumerate(cfg.layers) if s.weights_of is None}
        self.layers = nn.ModuleList([own[cfg.source_layer(i)] for i in range(cfg.n_layers)])
        self.final_norm = _param((cfg.d_model,), torch.float32 if self.parallel else dtype, device)
        self._moe = [] if self.parallel else [i for i, s in enumerate(cfg.layers) if s.mlp is not None]
        self._desc: Dict[Tuple, torch.Tensor] = {}
        mixing = [i for i, s in enumerate(cfg.layers) if isinstance(s.mixer, AttentionSpec) and s.mixer.value_mix]
        self.first_mix = mixing[0] if mixing else -1
        self.pos_turns = sops.sinusoid_turns(cfg.d_model, device) if cfg.sinusoid else None

    @property
    def device(self) -> torch.device:
        return self.w_head.device

    # ------------------------------------------------------------------ weights
    def checkpoint_views(self) -> Dict[str, object]:
        """Checkpoint tensor name -> the storage that holds it (a tuple: parts stacked along the rows)."""
        out: Dict[str, object] = {"embed": self.embed, "final.norm": self.final_norm}
        if not self.cfg.tied_head:
            out["head"] = self.w_head[:self.cfg.vocab_size, :self.cfg.d_model]
        for i, layer in enumerate(self.layers):
            if self.cfg.layers[i].weights_of is None:
                out.update(layer.checkpoint_views(f"l{i}."))
        return out

    def finish(self) -> "StackModel":
        """Values derived from the weights (after loading or drawing them)."""
        if self.parallel:
            for layer in self.layers:
                layer.finish()
        return self

    @torch.no_grad()
    def load(self, model_dir) -> "StackModel":
        from ..ckpt import safetensors_io as sio

        views = self.checkpoint_views()
        stacked = {k: v for k, v in views.items() if isinstance(v, tuple)}
        targets = {k: v.data for k, v in views.items() if k not in stacked}
        for k, parts in stacked.items():
            targets[k] = torch.empty(sum(p.shape[0] for p in parts), *parts[0].shape[1:], dtype=parts[0].dtype, device=parts[0].device)
        unused = f"l{self.first_mix}.mix.vmix"   # the first mixing layer has nothing to mix with
        if unused in targets and unused not in sio.tensor_files(model_dir):
            del targets[unused]
        sio.load_into(model_dir, targets)
        for k, parts in stacked.items():
            for p, src in zip(parts, targets[k].split([p.shape[0] for p in parts])):
                p.copy_(src)
        return self.check_tables().finish()

    def check_tables(self) -> "StackModel":
        for i in self._moe:
            t = self.layers[i].table
            if int(t.min()) < 0 or int(t.max()) >= self.cfg.layers[i].mlp.experts:
                raise ValueError(f"layer {i}: the routing table names experts that do not exist")
        return self

    @torch.no_grad()
    def save(self, model_dir) -> None:
        import json

        from ..ckpt import safetensors_io as sio

        whole = {k: torch.cat(v) if isinstance(v, tuple) else v for k, v in self.checkpoint_views().items()}
        half = {k: v.detach().to(torch.bfloat16) if v.is_floating_point() else v for k, v in whole.items()}
        sio.save_sharded(half, model_dir)
        (Path(model_dir) / "config.json").write_text(json.dumps(self.cfg.to_dict(), indent=1))

    @torch.no_grad()
    def init_weights(self, seed: int = 0) -> "StackModel":
        """Random weights: N(0, init_std) matrices, neutral norms, mild biases, random routing tables without repeats in a row,
        decays and step sizes over the usual range of selective scans, forget gates mostly open."""
        dev, std = self.device, self.cfg.init_std
        g = torch.Generator(device=dev)
        g.manual_seed(seed)

        def rand(v, lo, hi):
            return torch.rand(v.shape, generator=g, device=dev) * (hi - lo) + lo

        views = [(name, v) for name, vs in self.checkpoint_views().items() for v in (vs if isinstance(vs, tuple) else (vs,))]
        for name, v in views:
            leaf = name.split(".")[-1]
            if leaf in ("norm1", "norm2") or name == "final.norm":
                v.fill_(1.0 - self.cfg.norm_add)
            elif leaf in ("norm", "out") or leaf == "D":
                v.fill_(1.0)
            elif leaf == "table":
                e = self.cfg.layers[int(name[1:name.index(".")])].mlp.experts
                v.copy_(torch.rand(v.shape[0], e, generator=g, device=dev).argsort(1)[:, :v.shape[1]].to(torch.int32))
            elif leaf in ("r1", "r2"):
                v.copy_(rand(v, 0.05, 0.55))
            elif leaf == "vmix":
                v.fill_(0.5)
            elif leaf == "A_log":
                v.copy_(torch.arange(1, v.shape[1] + 1, device=dev).float().log().expand_as(v))
            elif name.endswith("mix.dt.b"):    # softplus of it between 0.001 and 0.1
                v.copy_(torch.expm1(torch.exp(rand(v, -6.9, -2.3))).log())
            elif name.endswith("right.f.b"):
                v.copy_(rand(v, 3.0, 6.0))
            elif leaf == "conv":
                v.copy_(rand(v, -0.5, 0.5))
            else:
                v.copy_(torch.randn(v.shape, generator=g, device=dev, dtype=torch.float32) * std)
        return self.finish()

    def kv_shapes(self) -> List[Tuple[int, int, int]]:
        """(kv heads, key size, value size) of every layer; no heads = a layer without attention."""
        att = [s.attention for s in self.cfg.layers]
        return [(0, 0, 0) if a is None else (a.kv_heads, a.dim, a.vdim) for a in att]

    def state_shapes(self) -> List[Dict[str, Tuple]]:
        """Per layer: name -> (shape, dtype) of what a sequence carries from token to token beside the paged cache."""
        return [layer.mixer.state_shapes(self.dtype) for layer in self.layers] if self.parallel else []

    def tile_sizes(self, page_size: int) -> List[int]:
        """Query rows per attention tile of every layer (which kernel takes its shape); 0 = no attention."""
        att = [s.attention for s in self.cfg.layers]
        return [0 if a is None else sops.attn_tile_rows(a.heads, a.kv_heads, a.dim, a.vdim, page_size, self.dtype, self.device)
                for a in att]

    # ------------------------------------------------------------------ the step
    def _route(self, tokens: torch.Tensor) -> Optional[sops.Routing]:
        if not self._moe:
            return None
        specs = [self.cfg.layers[i].mlp for i in self._moe]
        tables = [self.layers[i].table for i in self._moe]
        n = tokens.shape[0]
        tile_m = [sops.pick_tile_m(n, f.top, f.experts, self.dtype, self.device) for f in specs]
        experts = [f.experts for f in specs]
        desc = None
        if tokens.is_cuda:
            key = tuple(tile_m) + tuple(t.data_ptr() for t in tables)
            if key not in self._desc:
                self._desc[key] = sops.route_desc(tables, experts, tile_m)
            desc = self._desc[key]
        return sops.moe_route(tokens, self.cfg.vocab_size, tables, experts, tile_m, desc)

    def _attention(self, li: int, h: torch.Tensor, batch: StepBatch, cache, tile_rows: int, v_first: Dict) -> torch.Tensor:
        """Mixer of layer li on the normed rows h [n, d]: -> y [n, >= d] (or fp32 partial sums)."""
        layer, m, n = self.layers[li], self.cfg.layers[li].mixer, h.shape[0]
        w = layer.w_qkv[:, :layer.d]
        if split_k(n, w):
            qkv = sops.gemm_partial(h, w)
        else:
            qkv = ops.gemm(h, w, layer.b_qkv)
        first_in = first_out = None
        if m.value_mix:
            if li == self.first_mix:
                first_out = v_first["v"] = torch.empty(n, m.kv_heads, m.vdim, dtype=torch.float32, device=h.device)
            else:
                first_in = v_first["v"]
        q = sops.qkv_value_post(qkv, layer.b_qkv, m.heads, m.kv_heads, self.cfg.norm_eps, m.value_norm, batch.slots,
                                cache.k[li], cache.v[li], first_out, first_in, layer.vmix)
        o = sops.window_attn(q, cache.k[li], cache.v[li], batch.table, m.scale, m.window, layer.r1, layer.r2,
                             None if batch.tiles is None else batch.tiles[tile_rows], tile_rows, batch.lens, batch.max_len)
        w = layer.w_o[:, :layer.o_cols]
        return sops.gemm_partial(o, w) if split_k(n, w) else ops.gemm(o, w)

    def _experts(self, li: int, hs: torch.Tensor, rt: sops.Routing, k: int, n: int) -> torch.Tensor:
        """Feed-forward of layer li on the dispatched rows hs [n * top, d]: -> the experts' outputs in the same order."""
        layer, f = self.layers[li], self.cfg.layers[li].mlp
        tiles, cnt, tm = rt.tiles[k], rt.n_tiles[k], rt.tile_m[k]
        up, down = layer.w_up[:, :, :layer.d], layer.w_down
        split = self.dtype == torch.bfloat16 and hs.is_cuda
        ks = sops.expert_splits(n, f.top, f.experts, tm, up.shape[1], up.shape[2]) if split else 1
        a = sops.grouped_gemm(hs, up, tiles, cnt, tm, gelu=True, k_splits=ks)
        ks = sops.expert_splits(n, f.top, f.experts, tm, down.shape[1], down.shape[2]) if split else 1
        return sops.grouped_gemm(a, down, tiles, cnt, tm, k_splits=ks, partial=ks > 1)

    @torch.no_grad()
    def forward_step(self, batch: StepBatch, cache, tile_sizes: List[int], rows: Optional[torch.Tensor] = None,
                     layers_out: Optional[List[torch.Tensor]] = None) -> torch.Tensor:
        """Logits [len(rows), vocab] of the chosen rows (None = all). `layers_out` receives the residual stream after every
        layer (debugging)."""
        if self.parallel:
            return self._parallel_step(batch, cache, tile_sizes, rows, layers_out)
        cfg, dev, dt = self.cfg, self.device, self.dtype
        n, d, g, eps = batch.tokens.shape[0], cfg.d_model, cfg.norm_groups, cfg.norm_eps
        x = torch.empty(n, d, dtype=torch.float32, device=dev)
        h = torch.empty(n, pad8(d), dtype=dt, device=dev)
        rt = self._route(batch.tokens)
        gammas = [l.norm1 for l in self.layers] + [self.final_norm]
        sops.residual_norm_(x, gammas[0], g, eps, h, embed=self.embed, tokens=batch.tokens, embed_scale=cfg.embed_scale)
        v_first: Dict[str, torch.Tensor] = {}
        k = 0
        for li, spec in enumerate(cfg.layers):
            y, y_rows, weight = self._attention(li, h[:, :d], batch, cache, tile_sizes[li], v_first), None, 1.0
            if spec.mlp is not None:
                top = spec.mlp.top
                hs = torch.empty(n * top, pad8(d), dtype=dt, device=dev)
                sops.residual_norm_(x, self.layers[li].norm2, g, eps, hs, rt.rows[k], y=y, y_rows=y_rows, weight=weight)
                y, y_rows, weight = self._experts(li, hs[:, :d], rt, k, n), rt.rows[k], 1.0 / top
                k += 1
            last = li + 1 == cfg.n_layers
            if last and rows is not None:   # only the asked rows need the final norm and the head
                sops.residual_norm_(x, None, g, eps, y=y, y_rows=y_rows, weight=weight)
            else:
                sops.residual_norm_(x, gammas[li + 1], g, eps, h, y=y, y_rows=y_rows, weight=weight)
            if layers_out is not None:
                layers_out.append(x.clone())
        if rows is not None:
            if rows.shape[0] == 0:   # a portion in the middle of a prompt
                return torch.empty(0, cfg.vocab_size, dtype=dt, device=dev)
            xr = x[rows]
            h = torch.empty(xr.shape[0], pad8(d), dtype=dt, device=dev)
            sops.residual_norm_(xr, self.final_norm, g, eps, h)
        return ops.gemm(h[:, :d], self.w_head[:, :d])[:, :cfg.vocab_size]

    def _parallel_step(self, batch: StepBatch, cache, tile_sizes: List[int], rows: Optional[torch.Tensor],
                       layers_out: Optional[List[torch.Tensor]]) -> torch.Tensor:
        cfg, dev, dt = self.cfg, self.device, self.dtype
        n, d, eps, add = batch.tokens.shape[0], cfg.d_model, cfg.norm_eps, cfg.norm_add

        def buffer(m: int = n) -> torch.Tensor:
            return torch.empty(m, pad8(d), dtype=dt, device=dev)

        x = torch.empty(n, d, dtype=torch.float32, device=dev)
        first = dict(embed=self.embed, tokens=batch.tokens, embed_scale=cfg.embed_scale, pos_turns=self.pos_turns, positions=batch.positions)
        branches, plain = [], None
        for li, layer in enumerate(self.layers):
            h1, h2 = buffer(), None if layer.norm2 is None else buffer()
            sops.branch_norm_(x, eps, dt, branches, 0.5, plain, (layer.norm1, layer.norm2), add, (h1, h2), **first)
            first = {}
            if li > 0 and layers_out is not None:
                layers_out.append(x.clone())
            branches, plain = layer(h1[:, :d], None if h2 is None else h2[:, :d], batch, cache, li, tile_sizes[li])
        h = None
        if rows is None:
            h = buffer()
            sops.branch_norm_(x, eps, dt, branches, 0.5, plain, (self.final_norm,), add, (h,), **first)
        else:           # only the asked rows need the final norm and the head
            sops.branch_norm_(x, eps, dt, branches, 0.5, plain, **first)
            if rows.shape[0] > 0:
                h = buffer(rows.shape[0])
                sops.branch_norm_(x[rows], eps, dt, gammas=(self.final_norm,), gamma_add=add, hs=(h,))
        if layers_out is not None and cfg.n_layers > 0:
            layers_out.append(x.clone())
        if h is None:   # a portion in the middle of a prompt
            return torch.empty(0, cfg.vocab_size, dtype=dt, device=dev)
        return ops.gemm(h[:, :d], self.w_head[:, :d])[:, :cfg.vocab_size]


def is_stack_name(name_or_path) -> bool:
    """Whether a registered name or a checkpoint directory is a decoder stack."""
    if Path(name_or_path).is_dir():
        return stack_config_from_dir(name_or_path) is not None
    return name_or_path in MODEL_REGISTRY and isinstance(get_model_config(name_or_path), StackConfig)


def load_stack(name_or_path, dtype=torch.bfloat16, device="cpu", seed: int = 0, **overrides) -> StackModel:
    """A checkpoint directory (config.json + safetensors) or a registered name (random weights)."""
    if Path(name_or_path).is_dir():
        cfg = stack_config_from_dir(name_or_path)
        if cfg is None:
            raise ValueError(f"{name_or_path}: config.json names no decoder-stack architecture")
        return StackModel(cfg, dtype, device).load(name_or_path)
    return StackModel(get_model_config(str(name_or_path), **overrides), dtype, device).init_weights(seed)
