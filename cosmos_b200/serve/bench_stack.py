"""Throughput and kernel times of a decoder stack (models/stack.py) beside the Reasoner's tower at equal size: the same
width, heads, head size and number of layers, and as many active feed-forward parameters per layer. Random weights,
random token ids. Run through `bench.py --workload stack`.

Timing: CUDA events on the launching stream. Kernels: an L2 flush before every launch, median of the launches. Prefill
and decode: warm-up, then K steps between two events (weights and activations larger than L2)."""
from __future__ import annotations

import statistics
from dataclasses import dataclass
from typing import Callable, Dict, List

import torch

from .. import ops
from ..config import MoTConfig, StackConfig, lederax_preset, nano_config
from ..models import rope
from ..models.mot import MoTModel
from ..models.stack import StackModel
from ..ops import stack as sops
from .decoder import StackDecoder, TPDecoder


@dataclass
class Size:
    name: str
    d: int
    heads: int
    kv: int
    layers: int
    experts: int
    top: int
    ff: int
    window: int

    def stack(self) -> StackConfig:
        return lederax_preset(self.name, self.d, self.layers, self.heads, self.kv, 128, self.window, self.experts, self.top,
                              self.ff, 32000)

    def tower(self) -> MoTConfig:
        return nano_config(name="tower", d_model=self.d, n_layers=self.layers, n_heads=self.heads, n_kv_heads=self.kv,
                           ffn_dim=2 * self.top * self.ff // 3, vocab_size=32000)


SIZES = [Size("d4096", 4096, 32, 8, 4, 32, 4, 4608, 4096), Size("d2048", 2048, 16, 4, 8, 16, 2, 3072, 1024)]


def timed(fn: Callable, flush: torch.Tensor, iters: int = 12, warm: int = 3) -> float:
    """Median milliseconds of one call, cold L2."""
    ev = [(torch.cuda.Event(enable_timing=True), torch.cuda.Event(enable_timing=True)) for _ in range(iters)]
    for i in range(-warm, iters):
        ops.l2_flush(flush)
        if i >= 0:
            ev[i][0].record()
        fn()
        if i >= 0:
            ev[i][1].record()
    torch.cuda.synchronize()
    return statistics.median(a.elapsed_time(b) for a, b in ev)


def timed_steps(fn: Callable, steps: int, warm: int = 3) -> float:
    for _ in range(warm):
        fn()
    a, b = torch.cuda.Event(enable_timing=True), torch.cuda.Event(enable_timing=True)
    torch.cuda.synchronize()
    a.record()
    for _ in range(steps):
        fn()
    b.record()
    torch.cuda.synchronize()
    return a.elapsed_time(b) / steps


def pairs_seen(n: int, window: int) -> int:
    """Visible (query, key) pairs of a prompt of n tokens."""
    w = min(window, n)
    return w * (w + 1) // 2 + (n - w) * w


def kernels(sz: Size, n: int, batch: int, ctx: int, tflops: float, gbs: float) -> List[Dict]:
    """Kernel by kernel at one layer's shapes: milliseconds and the share of the roofline, with the tower's like kernel."""
    dev, bf = "cuda", torch.bfloat16
    flush = torch.empty(256 << 20, dtype=torch.uint8, device=dev)
    rows: List[Dict] = []

    def rnd(*s):
        return torch.randn(*s, device=dev, dtype=torch.float32).mul_(0.05).to(bf)

    def add(what, ms, flops=0.0, nbytes=0.0, like=None):
        floor = max(flops / (tflops * 1e12), nbytes / (gbs * 1e9)) * 1e3
        rows.append({"kernel": what, "ms": round(ms, 4), "roofline": round(floor / ms, 3), **({"like": like} if like else {})})
        return rows[-1]["roofline"]

    d, hq, hk, f, e, top = sz.d, sz.heads, sz.kv, sz.ff, sz.experts, sz.top
    cols = (hq + 2 * hk) * 128
    ffd = 2 * top * f // 3
    g = torch.Generator(device=dev).manual_seed(0)

    # ---- feed-forward products of a prompt and of a decode batch
    wu, wd = rnd(e, f, d), rnd(e, d, f)
    for m, label in ((n, f"prompt {n}"), (batch, f"decode batch {batch}")):
        table = torch.rand(32000, e, device=dev, generator=g).argsort(1)[:, :top].to(torch.int32).contiguous()
        tok = torch.randint(0, 32000, (m,), device=dev, generator=g)
        tm = sops.pick_tile_m(m, top, e, bf, dev)
        desc = sops.route_desc([table], [e], [tm])
        rt = sops.moe_route(tok, 32000, [table], [e], [tm], desc)
        hit = int((torch.bincount(table[tok].reshape(-1).long(), minlength=e) > 0).sum())
        hs = rnd(m * top, d)
        ku = sops.expert_splits(m, top, e, tm, f, d)
        kd = sops.expert_splits(m, top, e, tm, d, f)
        act = sops.grouped_gemm(hs, wu, rt.tiles[0], rt.n_tiles[0], tm, True, ku)
        fl, by = 2.0 * m * top * d * f, 2.0 * (hit * f * d + m * top * (d + f))
        up = timed(lambda: sops.grouped_gemm(hs, wu, rt.tiles[0], rt.n_tiles[0], tm, True, ku), flush)
        dn = timed(lambda: sops.grouped_gemm(act, wd, rt.tiles[0], rt.n_tiles[0], tm, False, kd, kd > 1), flush)
        h, wgu, wdn = rnd(m, d), rnd(2 * ffd, d), rnd(d, ffd)
        a2 = ops.gemm(h, wgu, epi=ops.EPI_SWIGLU)
        t_up = timed(lambda: ops.gemm(h, wgu, epi=ops.EPI_SWIGLU), flush)
        t_dn = timed(lambda: ops.gemm(a2, wdn), flush)
        l_up = add(f"tower: SwiGLU up GEMM, {label}", t_up, 2.0 * m * d * 2 * ffd, 2.0 * (2 * ffd * d + m * (d + ffd)))
        l_dn = add(f"tower: down GEMM, {label}", t_dn, 2.0 * m * d * ffd, 2.0 * (ffd * d + m * (d + ffd)))
        add(f"experts up GEMM + gelu, {label}", up, fl, by, l_up)
        add(f"experts down GEMM, {label}", dn, fl, by, l_dn)
        add(f"routing of one layer, {label}", timed(lambda: sops.moe_route(tok, 32000, [table], [e], [tm], desc), flush),
            0, m * (8.0 + 8.0 * top))
        # ---- residual add + norm + dispatch; combine + residual add + norm
        x, y, gam = torch.zeros(m, d, device=dev), rnd(m, d), torch.ones(d, device=dev, dtype=bf)
        out, ys = torch.empty(m * top, d, dtype=bf, device=dev), rnd(m * top, d)
        ho = torch.empty(m, d, dtype=bf, device=dev)
        l_n = add(f"tower: residual add + RMS norm, {label}", timed(lambda: ops.rmsnorm(y, gam, residual=h), flush), 0, m * d * 8.0)
        add(f"residual add + grouped norm + dispatch to {top} rows, {label}",
            timed(lambda: sops.residual_norm_(x, gam, 2, 1e-6, out, rt.rows[0], y=y), flush), 0, m * d * (10.0 + 2 * top), l_n)
        add(f"combine of {top} rows + residual add + grouped norm, {label}",
            timed(lambda: sops.residual_norm_(x, gam, 2, 1e-6, ho, y=ys, y_rows=rt.rows[0], weight=1 / top), flush), 0,
            m * d * (10.0 + 2 * top), l_n)
        # ---- q/k/v
        wq, b = rnd(cols, d), rnd(cols)
        lq = add(f"tower: q/k/v GEMM, {label}", timed(lambda: ops.gemm(h, wq), flush), 2.0 * m * d * cols, 2.0 * (cols * d + m * (d + cols)))
        if m == n:
            add(f"q/k/v GEMM + bias, {label}", timed(lambda: ops.gemm(h, wq, b), flush), 2.0 * m * d * cols, 2.0 * (cols * d + m * (d + cols)), lq)
        else:
            add(f"q/k/v GEMM, split sums, {label}", timed(lambda: sops.gemm_partial(h, wq), flush), 0, 2.0 * (cols * d + m * (d + cols)), lq)
    del wu, wd, hs, act, out, ys

    # ---- attention of a prompt
    page = 32
    n_pages = (n + page - 1) // page
    kc, vc = rnd(n_pages, hk, page, 128), rnd(n_pages, hk, page, 128)
    tab = torch.randperm(n_pages, device=dev).to(torch.int32)[None].contiguous()
    q = rnd(n, hq, 128)
    r1, r2 = torch.rand(hq, device=dev) + 0.1, torch.rand(hq, device=dev) * 0.3 + 0.1
    tiles = torch.tensor(sops.make_tiles([(0, 0, n, 0)], 256), dtype=torch.int32, device=dev)
    k4, v4 = rnd(1, n, hk, 128), rnd(1, n, hk, 128)
    q4 = q[None]
    l_full = add(f"tower: causal attention, prompt {n}", timed(lambda: ops.attention(q4, k4, v4, mask=ops.MASK_CAUSAL), flush),
                 4.0 * 128 * hq * pairs_seen(n, n))
    for w in (n, sz.window):
        add(f"windowed attention + bias, window {w}, prompt {n}",
            timed(lambda: sops.window_attn(q, kc, vc, tab, 0.09, w, r1, r2, tiles, 256), flush),
            4.0 * 128 * hq * pairs_seen(n, w), 0, l_full)
    qkv = rnd(n, cols)
    slots = torch.arange(n, device=dev)
    first = torch.randn(n, hk, 128, device=dev)
    lam = torch.tensor(0.4, device=dev)
    l_kv = add(f"tower: cache write, prompt {n}", timed(lambda: torch.ops.cosmos_b200.kv_cache_write(k4[0], v4[0], slots, kc, vc), flush),
               0, n * hk * 128 * 8.0)
    add(f"value norm + mixing + cache write, prompt {n}",
        timed(lambda: sops.qkv_value_post(qkv, None, hq, hk, 1e-6, True, slots, kc, vc, None, first, lam), flush), 0,
        n * hk * 128 * 12.0, l_kv)
    del kc, vc, q, k4, v4, q4, qkv, first

    # ---- attention of a decode step
    for c in sorted({min(ctx, sz.window), ctx}):
        per = (c + page - 1) // page
        kc, vc = rnd(batch * per, hk, page, 128), rnd(batch * per, hk, page, 128)
        tab = torch.randperm(batch * per, device=dev).to(torch.int32).view(batch, per).contiguous()
        lens = torch.full((batch,), c, dtype=torch.int32, device=dev)
        q = rnd(batch, hq, 128)
        l_d = add(f"tower: paged decode attention, {batch} x {c}", timed(lambda: ops.paged_decode(q, kc, vc, tab, lens, max_len=c), flush),
                  0, 4.0 * batch * c * hk * 128)
        seen = min(c, sz.window)
        add(f"windowed decode attention + bias, {batch} x {c}, window {sz.window}",
            timed(lambda: sops.window_attn(q, kc, vc, tab, 0.09, sz.window, r1, r2, seq_lens=lens, max_len=c), flush), 0,
            4.0 * batch * seen * hk * 128, l_d)
        del kc, vc
    ops.check_status()
    return rows


def throughput(sz: Size, prompt: int, batches, ctx: int, steps: int, tflops: float, gbs: float) -> Dict:
    """Prefill and decode tokens/s of both models."""
    dev, bf = torch.device("cuda"), torch.bfloat16
    out: Dict = {"layers": sz.layers, "prompt": prompt, "context": ctx, "window": sz.window, "experts": sz.experts, "top": sz.top}
    g = torch.Generator().manual_seed(1)
    new = steps + 16
    model = StackModel(sz.stack(), bf, dev).init_weights(0)
    ids = torch.randint(0, 32000, (prompt,), generator=g).tolist()
    dec = StackDecoder(model, 32, max_batch=1, max_len=prompt + 64)
    assert dec.cache.reserve(0, prompt)
    ms = timed_steps(lambda: dec.run_portions([(0, ids, 0, [prompt - 1])]), max(3, steps // 8))
    d, f = sz.d, sz.ff
    lin = 2.0 * d * ((sz.heads + 2 * sz.kv) * 128 + sz.heads * 128 + 2 * sz.top * f) * sz.layers
    floor = (lin * prompt + 4.0 * 128 * sz.heads * sz.layers * pairs_seen(prompt, sz.window)) / (tflops * 1e12) * 1e3
    out["prefill"] = {"tokens_per_s": round(prompt / ms * 1e3), "ms": round(ms, 2), "roofline": round(floor / ms, 3)}
    del dec
    for b in batches:
        dec = StackDecoder(model, 32, max_batch=b, max_len=ctx + new)
        part = ids[:min(ctx, prompt)]
        dec.start_batch([part] * b, new)
        dec.tokens.copy_(torch.randint(0, 32000, (b,), generator=g).to(dev))
        dec.step_inc = None
        dec.capture(warmup=4)
        torch.cuda.synchronize()
        ms = timed_steps(dec.step, steps, warm=2)
        hit = min(sz.experts, b * sz.top) if b > 1 else sz.top
        hit = sz.experts * (1 - (1 - sz.top / sz.experts) ** b)     # expected number of experts a batch touches
        by = sz.layers * 2.0 * (d * ((sz.heads * 2 + 2 * sz.kv) * 128) + 2 * hit * d * f
                                + 2 * b * min(ctx, sz.window) * sz.kv * 128) + 2.0 * 32000 * d
        out[f"decode_batch_{b}"] = {"tokens_per_s": round(b / ms * 1e3), "ms": round(ms, 4),
                                    "roofline": round(by / (gbs * 1e9) * 1e3 / ms, 3)}
        dec.graph = None
        del dec
    del model
    torch.cuda.empty_cache()
    # the Reasoner's tower
    cfg = sz.tower()
    tower = MoTModel(cfg, dtype=bf, device=dev, towers=("ar",))
    tower.init_weights(seed=0)
    tok = torch.tensor([ids], device=dev)
    pos = rope.text_positions(prompt, 0, dev)

    def prefill():
        with torch.no_grad():
            h, _ = tower.ar_forward(tower.embed_tokens(tok), pos)
            tower.lm_logits(h[:, -1:])

    ms = timed_steps(prefill, max(3, steps // 8))
    floor = (lin * prompt + 4.0 * 128 * sz.heads * sz.layers * pairs_seen(prompt, prompt)) / (tflops * 1e12) * 1e3
    out["tower_prefill"] = {"tokens_per_s": round(prompt / ms * 1e3), "ms": round(ms, 2), "roofline": round(floor / ms, 3)}
    for b in batches:
        dec = TPDecoder(cfg, 1, 0, None, dev, max_batch=b, max_len=ctx + new)
        dec.load_from(tower)
        dec.prefill_synthetic(b, ctx, new)
        dec.capture(warmup=4)
        ms = timed_steps(dec.step, steps, warm=2)
        by = sz.layers * 2.0 * (d * ((sz.heads * 2 + 2 * sz.kv) * 128) + 3 * d * cfg.ffn_dim + 2 * b * ctx * sz.kv * 128) + 2.0 * 32000 * d
        out[f"tower_decode_batch_{b}"] = {"tokens_per_s": round(b / ms * 1e3), "ms": round(ms, 4),
                                          "roofline": round(by / (gbs * 1e9) * 1e3 / ms, 3)}
        dec.graph = None
        del dec
    ops.check_status()
    return out


def run(steps: int, tflops: float, gbs: float, sampler=None) -> Dict:
    """All sizes: {"throughput": ..., "kernels": ...} and the clocks seen meanwhile."""
    res: Dict = {"throughput": {}, "kernels": {}}
    for sz in SIZES:
        res["throughput"][sz.name] = throughput(sz, 16384, (1, 32, 128), 8192, steps, tflops, gbs)
        torch.cuda.empty_cache()
        res["kernels"][sz.name] = kernels(sz, 16384, 32, 8192, tflops, gbs)
        torch.cuda.empty_cache()
    return res
