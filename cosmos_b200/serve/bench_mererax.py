"""Throughput and kernel times of Mererax layers (models/stack_parallel.py) beside the Reasoner's tower at equal size: the same
width, attention heads, feed-forward and number of layers. Random weights, random token ids. Run through
`bench.py --workload mererax`; timing as in bench_stack.py."""
from __future__ import annotations

from dataclasses import dataclass
from typing import Dict, List

import torch

from .. import ops
from ..config import MoTConfig, ParallelSpec, StackConfig, mererax_preset, nano_config
from ..models import rope
from ..models.mot import MoTModel
from ..models.stack import StackModel
from ..models.stack_parallel import ParallelLayer, product
from ..ops import stack as sops
from .bench_stack import pairs_seen, timed, timed_steps
from .decoder import StackDecoder, TPDecoder

VOCAB = 32000


@dataclass
class Size:
    name: str
    d: int
    heads: int
    kv: int
    layers: int      # every third one has attention and a memory
    mem_heads: int
    mem_dim: int
    mem_vdim: int
    inner: int
    state: int
    rank: int
    ff: int

    def stack(self) -> StackConfig:
        return mererax_preset(self.name, self.d, self.layers, self.heads, self.kv, 128, self.mem_heads, self.mem_dim, self.mem_vdim, self.inner,
                              self.state, self.rank, self.ff, VOCAB)

    def tower(self) -> MoTConfig:
        return nano_config(name="tower", d_model=self.d, n_layers=self.layers, n_heads=self.heads, n_kv_heads=self.kv, ffn_dim=self.ff,
                           vocab_size=VOCAB)


SIZES = [Size("d4096", 4096, 32, 8, 6, 8, 256, 512, 8192, 16, 256, 12288),
         Size("d2048", 2048, 16, 4, 6, 4, 256, 512, 4096, 16, 128, 6144)]
SFU_PER_S = 148 * 16 * 1.9e9     # exponentials a second: 16 a clock and SM


def kernels(sz: Size, n: int, batch: int, ctx: int, tflops: float, gbs: float) -> List[Dict]:
    """Kernel by kernel at one layer's shapes: milliseconds and the share of the roofline, with the tower's like kernel."""
    dev, bf = "cuda", torch.bfloat16
    flush = torch.empty(256 << 20, dtype=torch.uint8, device=dev)
    rows: List[Dict] = []

    def rnd(*s, scale=0.05):
        return torch.randn(*s, device=dev, dtype=torch.float32).mul_(scale).to(bf)

    def add(what, fn, flops=0.0, nbytes=0.0, like=None, exps=0.0):
        ms = timed(fn, flush)
        floor = max(flops / (tflops * 1e12), nbytes / (gbs * 1e9), exps / SFU_PER_S) * 1e3
        rows.append({"kernel": what, "ms": round(ms, 4), "roofline": round(floor / ms, 3), **({"like": like} if like else {})})
        return rows[-1]["roofline"]

    cfg = sz.stack()
    scan = ParallelLayer(cfg, cfg.layers[0], bf, dev)
    par = ParallelLayer(cfg, cfg.layers[2], bf, dev)
    for layer in (scan, par):
        for name, p in layer.named_parameters():
            p.copy_(torch.randn(p.shape, device=dev).mul_(0.02 if p.dim() > 1 else 1.0))
        layer.mixer.a_log.fill_(0.5) if layer is scan else None
        layer.finish()
    d, hq, hk, f, c, ns, rk = sz.d, sz.heads, sz.kv, sz.ff, sz.inner, sz.state, sz.rank
    H, dim, vdim = sz.mem_heads, sz.mem_dim, sz.mem_vdim
    sl, page = sops.memory_slices(vdim), 32
    g = torch.Generator(device=dev).manual_seed(0)

    def gemm_cost(m, cols, k, out=None):
        return 2.0 * m * cols * k, 2.0 * (cols * k + m * (k + (cols if out is None else out)))

    for m, label in ((n, f"prompt {n}"), (batch, f"decode batch {batch}")):
        prompt = m == n
        if prompt:
            st = sops.StepRows(torch.zeros(1, dtype=torch.int32, device=dev), portions=torch.tensor([[0, 0, n, 0]], dtype=torch.int32, device=dev),
                               conv_tiles=torch.tensor(sops.make_conv_tiles([(0, 0, n, 0)]), dtype=torch.int32, device=dev))
            seqs = 1
        else:
            st = sops.StepRows(torch.arange(m, dtype=torch.int32, device=dev), lens=torch.full((m,), ctx, dtype=torch.int32, device=dev))
            seqs = m
        h = rnd(m, d, scale=1.0)
        # ---- like kernels of the tower
        wgu, wdn, wq = rnd(2 * f, d), rnd(d, f), rnd((hq + 2 * hk) * 128, d)
        a2 = ops.gemm(h, wgu, epi=ops.EPI_SWIGLU)
        l_up = add(f"tower: SwiGLU up GEMM, {label}", lambda: ops.gemm(h, wgu, epi=ops.EPI_SWIGLU), *gemm_cost(m, 2 * f, d, f))
        l_dn = add(f"tower: down GEMM, {label}", lambda: ops.gemm(a2, wdn), *gemm_cost(m, d, f))
        l_q = add(f"tower: q/k/v GEMM, {label}", lambda: ops.gemm(h, wq), *gemm_cost(m, wq.shape[0], d))
        gam, y = torch.ones(d, device=dev, dtype=bf), rnd(m, d)
        l_n = add(f"tower: residual add + RMS norm, {label}", lambda: ops.rmsnorm(y, gam, residual=h), 0, m * d * 8.0)
        del wgu, wdn, wq
        # ---- products
        act = torch.empty(m, scan.w_out.shape[1], dtype=bf, device=dev)
        act.normal_(0, 0.1)
        add(f"SwiGLU up GEMM, {label}", lambda: ops.gemm(h, scan.w_gate_up, epi=ops.EPI_SWIGLU, out=act[:, c:]), *gemm_cost(m, 2 * f, d, f), like=l_up)
        add(f"[W_o | W_down] GEMM, {label}", lambda: product(act, scan.w_out), *gemm_cost(m, d, c + f), like=l_dn)
        mx = scan.mixer
        add(f"scan in GEMM, {label}", lambda: product(h, mx.w_in), *gemm_cost(m, 2 * c, d), like=l_q)
        xz = product(h, mx.w_in)
        state = {k: torch.zeros((seqs, *s), dtype=dt, device=dev) for k, (s, dt) in mx.state_shapes(bf).items()}
        in_bytes = xz.element_size() * (xz.shape[0] if xz.dim() == 3 else 1)
        add(f"convolution, {label}", lambda: sops.causal_conv(xz[..., :c], mx.conv_w, mx.conv_b, state["conv"], st, m), 0,
            m * c * (in_bytes + 2.0) + (0 if prompt else m * c * 3 * 4.0), l_n)
        u = sops.causal_conv(xz[..., :c], mx.conv_w, mx.conv_b, state["conv"], st, m)
        add(f"scan x GEMM, {label}", lambda: ops.gemm(u, mx.w_x), *gemm_cost(m, mx.w_x.shape[0], c), like=l_q)
        dbc = ops.gemm(u, mx.w_x)
        add(f"scan dt GEMM, {label}", lambda: ops.gemm(dbc[:, :rk], mx.w_dt[:, :rk]), *gemm_cost(m, c, rk), like=l_q)
        dt = ops.gemm(dbc[:, :rk], mx.w_dt[:, :rk])
        rows_bytes = m * (c * (6.0 + in_bytes) + 4 * ns) + (0 if prompt else m * c * ns * 8.0)
        l_mix = l_n
        add(f"selective scan, {label}", lambda: sops.selective_scan(u, dt, xz[..., c:], dbc[:, rk:], mx.dt_bias, mx.a2, mx.skip, state["S"], st, act, c),
            0, rows_bytes, l_mix, exps=float(m) * c * ns)
        # ---- attention beside a memory
        bx = par.mixer
        at = bx.at
        main = at["gates"]
        if prompt:
            add(f"branches in GEMM, {label}", lambda: ops.gemm(h, bx.w_in[:main]), *gemm_cost(m, main, d), like=l_q)
            p = ops.gemm(h, bx.w_in[:main])
            add(f"memory gates GEMM (fp32 sums), {label}", lambda: sops.gemm_partial(h, bx.w_in[main:]), 0, 2.0 * m * d, l_n)
            gates = sops.gemm_partial(h, bx.w_in[main:])
        else:
            add(f"branches in GEMM, {label}", lambda: product(h, bx.w_in), *gemm_cost(m, bx.rows, d), like=l_q)
            p = product(h, bx.w_in)
            gates = p[..., main:]
        in_bytes = p.element_size() * (p.shape[0] if p.dim() == 3 else 1)
        n_pages = m if not prompt else (n + page - 1) // page
        kc, vc = rnd(n_pages, hk, page, 128), rnd(n_pages, hk, page, 128)
        slots = torch.arange(m, device=dev) * (1 if prompt else page)
        pos = torch.arange(m, device=dev)
        add(f"q/k norm + cache write, {label}", lambda: sops.qk_norm_post(p[..., at["lq"]:], p[..., at["lk"]:], hq, hk, bx.q_norm, bx.k_norm, 1e-6,
                                                                      (0.1, 1024), pos, slots, kc, vc), 0,
            m * 128.0 * (hq * (in_bytes + 2) + hk * (in_bytes + 4)), l_n)
        state = {k: torch.zeros((seqs, *s), dtype=t, device=dev) for k, (s, t) in bx.state_shapes(bf).items()}

        def memory():
            return sops.matrix_memory(p[..., at["q"]:], p[..., at["k"]:], p[..., at["v"]:], gates, bx.gate_bias, 15.0, state["S"], state["n"],
                                      state["m"], st, m, bf)
        io = m * H * ((2 * dim + vdim) * float(in_bytes) + 2.0 * vdim)
        memory_row = len(rows)
        add(f"matrix memory, {label}", memory, 4.0 * m * H * dim * vdim if prompt else 0, io + (0 if prompt else m * H * dim * vdim * 8.0))
        o = memory()
        add(f"head norm + gate, {label}", lambda: sops.head_norm_gate(o, p[..., at["g"]:], bx.norm, H, 1e-6), 0, m * H * vdim * (4.0 + in_bytes), l_n)
        add(f"memory W_o GEMM, {label}", lambda: product(o, bx.w_right), *gemm_cost(m, d, H * vdim), like=l_dn)
        left, right, plain = product(rnd(m, hq * 128), bx.w_left), product(o, bx.w_right), product(act[:, :f].contiguous(), par.w_out)
        x, h1, h2 = torch.zeros(m, d, device=dev), torch.empty(m, d, dtype=bf, device=dev), torch.empty(m, d, dtype=bf, device=dev)
        parts = sum(float(t.numel()) * t.element_size() for t in (left, right, plain))
        add(f"three branches + residual add + two norms, {label}",
            lambda: sops.branch_norm_(x, 1e-6, bf, [(left, bx.left_out), (right, bx.right_out)], 0.5, plain, (par.norm1, par.norm2), 1.0, (h1, h2)), 0,
            m * d * 12.0 + parts, l_n)
        parts = float(plain.numel()) * plain.element_size()
        add(f"residual add + two norms, {label}", lambda: sops.branch_norm_(x, 1e-6, bf, plain=plain, gammas=(par.norm1, par.norm2), gamma_add=1.0,
                                                                      hs=(h1, h2)), 0, m * d * 12.0 + parts, l_n)
        tok = torch.randint(0, VOCAB, (m,), device=dev, generator=g)
        emb, turns = rnd(VOCAB, d), sops.sinusoid_turns(d, dev)
        add(f"embedding + position + two norms, {label}",
            lambda: sops.branch_norm_(x, 1e-6, bf, gammas=(par.norm1, par.norm2), gamma_add=1.0, hs=(h1, h2), embed=emb, tokens=tok, embed_scale=2.0,
                                      pos_turns=turns, positions=pos), 0, m * d * 10.0, l_n)
        del emb, act, a2, o, p, xz, left, right, plain
        # ---- attention
        slopes = bx.slopes
        if prompt:
            tab = torch.randperm(n_pages, device=dev).to(torch.int32)[None].contiguous()
            q, q4, k4, v4 = rnd(n, hq, 128), rnd(1, n, hq, 128), rnd(1, n, hk, 128), rnd(1, n, hk, 128)
            tiles = torch.tensor(sops.make_tiles([(0, 0, n, 0)], 256), dtype=torch.int32, device=dev)
            l_a = add(f"tower: causal attention, {label}", lambda: ops.attention(q4, k4, v4, mask=ops.MASK_CAUSAL), 4.0 * 128 * hq * pairs_seen(n, n))
            add(f"attention + linear bias, {label}", lambda: sops.window_attn(q, kc, vc, tab, 0.09, None, slopes, None, tiles, 256),
                4.0 * 128 * hq * pairs_seen(n, n), 0, l_a)
        else:
            per = (ctx + page - 1) // page
            kc, vc = rnd(m * per, hk, page, 128), rnd(m * per, hk, page, 128)
            tab = torch.randperm(m * per, device=dev).to(torch.int32).view(m, per).contiguous()
            q = rnd(m, hq, 128)
            l_a = add(f"tower: paged decode attention, {m} x {ctx}", lambda: ops.paged_decode(q, kc, vc, tab, st.lens, max_len=ctx), 0,
                      4.0 * m * ctx * hk * 128)
            add(f"decode attention + linear bias, {m} x {ctx}", lambda: sops.window_attn(q, kc, vc, tab, 0.09, None, slopes, None, seq_lens=st.lens,
                                                                                    max_len=ctx), 0, 4.0 * m * ctx * hk * 128, l_a)
        rows[memory_row]["like"] = l_a
        del kc, vc, q
    ops.check_status()
    return rows


def throughput(sz: Size, prompt: int, batches, ctx: int, steps: int, tflops: float, gbs: float) -> Dict:
    """Prefill and decode tokens/s of both models."""
    dev, bf = torch.device("cuda"), torch.bfloat16
    out: Dict = {"layers": sz.layers, "prompt": prompt, "context": ctx}
    g = torch.Generator().manual_seed(1)
    new = steps + 16
    cfg = sz.stack()
    model = StackModel(cfg, bf, dev).init_weights(0)
    ids = torch.randint(0, VOCAB, (prompt,), generator=g).tolist()
    dec = StackDecoder(model, 32, max_batch=1, max_len=prompt + 64)
    assert dec.cache.reserve(0, prompt)
    ms = timed_steps(lambda: dec.run_portions([(0, ids, 0, [prompt - 1])]), max(3, steps // 8))
    n_par = sum(isinstance(l.mixer, ParallelSpec) for l in cfg.layers)
    n_scan = sz.layers - n_par
    w_par = sz.d * ((2 * sz.heads + sz.kv) * 128 + sz.mem_heads * (2 * sz.mem_dim + 3 * sz.mem_vdim) + 3 * sz.ff)
    w_scan = sz.d * (3 * sz.inner + 3 * sz.ff) + sz.inner * (2 * sz.rank + 2 * sz.state)
    weights = float(n_par * w_par + n_scan * w_scan)
    flops = 2.0 * weights * prompt + n_par * (4.0 * 128 * sz.heads * pairs_seen(prompt, prompt) + 4.0 * prompt * sz.mem_heads * sz.mem_dim * sz.mem_vdim)
    floor = flops / (tflops * 1e12) * 1e3 + n_scan * prompt * sz.inner * sz.state / SFU_PER_S * 1e3
    out["prefill"] = {"tokens_per_s": round(prompt / ms * 1e3), "ms": round(ms, 2), "roofline": round(floor / ms, 3)}
    del dec
    state = n_scan * sz.inner * (sz.state * 4 + 6) + n_par * sz.mem_heads * sz.mem_dim * sz.mem_vdim * 4
    for b in batches:
        dec = StackDecoder(model, 32, max_batch=b, max_len=ctx + new)
        for i in range(b):      # contexts of zeros: only the traffic counts
            assert dec.cache.reserve(i, ctx + new)
        dec.seq_ids = list(range(b))
        dec.table, _ = dec.cache.tables(dec.seq_ids)
        dec.state_slots = dec.cache.state_slots(dec.seq_ids)
        dec.lens = torch.full((b,), ctx, dtype=torch.int32, device=dev)
        dec.max_len = ctx + new
        dec.tokens = torch.randint(0, VOCAB, (b,), generator=g).to(dev)
        dec.next_tokens = torch.zeros_like(dec.tokens)
        dec.capture(warmup=4)
        torch.cuda.synchronize()
        ms = timed_steps(dec.step, steps, warm=2)
        by = 2.0 * (weights + VOCAB * sz.d) + b * (2.0 * state + n_par * 4.0 * ctx * sz.kv * 128)
        out[f"decode_batch_{b}"] = {"tokens_per_s": round(b / ms * 1e3), "ms": round(ms, 4), "roofline": round(by / (gbs * 1e9) * 1e3 / ms, 3)}
        dec.graph = None
        del dec
    del model
    torch.cuda.empty_cache()
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
    lin = float(sz.layers) * sz.d * ((2 * sz.heads + 2 * sz.kv) * 128 + 3 * sz.ff)
    floor = (2.0 * lin * prompt + 4.0 * 128 * sz.heads * sz.layers * pairs_seen(prompt, prompt)) / (tflops * 1e12) * 1e3
    out["tower_prefill"] = {"tokens_per_s": round(prompt / ms * 1e3), "ms": round(ms, 2), "roofline": round(floor / ms, 3)}
    for b in batches:
        dec = TPDecoder(cfg, 1, 0, None, dev, max_batch=b, max_len=ctx + new)
        dec.load_from(tower)
        dec.prefill_synthetic(b, ctx, new)
        dec.capture(warmup=4)
        ms = timed_steps(dec.step, steps, warm=2)
        by = 2.0 * (lin + VOCAB * sz.d) + 4.0 * sz.layers * b * ctx * sz.kv * 128
        out[f"tower_decode_batch_{b}"] = {"tokens_per_s": round(b / ms * 1e3), "ms": round(ms, 4), "roofline": round(by / (gbs * 1e9) * 1e3 / ms, 3)}
        dec.graph = None
        del dec
    ops.check_status()
    return out


def run(steps: int, tflops: float, gbs: float) -> Dict:
    """All sizes: {"throughput": ..., "kernels": ...}."""
    res: Dict = {"throughput": {}, "kernels": {}}
    with torch.no_grad():
        for sz in SIZES:
            res["kernels"][sz.name] = kernels(sz, 16384, 32, 8192, tflops, gbs)
            torch.cuda.empty_cache()
            res["throughput"][sz.name] = throughput(sz, 16384, (1, 32, 128), 8192, steps, tflops, gbs)
            torch.cuda.empty_cache()
    return res
