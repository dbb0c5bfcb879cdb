"""Mererax on a GPU (kernels in fp32 and bf16): the serving decoder against the plain implementation, and every kernel of its
mechanisms against the plain functions of oracle_mererax.py in float64."""
import pytest
import torch

from cosmos_b200 import ops
from cosmos_b200.ops import stack as sops
from tests import oracle_mererax as orc
from tests import stack_cases as cases
from tests import stack_checks as checks

pytestmark = pytest.mark.gpu
F32, BF16 = torch.float32, torch.bfloat16
DEV = "cuda"
TOL = {F32: 3e-5, BF16: 9e-2}     # bf16: rounding of weights' products and activations through peaky layers
KTOL = {F32: 4e-6, BF16: 8e-3}
FAM = checks.MERERAX


@pytest.fixture(autouse=True)
def _status_clean():
    assert ops.load_extension()
    torch.backends.cuda.matmul.allow_tf32 = False
    yield
    torch.cuda.synchronize()
    ops.check_status()


def _gen(seed=0):
    return torch.Generator().manual_seed(seed)


def _close(got, want, tol, what=""):
    got, want = got.double().cpu(), want.double().cpu()
    err = (got - want).abs().max().item()
    scale = max(1.0, want.abs().max().item())
    assert err <= tol * scale, f"{what}: max error {err:.3g} at scale {scale:.3g}"


# --------------------------------------------------------------------------- the decoder
@pytest.mark.parametrize("dtype", [F32, BF16])
@pytest.mark.parametrize("name", sorted(FAM.cases.CONFIGS))
def test_whole_prompt_and_residual_stream(tmp_path, name, dtype):
    checks.whole_prompt_and_layers(tmp_path, name, dtype, DEV, TOL[dtype], page_size=8, fam=FAM)


@pytest.mark.parametrize("dtype", [F32, BF16])
@pytest.mark.parametrize("name,page,n", [("mixed", 5, 61), ("bare", 8, 61), ("chain", 16, 61), ("tc", 8, 150), ("tc", 32, 150), ("wide", 16, 90)])
def test_portions_equal_the_whole_prompt(tmp_path, name, page, n, dtype):
    checks.portions_and_token_by_token(tmp_path, name, dtype, DEV, TOL[dtype], n=n, page_size=page, fam=FAM)


@pytest.mark.parametrize("dtype", [F32, BF16])
@pytest.mark.parametrize("name", ["mixed", "bare", "tc", "wide"])
def test_batches_of_unequal_requests_equal_each_alone(tmp_path, name, dtype):
    checks.mixed_batches(tmp_path, name, dtype, DEV, TOL[dtype], page_size=16, fam=FAM)


@pytest.mark.parametrize("dtype,slack", [(F32, 1e-4), (BF16, 0.2)])
@pytest.mark.parametrize("name,graph", [("mixed", True), ("tc", True), ("tc", False), ("wide", True)])
def test_greedy_generation_through_the_engine(tmp_path, name, graph, dtype, slack):
    checks.greedy_generation(tmp_path, name, dtype, DEV, slack, graph, page_size=8, fam=FAM)


@pytest.mark.parametrize("dtype", [F32, BF16])
def test_long_decoding_and_far_tokens(tmp_path, dtype):
    """330 tokens, most of them decoded one by one, over many pages, memory tiles and temperature steps."""
    cfg, t, dec = checks.setup(tmp_path, "tc", dtype, DEV, page_size=16, fam=FAM)
    ids = cases.tokens(cfg, 330, 8)
    want = orc.forward(cfg, t, ids)
    for k, cuts in enumerate(([30] + [1] * 300, [330], [257, 1, 72], [2, 63, 64, 65])):
        e = cases.error(cases.feed(dec, k, ids, cuts), want)
        assert e < TOL[dtype], f"{cuts[:3]}: {e:.3g}"
        dec.cache.release(k)


def test_results_do_not_depend_on_pages_and_states_left_by_others(tmp_path):
    """The same request on fresh pages and slots, and on ones that others have used: bit-equal logits per path."""
    cfg, t, dec = checks.setup(tmp_path, "tc", BF16, DEV, page_size=8, fam=FAM)
    ids = cases.tokens(cfg, 90, 1)
    cuts = [33, 1, 2, 40, 1, 1, 12]
    first = cases.feed(dec, 0, ids, cuts)
    for k in range(1, 4):
        cases.feed(dec, k, cases.tokens(cfg, 90, k), [41])
    slot = dec.cache.states.slot_of[2]
    dec.cache.release(0)
    dec.cache.release(2)
    again = cases.feed(dec, 9, ids, cuts)
    assert dec.cache.states.slot_of[9] == slot
    assert torch.equal(first, again)


# --------------------------------------------------------------------------- residual stream
@pytest.mark.parametrize("dtype", [F32, BF16])
@pytest.mark.parametrize("n,d", [(3, 64), (1, 30), (5, 1000), (300, 40), (4, 4096), (310, 4096), (2, 1031), (3, 16384), (2, 9001), (299, 8200)])
def test_branch_norm(dtype, n, d):
    g = _gen(d)
    emb, tok = torch.randn(50, d, generator=g).to(dtype), torch.randint(0, 50, (n,), generator=g)
    pos = torch.randint(0, 100000, (n,), generator=g)
    pos[0] = 0
    w = [torch.randn(d, generator=g) for _ in range(4)]
    x = torch.empty(n, d, device=DEV)
    h1, h2 = (torch.empty(n, sops.pad8(d), dtype=dtype, device=DEV) for _ in range(2))
    wd = [v.to(DEV) for v in w]
    sops.branch_norm_(x, 1e-5, dtype, gammas=wd[:2], gamma_add=1.0, hs=(h1, h2), embed=emb.to(DEV), tokens=tok.to(DEV), embed_scale=3.3,
                      pos_turns=sops.sinusoid_turns(d, DEV), positions=pos.to(DEV))
    want = emb.double()[tok] * 3.3 + orc.sinusoid(pos, d)
    _close(x, want, 1e-6, "embedding + position")
    for h, gam in ((h1, w[0]), (h2, w[1])):
        _close(h[:, :d], orc.one_plus_norm(want, gam.double(), 1e-5), KTOL[dtype], "norm")
    ya, yb, yc = (torch.randn(n, d, generator=g).to(dtype) * s for s in (1.0, 20.0, 0.5))
    part = torch.randn(3, n, sops.pad8(d), generator=g)
    for left, l64 in ((ya, ya.double()), (part, part.double().sum(0)[:, :d])):
        sops.branch_norm_(x, 1e-5, dtype, [(left.to(DEV), wd[2]), (yb.to(DEV), wd[3])], 0.5, yc.to(DEV), (wd[0], None), 0.0, (h1, None))
        want = want + 0.5 * (orc.unit_rms(l64, 1e-5) * w[2].double() + orc.unit_rms(yb.double(), 1e-5) * w[3].double()) + yc.double()
        _close(x, want, 2e-6, "branches")
        _close(h1[:, :d], orc.unit_rms(want, 1e-5) * w[0].double(), KTOL[dtype], "norm after branches")
    sops.branch_norm_(x, 1e-5, dtype, plain=part.to(DEV))
    _close(x, want + part.double().sum(0)[:, :d], 3e-6, "plain sums")


# --------------------------------------------------------------------------- queries and keys
@pytest.mark.parametrize("dtype", [F32, BF16])
@pytest.mark.parametrize("partial", [False, True])
@pytest.mark.parametrize("heads,kv,dim,page,temp", [(4, 2, 24, 4, (0.5, 7)), (6, 6, 64, 16, None), (3, 1, 5, 3, (0.2, 1)), (32, 8, 128, 32, (0.1, 100))])
def test_whole_projection_norm_temperature_and_cache_rows(dtype, partial, heads, kv, dim, page, temp):
    g = _gen(dim)
    n, pages = 11, 9
    qc, kc = heads * dim, kv * dim
    rows = torch.randn(n, sops.pad8(qc) + sops.pad8(kc), generator=g) * 3
    src = torch.stack([rows * 0.25, rows * 0.75]).to(DEV) if partial else rows.to(dtype).to(DEV)
    rows = rows.double() if partial else rows.to(dtype).double()
    q64, k64 = rows[:, :qc], rows[:, sops.pad8(qc):sops.pad8(qc) + kc]
    wq, wk = torch.randn(qc, generator=g), torch.randn(kc, generator=g)
    slots = torch.randperm(pages * page, generator=g)[:n]
    pos = torch.tensor([0, 5, 6, 7, 12, 13, 98, 99, 100, 5000, 99999])
    ck, cv = (torch.zeros(pages, kv, page, dim, dtype=dtype, device=DEV) for _ in range(2))
    q = sops.qk_norm_post(src[..., :qc], src[..., sops.pad8(qc):], heads, kv, wq.to(DEV), wk.to(DEV), 1e-5, temp, pos.to(DEV), slots.to(DEV), ck, cv)
    want = orc.unit_rms(q64, 1e-5) * wq.double()
    if temp:
        want = want * torch.tensor([orc.temperature(int(p), *temp) for p in pos], dtype=torch.float64)[:, None]
    _close(q.reshape(n, -1), want, KTOL[dtype], "q")
    _close(ck[slots // page, :, slots % page].reshape(n, -1), orc.unit_rms(k64, 1e-5) * wk.double(), KTOL[dtype], "k")
    _close(cv[slots // page, :, slots % page].reshape(n, -1), k64, KTOL[dtype], "v")
    assert int((cv.float().abs().sum((1, 3)) > 0).sum()) == n, "only the given slots are written"


# --------------------------------------------------------------------------- attention with a linear bias
@pytest.mark.parametrize("dtype,heads,kv,dim,page,lens", [
    (F32, 4, 2, 24, 4, (40, 1, 17)), (F32, 3, 1, 50, 5, (90,)), (BF16, 4, 2, 20, 8, (40, 3)), (BF16, 8, 2, 64, 32, (300, 129, 2)),
    (BF16, 2, 1, 128, 16, (420,)), (BF16, 3, 3, 72, 8, (150, 77)), (BF16, 16, 2, 128, 128, (261,))])
def test_attention_with_linear_bias_sees_far_keys(dtype, heads, kv, dim, page, lens):
    """Every fifth query has one loud key, far back or at a page's or block's edge; portions and decode steps."""
    g = _gen(dim + page)
    scale = dim ** -0.5
    pool = torch.randperm(sum((l + page - 1) // page for l in lens) + 3, generator=g)
    kc, vc = (torch.randn(len(pool), kv, page, dim, generator=g).to(dtype) for _ in range(2))
    table = torch.full((len(lens), max(lens) // page + 2), -1, dtype=torch.int32)
    qs, want, used = [], [], 0
    for b, l in enumerate(lens):
        q, k, v = torch.randn(l, heads, dim, generator=g), torch.randn(l, kv, dim, generator=g), torch.randn(l, kv, dim, generator=g)
        for i in range(0, l, 5):
            j = [0, i // 2, max(0, i - page), max(0, i - 128), i // page * page][(i // 5) % 5]
            k[j] = 6 * q[i, -kv:] / q[i, -kv:].norm(dim=-1, keepdim=True) * dim ** 0.25
        q, k, v = q.to(dtype), k.to(dtype), v.to(dtype)
        n_pg = (l + page - 1) // page
        table[b, :n_pg] = pool[used:used + n_pg].to(torch.int32)
        used += n_pg
        for j in range(l):
            kc[table[b, j // page], :, j % page], vc[table[b, j // page], :, j % page] = k[j], v[j]
        qs.append(q)
        want.append(orc.biased_attention(q.double(), k.double(), v.double(), scale))
    slopes = torch.tensor([orc.slope(h, heads) for h in range(heads)], device=DEV)
    kd, vd, td = kc.to(DEV), vc.to(DEV), table.to(DEV)
    tol = 2e-5 if dtype == F32 else 1.5e-2
    rows = sops.attn_tile_rows(heads, kv, dim, dim, page, dtype, DEV)
    for impl, tr in {(0, rows), (1, sops.SIMT_TILE_ROWS)}:
        for cut in (0.0, 0.35, 0.9):
            first = [min(int(l * cut), l - 1) for l in lens]
            portions, row0 = [], 0
            for b, (l, f) in enumerate(zip(lens, first)):
                portions.append((b, row0, l - f, f))
                row0 += l - f
            tiles = torch.tensor(sops.make_tiles(portions, tr), dtype=torch.int32, device=DEV)
            q = torch.cat([x[f:] for x, f in zip(qs, first)]).to(DEV)
            o = sops.window_attn(q, kd, vd, td, scale, None, slopes, None, tiles, tr, impl=impl)
            _close(o.reshape(-1, heads, dim), torch.cat([w[f:] for w, f in zip(want, first)]), tol, f"impl {impl} cut {cut}")
    q = torch.stack([x[-1] for x in qs]).to(DEV)
    for impl in (0, 1):
        o = sops.window_attn(q, kd, vd, td, scale, None, slopes, None, seq_lens=torch.tensor(lens, dtype=torch.int32, device=DEV), impl=impl)
        _close(o.reshape(-1, heads, dim), torch.stack([w[-1] for w in want]), tol, f"decode, impl {impl}")


# --------------------------------------------------------------------------- recurrent kernels
def _runs(lens, cuts):
    """Steps of several sequences: portions (seq, n) per step; a single step of one token each runs the decode kernels."""
    at = [0] * len(lens)
    while any(a < l for a, l in zip(at, lens)):
        step = []
        for s, l in enumerate(lens):
            n = min(cuts[len(step) % len(cuts)] if cuts else l, l - at[s])
            if n:
                step.append((s, at[s], n))
                at[s] += n
        yield step


def _step_rows(step, state_slots):
    slots = state_slots[[s for s, _, _ in step]].to(DEV)
    if all(n == 1 for _, _, n in step):
        return sops.StepRows(slots, lens=torch.tensor([p + 1 for _, p, _ in step], dtype=torch.int32, device=DEV))
    row0, portions = 0, []
    for i, (_, p, n) in enumerate(step):
        portions.append((i, row0, n, p))
        row0 += n
    t = lambda x: torch.tensor(x, dtype=torch.int32, device=DEV)  # noqa: E731
    return sops.StepRows(slots, portions=t(portions), conv_tiles=t(sops.make_conv_tiles(portions)))


@pytest.mark.parametrize("dtype", [F32, BF16])
@pytest.mark.parametrize("inner,taps,partial", [(64, 4, False), (40, 3, True), (24, 1, False), (17, 2, False), (33, 7, True), (1200, 3, False), (8, 16, False)])
def test_causal_conv_and_its_state(dtype, inner, taps, partial):
    g = _gen(inner)
    lens, slots = (75, 1, 33, 2), torch.tensor([4, 0, 3, 1], dtype=torch.int32)
    w, b = torch.randn(inner, taps, generator=g), torch.randn(inner, generator=g)
    xs = [torch.randn(l, inner, generator=g).to(BF16) for l in lens]
    want = [orc.silu(orc.causal_conv(x.double(), w.double(), b.double())) for x in xs]
    for cuts in ((), (1,), (2,), (5, 32, 1), (33,)):
        state = torch.randn(5, taps - 1, inner, generator=g).to(dtype).to(DEV)   # what others left there
        for step in _runs(lens, cuts):
            x = torch.cat([xs[s][p:p + n] for s, p, n in step])
            n = x.shape[0]
            src = torch.zeros(n, sops.pad8(inner) + 8, dtype=dtype, device=DEV)
            src[:, :inner] = x.to(DEV).to(dtype)
            if partial:
                src = torch.stack([src.float() * 0.5, src.float() * 0.5])
            u = sops.causal_conv(src, w.to(DEV), b.to(DEV), state, _step_rows(step, slots), n)
            _close(u, torch.cat([want[s][p:p + k] for s, p, k in step]), KTOL[dtype], f"cuts {cuts} step {step}")


@pytest.mark.parametrize("dtype", [F32, BF16])
@pytest.mark.parametrize("inner,ns,partial", [(64, 16, False), (36, 24, True), (9, 1, False), (130, 5, False), (8, 40, False), (44, 128, False), (5000, 16, False),
                                              (12, 64, True)])
def test_selective_scan_and_its_state(dtype, inner, ns, partial):
    g = _gen(inner + ns)
    lens, slots = ((75, 1, 33, 2) if inner < 1000 else (40, 3)), torch.tensor([4, 0, 3, 1], dtype=torch.int32)
    a_log = torch.rand(inner, ns, generator=g) * 3 - 1.5
    bias, skip = torch.randn(inner, generator=g) - 2, torch.randn(inner, generator=g)
    us, dts, zs, bcs = ([torch.randn(l, c, generator=g).to(BF16) for l in lens] for c in (inner, inner, inner, 2 * ns))
    want = []
    for u, dt, z, bc in zip(us, dts, zs, bcs):
        step = torch.nn.functional.softplus(dt.double() + bias.double())
        y = orc.selective_scan(u.double(), step, -torch.exp(a_log.double()), bc.double()[:, :ns], bc.double()[:, ns:], skip.double())
        want.append(y * orc.silu(z.double()))
    a2 = sops.scan_decay(a_log).to(DEV)
    c8 = sops.pad8(inner)
    for cuts in ((), (1,), (2,), (5, 17, 1), (16,)):
        if inner >= 1000 and cuts not in ((), (1,)):
            continue
        state = torch.randn(5, inner, ns, generator=g).to(DEV) * 50
        for step in _runs(lens, cuts):
            def rows(src, pad):
                x = torch.cat([src[s][p:p + n] for s, p, n in step])
                out = torch.zeros(x.shape[0], pad, dtype=dtype, device=DEV)
                out[:, :x.shape[1]] = x.to(DEV).to(dtype)
                return out
            u, dt, z, bc = rows(us, c8), rows(dts, c8), rows(zs, c8), rows(bcs, sops.pad8(2 * ns))
            if partial:
                z = torch.stack([z.float() * 0.25, z.float() * 0.75])
                bc = torch.stack([bc.float(), bc.float() * 0])
            y = torch.full((u.shape[0], c8 + 16), 7.0, dtype=dtype, device=DEV)
            sops.selective_scan(u[:, :inner], dt, z, bc, bias.to(DEV), a2, skip.to(DEV), state, _step_rows(step, slots), y, c8)
            _close(y[:, :inner], torch.cat([want[s][p:p + n] for s, p, n in step]), 2e-5 if dtype == F32 else 8e-3, f"cuts {cuts} step {step}")
            assert float(y[:, inner:c8].float().abs().sum()) == 0 and float((y[:, c8:] - 7).float().abs().max()) == 0


MEMORIES = [(3, 10, 22, 7.0), (2, 40, 64, 11.0), (1, 16, 9, 3.0), (2, 64, 128, 9.0), (1, 128, 64, 15.0), (2, 256, 96, 12.0), (1, 3, 33, 5.0), (1, 300, 40, 6.0),
            (2, 128, 192, 4.0)]


@pytest.mark.parametrize("dtype", [F32, BF16])
@pytest.mark.parametrize("heads,dim,vdim,cap", MEMORIES)
def test_matrix_memory_and_its_state(dtype, heads, dim, vdim, cap):
    """Random gates, with stretches of open forget gates and of large and small input gates, so that the running maximum moves
    both ways and old keys stay visible over many tiles."""
    g = _gen(heads * dim + vdim)
    lens, slots = (300, 1, 70, 2), torch.tensor([4, 0, 3, 1], dtype=torch.int32)
    bias = torch.randn(2 * heads, generator=g)
    qs, ks, vs = ([torch.randn(l, c, generator=g).to(BF16) for l in lens] for c in (heads * dim, heads * dim, heads * vdim))
    gates = [torch.randn(l, 2 * heads, generator=g) * 2 for l in lens]
    gates[0][:, heads:] += 6
    gates[0][60:64, :heads] += 8
    gates[0][150:200, :heads] -= 9
    gates[0][220, heads:] -= 20
    want = []
    for q, k, v, gt in zip(qs, ks, vs, gates):
        n = q.shape[0]
        i, f = orc.mlstm_gates(gt.double()[:, :heads] + bias.double()[:heads], gt.double()[:, heads:] + bias.double()[heads:], cap)
        want.append(orc.mlstm(q.double().reshape(n, heads, dim) * dim ** -0.5, k.double().reshape(n, heads, dim), v.double().reshape(n, heads, vdim),
                              i, f).reshape(n, -1))
    sl = sops.memory_slices(vdim)
    for cuts in ((), (1,), (2, 63), (100, 1, 64), (65,)):
        if cuts == (1,) and dim * vdim > 5000:
            cuts = (37, 1, 1, 1, 128)
        s, z, m = (torch.randn(5, *sh, generator=g).to(DEV) * 9 for sh in ((heads, dim, vdim), (heads, sl, dim), (heads, sl)))
        got = []
        for step in _runs(lens, cuts):
            def rows(src):
                x = torch.cat([src[a][p:p + n] for a, p, n in step]).to(DEV)
                return torch.nn.functional.pad(x, (0, sops.pad8(x.shape[1]) - x.shape[1])).to(dtype)
            gt = torch.cat([gates[a][p:p + n] for a, p, n in step]).to(DEV)
            gt = torch.stack([gt * 0.5, gt * 0.5])
            n = gt.shape[1]
            o = sops.matrix_memory(rows(qs), rows(ks), rows(vs), gt, bias.to(DEV), cap, s, z, m, _step_rows(step, slots), n, dtype)
            w = torch.cat([want[a][p:p + k] for a, p, k in step])
            got.append(torch.stack([o.double().cpu(), w]).reshape(2, -1, heads, vdim))
        o, w = torch.cat(got, 1)
        tol = 5e-5 if dtype == F32 else 2e-2
        # n . q may all but cancel, which scales a whole row; the direction of every row is well conditioned
        e = (orc.unit_rms(o, 1e-12) - orc.unit_rms(w, 1e-12)).pow(2).mean(-1).sqrt()
        assert float(e.max()) < tol, f"cuts {cuts}: direction {float(e.max()):.3g}"
        e = ((o - w).pow(2).mean(-1) / (w.pow(2).mean(-1) + 1e-6)).sqrt().flatten().sort().values
        assert float(e[int(0.9 * len(e))]) < tol and float(e[-1]) < 20 * tol, f"cuts {cuts}: size {float(e[-1]):.3g}"


@pytest.mark.parametrize("dtype", [F32, BF16])
@pytest.mark.parametrize("heads,vdim", [(3, 22), (2, 64), (8, 512), (1, 9)])
def test_head_norm_and_gate(dtype, heads, vdim):
    g = _gen(vdim)
    n, c = 21, heads * vdim
    o, gt, w = torch.randn(n, c, generator=g).to(dtype), torch.randn(n, c, generator=g).to(dtype), torch.randn(c, generator=g)
    want = orc.unit_rms(o.double().reshape(n, heads, vdim), 1e-5).reshape(n, c) * w.double() * torch.sigmoid(gt.double())
    _close(sops.head_norm_gate(o.to(DEV), gt.to(DEV), w.to(DEV), heads, 1e-5), want, KTOL[dtype], "rows")
    _close(sops.head_norm_gate(o.to(DEV), torch.stack([gt.float(), gt.float() * 0]).to(DEV), w.to(DEV), heads, 1e-5), want, KTOL[dtype], "sums")
