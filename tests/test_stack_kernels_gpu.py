"""Kernels of the decoder stacks (ops/stack.py) on a GPU against the plain functions of oracle_lederax.py in float64:
residual + grouped norm with dispatch / combine, the value side of the projection, expert routing and products, and
windowed attention over shuffled pages (portions and decode steps, keys planted at the window's edges)."""
import pytest
import torch

from tests import oracle_lederax as orc
from cosmos_b200 import ops
from cosmos_b200.ops import stack as sops

pytestmark = pytest.mark.gpu
DEV = "cuda"


@pytest.fixture(autouse=True)
def _status_clean():
    assert ops.load_extension()
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


TOL = {torch.float32: 3e-6, torch.bfloat16: 8e-3}


# --------------------------------------------------------------------------- residual stream + norm
@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("n,d,groups", [(3, 64, 1), (5, 96, 3), (2, 1000, 8), (700, 40, 5), (4, 4096, 2), (3, 90, 45), (2, 72, 36), (1, 16384, 4),
                                        (300, 512, 2), (310, 2056, 1), (297, 4096, 2), (300, 8192, 2), (299, 48, 2)])
def test_residual_norm_sum_norm_and_embedding(dtype, n, d, groups):
    g = _gen(d)
    vocab = 50
    emb = torch.randn(vocab, d, generator=g).to(dtype)
    gamma = (1 + 0.3 * torch.randn(d, generator=g)).to(dtype)
    tok = torch.randint(0, vocab, (n,), generator=g)
    y = torch.randn(n, d, generator=g).to(dtype)
    x = torch.empty(n, d, device=DEV)
    h = torch.empty(n, sops.pad8(d), dtype=dtype, device=DEV)
    sops.residual_norm_(x, gamma.to(DEV), groups, 1e-5, h, embed=emb.to(DEV), tokens=tok.to(DEV), embed_scale=0.37)
    want = emb.double()[tok] * 0.37
    _close(x, want, 1e-6, "embedding")
    _close(h[:, :d], orc.grouped_rms_norm(want, gamma.double(), 1e-5, groups), TOL[dtype], "norm")
    sops.residual_norm_(x, gamma.to(DEV), groups, 1e-5, h, y=y.to(DEV), weight=0.5)
    want = want + 0.5 * y.double()
    _close(x, want, 1e-6, "sum")
    _close(h[:, :d], orc.grouped_rms_norm(want, gamma.double(), 1e-5, groups), TOL[dtype], "norm after sum")
    part = torch.randn(3, n, sops.pad8(d), generator=g)
    sops.residual_norm_(x, None, groups, 1e-5, y=part.to(DEV))
    _close(x, want + part.double().sum(0)[:, :d], 2e-6, "split sums")


@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("top,n,groups", [(1, 37, 4), (3, 37, 4), (3, 400, 2), (2, 400, 1)])
def test_residual_norm_dispatch_and_combine(dtype, top, n, groups):
    g = _gen(top)
    d = 136
    x0 = torch.randn(n, d, generator=g)
    gamma = torch.randn(d, generator=g).to(dtype)
    rows = torch.randperm(n * top, generator=g).to(torch.int32)
    x = x0.to(DEV)
    hs = torch.zeros(n * top, sops.pad8(d), dtype=dtype, device=DEV)
    sops.residual_norm_(x, gamma.to(DEV), groups, 1e-6, hs, rows.to(DEV))
    want = orc.grouped_rms_norm(x0.double(), gamma.double(), 1e-6, groups)
    _close(hs[:, :d][rows.long().to(DEV)].reshape(n, top, d), want[:, None].expand(n, top, d), TOL[dtype], "dispatch")
    y = torch.randn(n * top, d, generator=g)
    ys = torch.empty_like(y)
    ys[rows.long()] = y                                   # expert order
    sops.residual_norm_(x, None, groups, 1e-6, y=ys.to(dtype).to(DEV), y_rows=rows.to(DEV), weight=1.0 / top)
    _close(x, x0.double() + y.to(dtype).double().reshape(n, top, d).sum(1) / top, 2e-6, "combine")


# --------------------------------------------------------------------------- values
@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("partial", [False, True])
@pytest.mark.parametrize("heads,kv,dim,vdim,page", [(4, 2, 24, 40, 4), (6, 3, 64, 64, 16), (2, 2, 7, 5, 3), (8, 1, 128, 96, 32), (1, 1, 300, 130, 8)])
def test_value_norm_mixing_and_cache_rows(dtype, partial, heads, kv, dim, vdim, page):
    if partial and dtype == torch.float32:
        pytest.skip("split-K sums exist for bf16 models only")
    g = _gen(dim)
    n, pages = 9, 7
    cols = heads * dim + kv * (dim + vdim)
    qkv = torch.randn(n, cols, generator=g)
    bias = torch.randn(cols, generator=g).to(dtype)
    slots = torch.randperm(pages * page, generator=g)[:n]
    kc, vc = (torch.zeros(pages, kv, page, s, dtype=dtype, device=DEV) for s in (dim, vdim))
    lam = torch.tensor(0.3, device=DEV)
    first = torch.randn(n, kv, vdim, generator=g)
    out = torch.empty(n, kv, vdim, device=DEV)
    if partial:
        src = torch.stack([qkv * 0.25, qkv * 0.75]).to(DEV)
        rows = qkv.double() + bias.double()
    else:
        src = qkv.to(dtype).to(DEV)
        rows = qkv.to(dtype).double()
    q = sops.qkv_value_post(src, bias.to(DEV), heads, kv, 1e-5, True, slots.to(DEV), kc, vc, out, first.to(DEV), lam)
    v = orc.value_norm(rows[:, heads * dim + kv * dim:].reshape(n, kv, vdim), 1e-5)
    _close(q, rows[:, :heads * dim].reshape(n, heads, dim), TOL[dtype], "q")
    _close(kc[slots // page, :, slots % page], rows[:, heads * dim:heads * dim + kv * dim].reshape(n, kv, dim), TOL[dtype], "k")
    _close(out, v, 3e-6, "values for later layers")
    _close(vc[slots // page, :, slots % page], orc.value_mix(v, first.double(), float(lam)), TOL[dtype], "mixed v")
    assert int((kc.float().abs().sum((1, 3)) > 0).sum()) == n, "only the given slots are written"


# --------------------------------------------------------------------------- experts
def _moe_case(dtype, n, d, ff, experts, top, seed, skew=False):
    g = _gen(seed)
    vocab = 60
    table = torch.rand(vocab, experts, generator=g).argsort(1)[:, :top].to(torch.int32)
    if skew:   # most tokens to one expert, some experts empty
        table[:50, 0] = 0
        for t in range(50):
            if top > 1:
                table[t, 1:] = torch.arange(1, top)
    tok = torch.randint(0, vocab, (n,), generator=g)
    up = torch.zeros(experts, sops.pad8(ff), sops.pad8(d))
    down = torch.zeros(experts, sops.pad8(d), sops.pad8(ff))
    up[:, :ff, :d] = torch.randn(experts, ff, d, generator=g) * d ** -0.5 * 2
    down[:, :d, :ff] = torch.randn(experts, d, ff, generator=g) * ff ** -0.5
    return tok, vocab, table, up.to(dtype), down.to(dtype), torch.randn(n, d, generator=g).to(dtype)


@pytest.mark.parametrize("dtype,tile", [(torch.float32, 128), (torch.bfloat16, 128), (torch.bfloat16, 256)])
@pytest.mark.parametrize("n,d,ff,experts,top,skew", [(1, 64, 48, 4, 2, False), (33, 72, 40, 5, 1, False), (700, 136, 264, 3, 2, True),
                                                      (300, 512, 300, 40, 3, False), (5, 600, 1030, 8, 8, False)])
def test_table_routed_experts(dtype, tile, n, d, ff, experts, top, skew):
    tok, vocab, table, up, down, h = _moe_case(dtype, n, d, ff, experts, top, n + ff, skew)
    tabs = [table.to(DEV)]
    rt = sops.moe_route(tok.to(DEV), vocab, tabs, [experts], [tile], sops.route_desc(tabs, [experts], [tile]))
    rows = rt.rows[0].long().cpu()
    assert sorted(rows.tolist()) == list(range(n * top))
    hs = torch.zeros(n * top, sops.pad8(d), dtype=dtype, device=DEV)
    hs[rows.to(DEV), :d] = h.to(DEV).repeat_interleave(top, 0)
    upd, dd = up.to(DEV), down.to(DEV)
    want_a = torch.zeros(n * top, ff, dtype=torch.float64)
    ex = table[tok].reshape(-1)
    for p in range(n * top):
        want_a[rows[p]] = orc.gelu_erf(up[ex[p], :ff, :d].double() @ h[p // top].double())
    for ks in ((1,) if dtype == torch.float32 else (1, 2, 5)):
        a = sops.grouped_gemm(hs[:, :d], upd[:, :, :d], rt.tiles[0], rt.n_tiles[0], tile, gelu=True, k_splits=ks)
        _close(a[:, :ff], want_a, TOL[dtype], f"up + gelu, {ks} splits")
    want_y = torch.zeros(n * top, d, dtype=torch.float64)
    a_c = a.double().cpu()
    for p in range(n * top):
        want_y[rows[p]] = down[ex[p], :d, :ff].double() @ a_c[rows[p], :ff]
    y = sops.grouped_gemm(a, dd, rt.tiles[0], rt.n_tiles[0], tile)
    _close(y[:, :d], want_y, TOL[dtype], "down")
    if dtype == torch.bfloat16:
        for ks in (1, 3):
            part = sops.grouped_gemm(a, dd, rt.tiles[0], rt.n_tiles[0], tile, k_splits=ks, partial=True)
            _close(part.sum(0)[:, :d], want_y, 1e-4, "down, partial sums")


def test_routing_of_several_layers_at_once():
    g = _gen(5)
    vocab, n = 40, 257
    specs = [(4, 2), (9, 1), (33, 5)]
    tables = [torch.rand(vocab, e, generator=g).argsort(1)[:, :t].to(torch.int32) for e, t in specs]
    tok = torch.randint(0, vocab, (n,), generator=g)
    dev = [t.to(DEV) for t in tables]
    experts, tile = [e for e, _ in specs], [128, 256, 128]
    rt = sops.moe_route(tok.to(DEV), vocab, dev, experts, tile, sops.route_desc(dev, experts, tile))
    for i, (e, top) in enumerate(specs):
        ex = tables[i][tok].reshape(-1)
        rows = rt.rows[i].cpu().long()
        assert sorted(rows.tolist()) == list(range(n * top))
        owner = torch.empty(n * top, dtype=torch.long)
        owner[rows] = ex.long()
        assert bool((owner[1:] >= owner[:-1]).all()), "rows are sorted by expert"
        tiles = rt.tiles[i][:int(rt.n_tiles[i])].cpu()
        covered = torch.zeros(n * top, dtype=torch.long)
        for ee, r0, cnt, _ in tiles.tolist():
            assert 1 <= cnt <= tile[i] and bool((owner[r0:r0 + cnt] == ee).all())
            covered[r0:r0 + cnt] += 1
        assert bool((covered == 1).all())


# --------------------------------------------------------------------------- windowed attention
def _paged_case(dtype, lens, heads, kv, dim, vdim, page, seed, edge_window=None, loud=6.0):
    """Random q / k / v of whole sequences in shuffled pages. With `edge_window`, some queries get one key that stands out
    (aligned with the query, loud) just inside or just outside the window."""
    g = _gen(seed)
    max_pages = max((l + page - 1) // page for l in lens) + 1
    pool = torch.randperm(len(lens) * max_pages + 3, generator=g)
    kc = torch.randn(len(pool), kv, page, dim, generator=g).to(dtype)      # stale contents everywhere
    vc = torch.randn(len(pool), kv, page, vdim, generator=g).to(dtype)
    table = torch.full((len(lens), max_pages), -1, dtype=torch.int32)
    qs, ks, vs, used = [], [], [], 0
    for b, l in enumerate(lens):
        q = torch.randn(l, heads, dim, generator=g)
        k = torch.randn(l, kv, dim, generator=g)
        v = torch.randn(l, kv, vdim, generator=g)
        if edge_window:
            for i in range(0, l, 5):
                for off in ((edge_window - 1) if (i // 5) % 2 else edge_window, 0):
                    j = i - off
                    if j >= 0:
                        k[j] = loud * q[i, :kv] / q[i, :kv].norm(dim=-1, keepdim=True) * dim ** 0.25
                        break
        q, k, v = q.to(dtype), k.to(dtype), v.to(dtype)
        n_pg = (l + page - 1) // page
        table[b, :n_pg] = pool[used:used + n_pg].to(torch.int32)
        used += n_pg
        for j in range(l):
            kc[table[b, j // page], :, j % page] = k[j]
            vc[table[b, j // page], :, j % page] = v[j]
        qs.append(q), ks.append(k), vs.append(v)
    r1 = torch.rand(heads, generator=g) * 1.5 + 0.1
    r2 = torch.rand(heads, generator=g) * 0.4 + 0.05
    return qs, ks, vs, kc.to(DEV), vc.to(DEV), table.to(DEV), r1, r2


def _want(qs, ks, vs, scale, window, r1, r2):
    return [orc.windowed_attention(q.double(), k.double(), v.double(), scale, window, r1.double(), r2.double())
            for q, k, v in zip(qs, ks, vs)]


PORTIONS = [
    # dtype, heads, kv, dim, vdim, page, window, lens
    (torch.float32, 4, 2, 24, 40, 4, 7, (30, 1, 17)),
    (torch.float32, 3, 1, 50, 33, 5, 64, (70, 40)),
    (torch.float32, 2, 2, 130, 200, 16, 1, (19,)),
    (torch.bfloat16, 4, 2, 20, 36, 8, 9, (40, 3)),
    (torch.bfloat16, 4, 2, 64, 56, 32, 90, (300, 129, 2)),
    (torch.bfloat16, 2, 1, 128, 128, 16, 128, (400,)),
    (torch.bfloat16, 3, 3, 72, 40, 8, 33, (150, 77)),
    (torch.bfloat16, 2, 2, 40, 128, 64, 257, (600,)),
    (torch.bfloat16, 2, 1, 128, 72, 128, 1000, (520,)),
    (torch.bfloat16, 6, 2, 8, 16, 32, 1, (140,)),
]


@pytest.mark.parametrize("dtype,heads,kv,dim,vdim,page,window,lens", PORTIONS)
def test_portions_see_exactly_their_window(dtype, heads, kv, dim, vdim, page, window, lens):
    qs, ks, vs, kc, vc, table, r1, r2 = _paged_case(dtype, lens, heads, kv, dim, vdim, page, dim + window, edge_window=window)
    scale = dim ** -0.5
    want = _want(qs, ks, vs, scale, window, r1, r2)
    tile_rows = sops.attn_tile_rows(heads, kv, dim, vdim, page, dtype, DEV)
    for impl, rows in {(0, tile_rows), (1, sops.SIMT_TILE_ROWS)}:
        # the last part of every sequence at once, cut at several places
        for cut in (0.0, 0.35, 0.9):
            first = [min(int(l * cut), l - 1) for l in lens]
            q = torch.cat([x[f:] for x, f in zip(qs, first)])
            row0, portions = 0, []
            for b, (l, f) in enumerate(zip(lens, first)):
                portions.append((b, row0, l - f, f))
                row0 += l - f
            tiles = torch.tensor(sops.make_tiles(portions, rows), dtype=torch.int32, device=DEV)
            o = sops.window_attn(q.to(DEV), kc, vc, table, scale, window, r1.to(DEV), r2.to(DEV), tiles, rows, impl=impl)
            _close(o.reshape(-1, heads, vdim), torch.cat([w[f:] for w, f in zip(want, first)]),
                   2e-5 if dtype == torch.float32 else 1.5e-2, f"impl {impl} cut {cut}")


DECODE = [
    (torch.float32, 4, 2, 24, 40, 4, 7, (30, 1, 17)),
    (torch.float32, 5, 1, 50, 33, 5, 64, (70, 40)),
    (torch.bfloat16, 6, 2, 64, 64, 32, 40, (90, 41, 40, 39)),      # group of 3: CUDA-core kernel
    (torch.bfloat16, 8, 4, 64, 48, 32, 90, (300, 91, 90, 89, 1)),
    (torch.bfloat16, 8, 1, 128, 128, 16, 128, (400, 129, 5)),
    (torch.bfloat16, 4, 2, 72, 40, 8, 33, (150, 34, 33)),
    (torch.bfloat16, 2, 2, 40, 128, 64, 257, (600, 258, 257)),
    (torch.bfloat16, 4, 1, 128, 72, 128, 1000, (1400, 520)),
    (torch.bfloat16, 2, 1, 16, 8, 8, 1, (33, 1)),
]


@pytest.mark.parametrize("dtype,heads,kv,dim,vdim,page,window,lens", DECODE)
def test_decode_steps_see_exactly_their_window(dtype, heads, kv, dim, vdim, page, window, lens):
    qs, ks, vs, kc, vc, table, r1, r2 = _paged_case(dtype, lens, heads, kv, dim, vdim, page, dim + window, edge_window=window)
    scale = dim ** -0.5
    q = torch.stack([x[-1] for x in qs] + [qs[0][0]]).to(DEV)          # one idle slot at the end
    tab = torch.cat([table, table[:1]])
    seq = torch.tensor(list(lens) + [0], dtype=torch.int32, device=DEV)
    want = []
    for qq, k, v in zip(qs, ks, vs):   # the last query only
        l = qq.shape[0]
        o = []
        for h in range(heads):
            lo = max(0, l - window)
            dist = torch.arange(l - 1 - lo, -1, -1).double()
            s = k[lo:, h // (heads // kv)].double() @ qq[-1, h].double() * scale - orc.distance_bias(r1[h].double(), r2[h].double(), dist)
            o.append(torch.softmax(s, 0) @ v[lo:, h // (heads // kv)].double())
        want.append(torch.stack(o))
    want.append(torch.zeros_like(want[0]))
    for impl in (0, 1):
        for max_len in (None, max(lens)):
            o = sops.window_attn(q, kc, vc, tab, scale, window, r1.to(DEV), r2.to(DEV), seq_lens=seq, max_len=max_len, impl=impl)
            _close(o.reshape(-1, heads, vdim), torch.stack(want), 2e-5 if dtype == torch.float32 else 1.5e-2, f"impl {impl}")


def test_far_key_wins_through_the_bias_and_no_bias_is_plain_attention():
    """One loud key at the far end of a long window must dominate; without r1 / r2 the op is plain windowed attention."""
    l, window, dim = 700, 650, 64
    qs, ks, vs, kc, vc, table, r1, r2 = _paged_case(torch.bfloat16, (l,), 2, 1, dim, dim, 16, 3)
    q, k = qs[0], ks[0].clone()
    j = l - window
    k[j] = (14.0 * q[-1, 0] / q[-1, 0].float().norm()).to(torch.bfloat16)
    kc[table[0, j // 16].long(), :, j % 16] = k[j].to(DEV)
    o = {}
    for name, (a, b) in {"bias": (r1, r2), "none": (None, None)}.items():
        aa, bb = (None, None) if a is None else (a.to(DEV), b.to(DEV))
        zero = torch.zeros(2)
        want = orc.windowed_attention(q.double(), k.double(), vs[0].double(), 1.0, window, (zero if a is None else a).double(),
                                      (zero if b is None else b).double())[-1]
        dec = sops.window_attn(q[-1:].to(DEV), kc, vc, table, 1.0, window, aa, bb,
                               seq_lens=torch.tensor([l], dtype=torch.int32, device=DEV))
        tiles = torch.tensor([(0, 0, 2, l - 2)], dtype=torch.int32, device=DEV)
        pre = sops.window_attn(q[-2:].to(DEV), kc, vc, table, 1.0, window, aa, bb, tiles, 256)[1:]
        _close(dec.reshape(2, dim), want, 1.5e-2, name)
        _close(pre.reshape(2, dim), want, 1.5e-2, name)
        o[name] = want
    assert (o["bias"][0] - vs[0][j, 0].double()).abs().max() < 0.2, "the planted key dominates head 0"
