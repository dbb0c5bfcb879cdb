"""Checks shared by the CPU tests (plain definitions) and the GPU tests (kernels) of the decoder stacks: the serving decoder
of a small model against the plain implementation of its family."""
from types import SimpleNamespace

import torch

from tests import mererax_cases, oracle_lederax, oracle_mererax
from tests import stack_cases as cases

LEDERAX = SimpleNamespace(cases=cases, orc=oracle_lederax)
MERERAX = SimpleNamespace(cases=mererax_cases, orc=oracle_mererax)


def setup(tmp_path, name, dtype, device, seed=1, page_size=4, fam=LEDERAX):
    cfg = fam.cases.CONFIGS[name]
    t = fam.cases.weights(cfg, seed)
    return cfg, t, cases.decoder(fam.cases.write(cfg, t, tmp_path / name), dtype, device, page_size)


def whole_prompt_and_layers(tmp_path, name, dtype, device, tol, n=61, page_size=4, fam=LEDERAX):
    cfg, t, dec = setup(tmp_path, name, dtype, device, page_size=page_size, fam=fam)
    ids = cases.tokens(cfg, n)
    want_layers, got_layers = [], []
    want = fam.orc.forward(cfg, t, ids, layers_out=want_layers)
    assert dec.cache.reserve(7, n)
    got = dec.run_portions([(7, ids, 0, list(range(n)))], got_layers)
    for i, (a, b) in enumerate(zip(got_layers, want_layers)):
        err = float((a.double().cpu() - b).abs().max() / b.abs().max())
        assert err < tol, f"residual stream after layer {i}: {err:.3g}"
    assert len(got_layers) == len(want_layers)
    e = cases.error(got, want)
    assert e < tol, f"logits: {e:.3g}"
    # asked rows only, in any order
    assert dec.cache.reserve(8, n)
    some = dec.run_portions([(8, ids, 0, [n - 1, 0, 17])])
    assert cases.error(some, want[[n - 1, 0, 17]]) < tol


def portions_and_token_by_token(tmp_path, name, dtype, device, tol, n=61, page_size=4, fam=LEDERAX):
    cfg, t, dec = setup(tmp_path, name, dtype, device, page_size=page_size, fam=fam)
    ids = cases.tokens(cfg, n, 3)
    want = fam.orc.forward(cfg, t, ids)
    for k, cuts in enumerate(([n], [1], [2], [3, 1, 7, 2], [page_size], [page_size + 1], [n - 20] + [1] * 20, [1, n - 1])):
        got = cases.feed(dec, k, ids, cuts)
        e = cases.error(got, want)
        assert e < tol, f"portions {cuts[:4]}: {e:.3g}"
        dec.cache.release(k)   # its pages serve the next run
    assert dec.cache.alloc.num_free() == dec.cache.k[0].shape[0]
    if dec.cache.states is not None:
        assert len(dec.cache.states.free) == dec.cache.states.slots


def mixed_batches(tmp_path, name, dtype, device, tol, page_size=4, fam=LEDERAX):
    """Requests of unequal length whose portions share steps, with others that decode; each as if alone."""
    cfg, t, dec = setup(tmp_path, name, dtype, device, page_size=page_size, fam=fam)
    lens = (37, 5, 50, 1, 22)
    ids = [cases.tokens(cfg, n, 10 + i) for i, n in enumerate(lens)]
    want = [fam.orc.forward(cfg, t, x) for x in ids]
    at, got = [0] * 5, [[] for _ in lens]
    g = torch.Generator().manual_seed(4)
    while any(a < n for a, n in zip(at, lens)):
        entries = []
        for i, n in enumerate(lens):
            take = min(int(torch.tensor([0, 1, 1, 2, 3, 11])[torch.randint(0, 6, (1,), generator=g)]), n - at[i])
            if take:
                assert dec.cache.reserve(i, take)
                entries.append((i, ids[i][at[i]:at[i] + take], at[i], list(range(take))))
        if not entries:
            continue
        lg = dec.run_portions(entries).float().cpu()
        for i, toks, _, _ in entries:
            got[i].append(lg[:len(toks)])
            lg = lg[len(toks):]
            at[i] += len(toks)
    for i in range(len(lens)):
        e = cases.error(torch.cat(got[i]), want[i])
        assert e < tol, f"request {i}: {e:.3g}"


def greedy_generation(tmp_path, name, dtype, device, slack, use_graph, page_size=4, new=30, max_prefill=13, fam=LEDERAX):
    """The serving engine (admission, portions, decode steps, slots and pages used again) against teacher-forced oracle
    logits: every token it emits is the oracle's best up to `slack` (a share of the logits' spread)."""
    from cosmos_b200.models.stack import load_stack
    from cosmos_b200.serve.engine import BatchEngine

    cfg = fam.cases.CONFIGS[name]
    t = fam.cases.weights(cfg, 1)
    model = load_stack(fam.cases.write(cfg, t, tmp_path / name), dtype, device)
    eng = BatchEngine(model, max_batch=2, max_len=120, page_size=page_size, use_graph=use_graph, max_prefill_tokens=max_prefill)
    free = eng.dec.cache.alloc.num_free()
    reqs = [eng.submit(cases.tokens(cfg, n, 20 + n), k) for n, k in ((40, new), (3, 8), (17, new), (1, 12), (29, 5))]
    eng.run_until_done(max_steps=500)
    assert eng.dec.cache.alloc.num_free() == free, "all pages went back"
    if eng.dec.cache.states is not None:
        assert list(eng.dec.cache.states.slot_of) == [eng.scratch_seq], "all state slots went back"
    for r in reqs:
        assert r.finish_reason == "length" and len(r.out) == r.max_new_tokens
        seq = r.ids + r.out[:-1]
        lg = fam.orc.forward(cfg, t, seq)[len(r.ids) - 1:]
        gap = lg.max(-1).values - lg.gather(1, torch.tensor(r.out)[:, None])[:, 0]
        assert float(gap.max()) <= slack * float(lg.std()), f"request {r.rid}: {float(gap.max()):.3g}"
    return reqs
