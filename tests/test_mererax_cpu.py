"""Mererax on the plain definitions (CPU, fp32): the serving decoder, cache, states, scheduler and loaders against the plain
implementation in oracle_mererax.py, and the oracle's own sensitivity to mistakes."""
import copy
import json
import math
import subprocess
import sys
from pathlib import Path

import pytest
import torch

from cosmos_b200.config import get_model_config, mererax_config_from_dict
from cosmos_b200.models.stack import is_stack_name, load_stack
from cosmos_b200.ops import stack as sops
from cosmos_b200.serve.paged import StateCache
from tests import mererax_cases as mcases
from tests import oracle_mererax as orc
from tests import stack_cases as cases
from tests import stack_checks as checks

ROOT = Path(__file__).resolve().parents[1]
TOL = 2e-5
FAM = checks.MERERAX
F32 = torch.float32


@pytest.mark.parametrize("name", sorted(mcases.CONFIGS))
def test_whole_prompt_and_residual_stream(tmp_path, name):
    checks.whole_prompt_and_layers(tmp_path, name, F32, "cpu", TOL, fam=FAM)


@pytest.mark.parametrize("name,page", [("mixed", 3), ("mixed", 4), ("bare", 4), ("chain", 5)])
def test_portions_equal_the_whole_prompt(tmp_path, name, page):
    checks.portions_and_token_by_token(tmp_path, name, F32, "cpu", TOL, page_size=page, fam=FAM)


@pytest.mark.parametrize("name", ["mixed", "bare"])
def test_batches_of_unequal_requests_equal_each_alone(tmp_path, name):
    checks.mixed_batches(tmp_path, name, F32, "cpu", TOL, fam=FAM)


def test_first_tokens_alone(tmp_path):
    """Sequences of one, two and three tokens, whole and token by token, on a slot that others have used."""
    cfg, t, dec = checks.setup(tmp_path, "mixed", F32, "cpu", fam=FAM)
    cases.feed(dec, 99, cases.tokens(cfg, 30, 5), [7])
    dec.cache.release(99)
    for n in (1, 2, 3):
        ids = cases.tokens(cfg, n, 40 + n)
        want = orc.forward(cfg, t, ids)
        for cuts in ([n], [1]):
            assert cases.error(cases.feed(dec, n, ids, cuts), want) < TOL
            dec.cache.release(n)


def test_greedy_generation_through_the_engine(tmp_path):
    reqs = checks.greedy_generation(tmp_path, "mixed", F32, "cpu", 1e-4, use_graph=False, fam=FAM)
    from cosmos_b200.serve.engine import BatchEngine
    eng = BatchEngine(load_stack(tmp_path / "mixed", F32), max_batch=1, max_len=120, page_size=8, use_graph=False)
    for r in reqs:   # one at a time through a fresh engine: the same tokens
        q = eng.submit(r.ids, r.max_new_tokens)
        eng.run_until_done()
        assert q.out == r.out


# --------------------------------------------------------------------------- would a mistake show?
MISTAKES = ["bias distance + 1 beyond one", "slope of the next head", "no temperature", "temperature one token late", "per-head q norm",
            "keys normed before they serve as values", "norm weights not around one", "no position vector", "sine and cosine swapped",
            "branches not halved", "branch norms swapped", "no floor of the denominator", "forget gate without cap", "state lost",
            "conv taps reversed", "conv bias lost", "skip lost", "B and C swapped", "step without bias", "decay not negated"]


@pytest.mark.parametrize("mistake", MISTAKES)
def test_every_mechanism_shows_in_the_logits(monkeypatch, mistake):
    """Plants a mistake in the plain implementation: its logits must move by far more than the tests allow."""
    cfg = copy.deepcopy(mcases.CONFIGS["mixed"])
    t = {k: v.double() for k, v in mcases.weights(cfg, 1).items()}
    ids = cases.tokens(cfg, 40)
    want = orc.forward(cfg, t, ids)

    def swap(name, fn):
        monkeypatch.setattr(orc, name, fn)

    slope, temperature, unit, one_plus, mlstm, scan, conv, sinus = (orc.slope, orc.temperature, orc.unit_rms, orc.one_plus_norm, orc.mlstm,
                                                                    orc.selective_scan, orc.causal_conv, orc.sinusoid)
    if mistake == "bias distance + 1 beyond one":
        swap("biased_attention", lambda q, k, v, s, first=0: _shifted_attention(q, k, v, s))
    elif mistake == "slope of the next head":
        swap("slope", lambda h, n: slope(h + 1, n))
    elif mistake == "no temperature":
        swap("temperature", lambda p, c, e: 1.0)
    elif mistake == "temperature one token late":
        swap("temperature", lambda p, c, e: temperature(p - 1, c, e))
    elif mistake == "per-head q norm":
        swap("unit_rms", lambda x, eps: unit(x.reshape(x.shape[0], 4, 12), eps).reshape(x.shape) if x.shape[-1] == 48 and x.dim() == 2 else unit(x, eps))
    elif mistake == "keys normed before they serve as values":
        att = orc.biased_attention
        swap("biased_attention", lambda q, k, v, s, first=0: att(q, k, k, s, first))
    elif mistake == "norm weights not around one":
        swap("one_plus_norm", lambda x, w, eps: one_plus(x, w - 1, eps))
    elif mistake == "no position vector":
        swap("sinusoid", lambda p, d: 0 * sinus(p, d))
    elif mistake == "sine and cosine swapped":
        swap("sinusoid", lambda p, d: sinus(p, d).reshape(len(p), -1, 2).flip(-1).reshape(len(p), -1))
    elif mistake == "branches not halved":
        mix = orc.parallel_mixer
        swap("parallel_mixer", lambda *a: 2 * mix(*a))
    elif mistake == "no floor of the denominator":
        swap("mlstm", _mlstm_without_floor)
    elif mistake == "forget gate without cap":
        gates = orc.mlstm_gates
        swap("mlstm_gates", lambda i, f, cap: (gates(i, f, cap)[0], torch.nn.functional.logsigmoid(f)))
    elif mistake == "state lost":
        swap("mlstm", lambda q, k, v, i, f: torch.cat([mlstm(*(a[:20] for a in (q, k, v, i, f))), mlstm(*(a[20:] for a in (q, k, v, i, f)))]))
    elif mistake == "conv taps reversed":
        swap("causal_conv", lambda x, w, b: conv(x, w.flip(1), b))
    elif mistake == "conv bias lost":
        swap("causal_conv", lambda x, w, b: conv(x, w, 0 * b))
    elif mistake == "skip lost":
        swap("selective_scan", lambda u, dt, a, b, c, d: scan(u, dt, a, b, c, 0 * d))
    elif mistake == "B and C swapped":
        swap("selective_scan", lambda u, dt, a, b, c, d: scan(u, dt, a, c, b, d))
    elif mistake == "decay not negated":
        swap("selective_scan", lambda u, dt, a, b, c, d: scan(u, dt, -0.01 * a, b, c, d))
    elif mistake == "branch norms swapped":
        t["l0.mix.left.out"], t["l0.mix.right.out"] = t["l0.mix.right.out"], t["l0.mix.left.out"]
    elif mistake == "step without bias":
        t["l1.mix.dt.b"] = 0 * t["l1.mix.dt.b"]
    got = orc.forward(cfg, t, ids)
    assert cases.error(got, want) > 10 * TOL


def _shifted_attention(q, k, v, scale):
    """Every distance but zero one too large: what an off-by-one in the cached part of the bias would do."""
    n, heads, _ = q.shape
    out = q.new_zeros(n, heads, v.shape[-1])
    for h in range(heads):
        g = h // (heads // k.shape[1])
        for i in range(n):
            dist = torch.arange(i, -1, -1, dtype=q.dtype)
            s = k[:i + 1, g] @ q[i, h] * scale - orc.slope(h, heads) * (dist + (dist > 0))
            out[i, h] = torch.softmax(s, 0) @ v[:i + 1, g]
    return out


def _mlstm_without_floor(q, k, v, i, f):
    n, heads, dim = q.shape
    out = q.new_zeros(n, heads, v.shape[-1])
    for h in range(heads):
        s, z = q.new_zeros(dim, v.shape[-1]), q.new_zeros(dim)
        for t in range(n):
            s = torch.exp(f[t, h]) * s + torch.exp(i[t, h]) * torch.outer(k[t, h], v[t, h])
            z = torch.exp(f[t, h]) * z + torch.exp(i[t, h]) * k[t, h]
            out[t, h] = (s.t() @ q[t, h]) / ((z @ q[t, h]).abs() + 1e-6)
    return out


# --------------------------------------------------------------------------- the plain functions themselves
def test_oracle_mechanisms_on_hand_made_inputs():
    d = torch.float64
    # equal scores: head 0 of one head has slope 2^-8
    k, v = torch.zeros(3, 1, 2, dtype=d), torch.tensor([1.0, 2.0, 4.0], dtype=d).reshape(3, 1, 1)
    o = orc.biased_attention(k, k, v, 1.0)
    w = [math.exp(-j / 256) for j in range(3)]
    assert abs(float(o[2, 0, 0]) - (4 + 2 * w[1] + w[2]) / sum(w)) < 1e-12
    assert orc.temperature(6, 0.5, 7) == 1 + 0.5 * math.log(2) and orc.temperature(5, 0.5, 7) == 1.0
    s = orc.sinusoid(torch.tensor([3]), 5)[0]
    want = [math.sin(3), math.cos(3), math.sin(3 * 10000 ** -0.4), math.cos(3 * 10000 ** -0.4), math.sin(3 * 10000 ** -0.8)]
    assert torch.allclose(s, torch.tensor(want, dtype=d))
    # one head, one key: the first token's memory with i below and above the starting maximum of zero
    one = torch.ones(1, 1, 1, dtype=d)
    for i, want in ((-1.0, math.exp(-0.5) * 3 / (math.exp(0.5) + 1e-6)), (2.0, 3 / (1 + 1e-6))):
        o = orc.mlstm(one, one, 3 * one, torch.full((1, 1), i, dtype=d), torch.full((1, 1), -0.5, dtype=d))
        assert abs(float(o) - want) < 1e-9
    y = orc.causal_conv(torch.tensor([[1.0], [10.0], [100.0]], dtype=d), torch.tensor([[0.5, 2.0]], dtype=d), torch.tensor([7.0], dtype=d))
    assert y[:, 0].tolist() == [9.0, 27.5, 212.0]
    z = torch.ones(2, 1, dtype=d)
    y = orc.selective_scan(z, 0.5 * z, -torch.ones(1, 1, dtype=d), 2 * z, 3 * z, torch.tensor([0.25], dtype=d))
    assert torch.allclose(y[:, 0], torch.tensor([3.25, 3 * (math.exp(-0.5) + 1) + 0.25], dtype=d))


# --------------------------------------------------------------------------- definitions used on CPU
def test_idle_decode_slots_leave_states_alone_and_positions_zero_start_clean():
    g = torch.Generator().manual_seed(0)
    state = torch.randn(3, 4, 2, generator=g)
    before = state.clone()
    rows = sops.StepRows(torch.tensor([2, 0], dtype=torch.int32), lens=torch.tensor([0, 1], dtype=torch.int32))
    u, y = torch.randn(2, 4, generator=g), torch.full((2, 8), 5.0)
    args = [torch.randn(2, 4, generator=g), torch.randn(2, 4, generator=g), torch.randn(2, 4, generator=g)]
    a2 = -torch.rand(4, 2, generator=g)
    sops.selective_scan(u, args[0], args[1], args[2], torch.zeros(4), a2, torch.ones(4), state, rows, y, 8)
    assert torch.equal(state[1:], before[1:]) and float(y[0].abs().max()) == 0 and float(y[:, 4:].abs().max()) == 0
    again = before * 7
    y2 = torch.empty(2, 8)
    sops.selective_scan(u, args[0], args[1], args[2], torch.zeros(4), a2, torch.ones(4), again, rows, y2, 8)
    assert torch.equal(y[1], y2[1]) and torch.equal(again[0], state[0])


def test_state_slots_are_handed_out_grown_and_taken_back():
    c = StateCache([{"a": ((2,), F32)}, {}], 2, "cpu")
    assert c.acquire(10) and c.acquire(11) and c.acquire(10) and c.slot_of[10] != c.slot_of[11]
    c.tensors[0]["a"][c.slot_of[11]] = 3.0
    assert c.acquire(12) and c.slots == 4 and c.tensors[0]["a"].shape == (4, 2)
    assert float(c.tensors[0]["a"][c.slot_of[11]].sum()) == 6.0
    assert c.acquire(13)
    c.frozen = True
    assert not c.acquire(14)
    freed = c.slot_of[10]
    c.release(10)
    assert c.acquire(14) and c.slot_of[14] == freed


def test_a_request_that_finds_no_pages_holds_no_state_slot(tmp_path):
    cfg, _, dec = checks.setup(tmp_path, "mixed", F32, "cpu", fam=FAM)
    assert not dec.cache.reserve(5, 10 ** 6) and 5 not in dec.cache.states.slot_of
    assert dec.cache.reserve(5, 3) and not dec.cache.reserve(5, 10 ** 6) and 5 in dec.cache.states.slot_of


def test_conv_tiles_cover_portions():
    assert sops.make_conv_tiles([(0, 0, 40, 5), (2, 40, 1, 0)]) == [(0, 0, 32, 5, 0, 0, 0, 0), (0, 32, 8, 5, 0, 0, 0, 0), (2, 40, 1, 0, 40, 0, 0, 0)]


# --------------------------------------------------------------------------- configuration and checkpoints
def test_config_round_trip_registry_and_checks():
    for doc in mcases.CONFIGS.values():
        cfg = mererax_config_from_dict(doc)
        assert mererax_config_from_dict(cfg.to_dict()) == cfg and cfg.to_dict() == doc
    assert is_stack_name("mererax-tiny")
    big, nano = get_model_config("mererax-8b"), get_model_config("Cosmos3-Nano")
    assert (big.d_model, big.n_layers) == (nano.d_model, nano.n_layers) and big.layers[2].mlp.ff == nano.ffn_dim
    for change, match in ((lambda d: d["layers"][1].update(type="rwkv"), "mixer type"),
                          (lambda d: d["layers"][1].update(mlp={"kind": "moe"}), "feed-forward kind"),
                          (lambda d: d["layers"][0].update(weights_of=9), "no layer 9"),
                          (lambda d: d["layers"][0].update(weights_of=3), "weights of its own"),
                          (lambda d: d["layers"][4].update(weights_of=2), "equal layer"),
                          (lambda d: d["layers"][0]["mixer"]["left"].update(vdim=8), "keys serve as values"),
                          (lambda d: d["layers"][1]["mixer"].update(conv=0), "positive sizes")):
        bad = copy.deepcopy(mcases.CONFIGS["mixed"])
        change(bad)
        with pytest.raises(ValueError, match=match):
            mererax_config_from_dict(bad)


@pytest.mark.parametrize("name", ["mixed", "chain", "bare"])
def test_checkpoints_load_save_and_are_checked(tmp_path, name):
    cfg = mcases.CONFIGS[name]
    t = mcases.weights(cfg, 4)
    m = load_stack(mcases.write(cfg, t, tmp_path / "a"), torch.bfloat16)

    def whole(model):
        return {k: torch.cat(v) if isinstance(v, tuple) else v for k, v in model.checkpoint_views().items()}

    assert set(whole(m)) == set(t)
    for k, v in whole(m).items():
        assert torch.equal(v.float(), t[k].float()), k
    m.save(tmp_path / "b")
    for k, v in whole(load_stack(tmp_path / "b", F32)).items():
        assert torch.equal(v.float(), t[k].float()), k
    some = sorted(k for k in t if ".mix." in k)[3]
    with pytest.raises(KeyError, match="missing"):
        load_stack(mcases.write(cfg, {k: v for k, v in t.items() if k != some}, tmp_path / "c"), F32)


# --------------------------------------------------------------------------- trace replay, command line, server
def test_trace_replay_writes_the_wanted_logits(tmp_path):
    import numpy as np
    cfg = mcases.CONFIGS["mixed"]
    t = mcases.weights(cfg, 5)
    model = mcases.write(cfg, t, tmp_path / "model")
    a, b, c = cases.tokens(cfg, 19, 1), cases.tokens(cfg, 8, 2), cases.tokens(cfg, 6, 3)
    steps = [{"step": 0, "entries": [{"id": "a", "tokens": a[:11], "want": [10, 2]}], "end": []},
             {"step": 1, "entries": [{"id": "a", "tokens": a[11:13], "want": []}, {"id": "c", "tokens": c[:2], "want": []}], "end": []},
             {"step": 2, "entries": [{"id": "a", "tokens": a[13:14], "want": [0]}, {"id": "b", "tokens": b, "want": [7]}], "end": ["b"]},
             {"step": 3, "entries": [{"id": "a", "tokens": a[14:], "want": [4]}], "end": ["a"]},
             {"step": 4, "entries": [{"id": "a", "tokens": b, "want": [0, 7]}, {"id": "c", "tokens": c[2:], "want": [3]}], "end": ["a"]}]
    r = subprocess.run([sys.executable, str(ROOT / "bin" / "trace_run"), "--model", str(model), "--dtype", "float32", "--device",
                        "cpu", "--out", str(tmp_path / "out"), "--max-tokens", "60", "--page-size", "4"],
                       input="".join(json.dumps(s) + "\n" for s in steps), capture_output=True, text=True, timeout=300)
    assert r.returncode == 0, r.stderr[-2000:]
    assert [l for l in r.stdout.splitlines() if l.startswith("done")] == [f"done {i}" for i in range(5)]
    la, lb, lc = (orc.forward(cfg, t, x) for x in (a, b, c))
    want = {0: la[[10, 2]], 2: torch.stack([la[13], lb[7]]), 3: la[[18]], 4: torch.stack([lb[0], lb[7], lc[5]])}
    for s, w in want.items():
        got = torch.from_numpy(np.fromfile(tmp_path / "out" / f"{s}.f32", dtype="<f4")).reshape(w.shape)
        assert cases.error(got, w) < TOL, s


def test_command_line_and_server_take_a_registered_name(tmp_path):
    from types import SimpleNamespace

    from cosmos_b200.scripts import inference
    from cosmos_b200.serve.server import stack_server
    spec = tmp_path / "specs.jsonl"
    spec.write_text(json.dumps({"model_mode": "reasoner", "name": "a", "prompt": "hello", "max_new_tokens": 6, "do_sample": False}))
    assert inference.main(["-i", str(spec), "-o", str(tmp_path / "o"), "--checkpoint-path", "mererax-tiny", "--device", "cpu"]) == 0
    assert (tmp_path / "o" / "a" / "reasoner_text.txt").exists()
    srv = stack_server(SimpleNamespace(model="mererax-tiny", max_num_seqs=2, max_model_len=128), None, F32)
    try:
        body = {"messages": [{"role": "user", "content": "hi there"}], "max_tokens": 7, "temperature": 0}
        a, b = srv.chat_completions(dict(body)), srv.chat_completions(dict(body, seed=3))
        assert a["choices"][0]["message"]["content"] == b["choices"][0]["message"]["content"]
    finally:
        srv.batch_engine.close()
