"""Decoder stacks on the plain definitions (CPU, fp32): the serving decoder, cache, scheduler and loaders of a Lederax model
against the plain implementation in oracle_lederax.py, and the oracle's own sensitivity to mistakes."""
import copy
import json
import subprocess
import sys
from pathlib import Path

import pytest
import torch

from cosmos_b200.config import get_model_config, lederax_config_from_dict, stack_config_from_dir
from cosmos_b200.models.stack import StackModel, is_stack_name, load_stack
from cosmos_b200.ops import stack as sops
from tests import oracle_lederax as orc
from tests import stack_cases as cases
from tests import stack_checks as checks

ROOT = Path(__file__).resolve().parents[1]
TOL = 2e-5


@pytest.mark.parametrize("name", sorted(cases.CONFIGS))
def test_whole_prompt_and_residual_stream(tmp_path, name):
    checks.whole_prompt_and_layers(tmp_path, name, torch.float32, "cpu", TOL)


@pytest.mark.parametrize("name", ["mixed", "late_mix", "no_mix"])
@pytest.mark.parametrize("page", [3, 4])
def test_portions_equal_the_whole_prompt(tmp_path, name, page):
    checks.portions_and_token_by_token(tmp_path, name, torch.float32, "cpu", TOL, page_size=page)


def test_batches_of_unequal_requests_equal_each_alone(tmp_path):
    checks.mixed_batches(tmp_path, "mixed", torch.float32, "cpu", TOL)


def test_greedy_generation_through_the_engine(tmp_path):
    reqs = checks.greedy_generation(tmp_path, "mixed", torch.float32, "cpu", 1e-4, use_graph=False)
    # the same prompts one at a time through a fresh engine: the same tokens
    from cosmos_b200.serve.engine import BatchEngine
    eng = BatchEngine(load_stack(tmp_path / "mixed", torch.float32), max_batch=1, max_len=120, page_size=8, use_graph=False)
    for r in reqs:
        q = eng.submit(r.ids, r.max_new_tokens)
        eng.run_until_done()
        assert q.out == r.out


def test_end_tokens_sampling_parameters_and_media_requests(tmp_path):
    from cosmos_b200.serve.engine import BatchEngine
    cfg = cases.CONFIGS["all_experts"]
    model = load_stack(cases.write(cfg, cases.weights(cfg, 2), tmp_path), torch.float32)
    eng = BatchEngine(model, max_batch=3, max_len=60, page_size=4, use_graph=False)
    probe = eng.submit([3, 1, 4], 6)
    eng.run_until_done()
    r = eng.submit([3, 1, 4], 6, eos_ids=(probe.out[2],))
    s = eng.submit([3, 1, 4], 6, temperature=0.8, top_k=5, top_p=0.9, presence_penalty=0.5, repetition_penalty=1.2)
    eng.run_until_done()
    assert r.finish_reason == "stop" and r.out == probe.out[:probe.out.index(probe.out[2]) + 1]
    assert len(s.out) == 6 and all(0 <= t < cfg["vocab"] for t in s.out)
    with pytest.raises(ValueError, match="media"):
        eng.submit([1, 2], 3, embeds=torch.zeros(2, cfg["width"]), positions=torch.zeros(3, 2))


def test_long_prompts_do_not_hold_up_the_running_requests(tmp_path):
    """A prompt longer than the portion limit is fed over several steps while another request keeps decoding."""
    from cosmos_b200.serve.engine import BatchEngine
    cfg = cases.CONFIGS["mixed"]
    model = load_stack(cases.write(cfg, cases.weights(cfg, 2), tmp_path), torch.float32)
    eng = BatchEngine(model, max_batch=2, max_len=90, page_size=4, use_graph=False, max_prefill_tokens=10)
    a = eng.submit([5], 20)
    eng.step()
    b = eng.submit(cases.tokens(cfg, 45, 9), 4)
    progress = []
    for _ in range(5):
        before = len(a.out)
        eng.step()
        progress.append((b.prefilled, len(a.out) - before))
    assert [p for p, _ in progress] == [10, 20, 30, 40, 45] and all(d == 1 for _, d in progress)
    eng.run_until_done()
    seq = b.ids + b.out[:-1]
    want = orc.forward(cfg, cases.weights(cfg, 2), seq)[len(b.ids) - 1:].argmax(-1)
    assert b.out == want.tolist()


# --------------------------------------------------------------------------- would a mistake show?
def _swap(monkeypatch, name, fn):
    monkeypatch.setattr(orc, name, fn)


MISTAKES = ["window + 1", "window - 1", "no bias", "bias distance + 1", "no value norm", "no mixing", "mixing swapped",
            "first layer's values for late_mix", "one norm group", "tanh gelu", "shifted table", "weights not divided", "no q bias"]


@pytest.mark.parametrize("mistake", MISTAKES)
def test_every_mechanism_shows_in_the_logits(monkeypatch, mistake):
    """Plants a mistake in the plain implementation: its logits must move by far more than the tests allow."""
    name = "late_mix" if mistake.startswith("first layer") else "mixed"
    cfg = copy.deepcopy(cases.CONFIGS[name])
    t = dict(cases.weights(cfg, 1))
    ids = cases.tokens(cfg, 40)
    want = orc.forward(cfg, t, ids)
    bias, norm = orc.distance_bias, orc.grouped_rms_norm
    if mistake in ("window + 1", "window - 1"):
        for entry in cfg["layers"]:
            entry["mixer"]["mask"]["size"] += 1 if mistake.endswith("+ 1") else -1
    elif mistake == "no bias":
        _swap(monkeypatch, "distance_bias", lambda r1, r2, d: 0.0 * d)
    elif mistake == "bias distance + 1":
        _swap(monkeypatch, "distance_bias", lambda r1, r2, d: bias(r1, r2, d + 1))
    elif mistake == "no value norm":
        _swap(monkeypatch, "value_norm", lambda v, eps: v)
    elif mistake == "no mixing":
        _swap(monkeypatch, "value_mix", lambda v, f, lam: v)
    elif mistake == "mixing swapped":
        _swap(monkeypatch, "value_mix", lambda v, f, lam: lam * v + (1 - lam) * f)
    elif mistake.startswith("first layer"):
        cfg["layers"][1]["mixer"]["v_mix"] = False   # the values then come from a later layer
    elif mistake == "one norm group":
        _swap(monkeypatch, "grouped_rms_norm", lambda x, w, eps, g: norm(x, w, eps, 1))
    elif mistake == "tanh gelu":
        _swap(monkeypatch, "gelu_erf", lambda z: torch.nn.functional.gelu(z, approximate="tanh"))
    elif mistake == "shifted table":
        t["l0.mlp.table"] = t["l0.mlp.table"].roll(1, 0)
    elif mistake == "weights not divided":
        moe = orc.table_moe
        _swap(monkeypatch, "table_moe", lambda h, i, table, ex: moe(h, i, table, ex) * table.shape[1])
    elif mistake == "no q bias":
        t["l0.mix.q.b"] = torch.zeros_like(t["l0.mix.q.b"])
    got = orc.forward(cfg, t, ids)
    assert cases.error(got, want) > 10 * TOL


# --------------------------------------------------------------------------- the plain functions themselves
def test_oracle_mechanisms_on_hand_made_inputs():
    x = torch.tensor([3.0, 4.0, 0.0, 2.0]).double()
    y = orc.grouped_rms_norm(x, torch.ones(4).double(), 0.0, 2)
    assert torch.allclose(y, torch.tensor([3.0, 4.0, 0.0, 2.0]).double() / torch.tensor([12.5, 12.5, 2.0, 2.0]).double().sqrt())
    v = orc.value_norm(torch.tensor([[[3.0, 4.0], [0.0, 2.0]]]).double(), 0.0)
    assert torch.allclose(v[0, 0], torch.tensor([3.0, 4.0]).double() / 12.5 ** 0.5)
    # equal scores: a window of two averages the values of the token and the one before it
    k = torch.zeros(4, 1, 3).double()
    vals = torch.arange(4).double().reshape(4, 1, 1)
    o = orc.windowed_attention(k, k, vals, 1.0, 2, torch.zeros(1).double(), torch.zeros(1).double())
    assert o[:, 0, 0].tolist() == [0.0, 0.5, 1.5, 2.5]
    # r1 = 1, r2 = 1: a key at distance d weighs 1 / (1 + d)
    o = orc.windowed_attention(k, k, vals, 1.0, 3, torch.ones(1).double(), torch.ones(1).double())
    assert abs(float(o[3, 0, 0]) - (3 + 2 / 2 + 1 / 3) / (1 + 1 / 2 + 1 / 3)) < 1e-12


# --------------------------------------------------------------------------- op definitions used on CPU
def test_decode_definition_reads_only_its_window_and_skips_idle_slots():
    g = torch.Generator().manual_seed(0)
    kc, vc = torch.randn(6, 1, 4, 8, generator=g), torch.randn(6, 1, 4, 8, generator=g)
    table = torch.tensor([[3, 1, 5], [0, 0, 0]], dtype=torch.int32)
    q = torch.randn(2, 2, 8, generator=g)
    r = torch.rand(2, generator=g)
    a = sops.window_attn(q, kc, vc, table, 0.3, 5, r, r, seq_lens=torch.tensor([11, 0], dtype=torch.int32))
    assert float(a[1].abs().max()) == 0.0
    kc2, vc2 = kc.clone(), vc.clone()
    kc2[3], vc2[3], kc2[1, :, :2] = 99.0, 99.0, 99.0     # positions 0..5: position 6 is the oldest visible key
    vc2[5, :, 3] = 99.0                                  # position 11: beyond the last token
    b = sops.window_attn(q, kc2, vc2, table, 0.3, 5, r, r, seq_lens=torch.tensor([11, 0], dtype=torch.int32))
    assert torch.equal(a, b)
    kc2[1, :, 2] = 99.0
    assert not torch.equal(a, sops.window_attn(q, kc2, vc2, table, 0.3, 5, r, r, seq_lens=torch.tensor([11, 0], dtype=torch.int32)))


def test_tiles_cover_portions():
    tiles = sops.make_tiles([(0, 0, 20, 5), (3, 20, 1, 0), (1, 21, 33, 100)], 16)
    assert tiles == [(0, 0, 16, 5), (0, 16, 4, 21), (3, 20, 1, 0), (1, 21, 16, 100), (1, 37, 16, 116), (1, 53, 1, 132)]


# --------------------------------------------------------------------------- configuration and checkpoints
def test_config_round_trip_and_registry(tmp_path):
    for name, doc in cases.CONFIGS.items():
        cfg = lederax_config_from_dict(doc)
        assert lederax_config_from_dict(cfg.to_dict()) == cfg
        assert cfg.n_layers == len(doc["layers"])
    assert is_stack_name("lederax-tiny") and not is_stack_name("tiny")
    big = get_model_config("lederax-8b")
    nano = get_model_config("Cosmos3-Nano")
    m, f = big.layers[0].mixer, big.layers[0].mlp
    assert (big.d_model, m.heads, m.kv_heads, m.dim) == (nano.d_model, nano.n_heads, nano.n_kv_heads, nano.head_dim)
    assert 2 * f.top * f.ff == 3 * nano.ffn_dim          # as many active feed-forward parameters
    bad = copy.deepcopy(cases.CONFIGS["mixed"])
    bad["layers"][1]["mixer"]["vdim"] = 16               # cannot be mixed with the first layer's values
    with pytest.raises(ValueError, match="mixed values"):
        lederax_config_from_dict(bad)
    for key, val, match in (("type", "recurrent", "mixer type"),):
        bad = copy.deepcopy(cases.CONFIGS["mixed"])
        bad["layers"][0][key] = val
        with pytest.raises(ValueError, match=match):
            lederax_config_from_dict(bad)
    (tmp_path / "config.json").write_text(json.dumps({"text_config": {}}))
    assert stack_config_from_dir(tmp_path) is None and not is_stack_name(str(tmp_path))


def test_checkpoints_load_save_and_are_checked(tmp_path):
    cfg = cases.CONFIGS["late_mix"]
    t = cases.weights(cfg, 4)
    src = cases.write(cfg, t, tmp_path / "a")
    m = load_stack(src, torch.bfloat16)
    views = m.checkpoint_views()
    assert set(views) == set(t) - {"l0.mix.vmix"}        # a layer that does not mix has no factor
    for k, v in views.items():
        assert torch.equal(v.float(), t[k].float()), k
    m.save(tmp_path / "b")
    again = load_stack(tmp_path / "b", torch.float32)
    for k, v in again.checkpoint_views().items():
        assert torch.equal(v.float(), t[k].float()), k
    missing = {k: v for k, v in t.items() if k != "l1.mix.r2"}
    with pytest.raises(KeyError, match="r2"):
        load_stack(cases.write(cfg, missing, tmp_path / "c"), torch.float32)
    wrong = dict(t, **{"l1.mlp.table": t["l1.mlp.table"] + 5})
    with pytest.raises(ValueError, match="experts that do not exist"):
        load_stack(cases.write(cfg, wrong, tmp_path / "d"), torch.float32)
    no_first = {k: v for k, v in t.items() if k != "l1.mix.vmix"}   # the first mixing layer's factor is never read
    ids = cases.tokens(cfg, 12)
    a = cases.feed(cases.decoder(cases.write(cfg, no_first, tmp_path / "e"), torch.float32, "cpu"), 0, ids, [12])
    assert cases.error(a, orc.forward(cfg, t, ids)) < TOL


def test_random_weights_and_bad_tokens():
    m = load_stack("lederax-tiny", torch.float32, n_layers=1)
    assert isinstance(m, StackModel) and len(m.layers) == 1
    tab = m.layers[0].table
    assert all(len(set(r)) == len(r) for r in tab.tolist())
    from cosmos_b200.serve.decoder import StackDecoder
    dec = StackDecoder(m, 4, max_batch=1, max_len=16)
    assert dec.cache.reserve(0, 3)
    with pytest.raises(ValueError, match="vocabulary"):
        dec.run_portions([(0, [1, 2, 300], 0, [])])
    with pytest.raises(ValueError, match="reserved"):
        dec.run_portions([(0, [1] * 9, 0, [])])


# --------------------------------------------------------------------------- trace replay and command line
def test_trace_replay_writes_the_wanted_logits(tmp_path):
    import numpy as np
    cfg = cases.CONFIGS["mixed"]
    t = cases.weights(cfg, 5)
    model = cases.write(cfg, t, tmp_path / "model")
    a, b = cases.tokens(cfg, 19, 1), cases.tokens(cfg, 8, 2)
    steps = [{"step": 0, "entries": [{"id": "a", "tokens": a[:11], "want": [10, 2]}], "end": []},
             {"step": 1, "entries": [{"id": "a", "tokens": a[11:13], "want": []}], "end": []},
             {"step": 2, "entries": [{"id": "a", "tokens": a[13:14], "want": [0]}, {"id": "b", "tokens": b, "want": [7]}], "end": ["b"]},
             {"step": 3, "entries": [{"id": "a", "tokens": a[14:], "want": [4]}], "end": ["a"]},
             {"step": 4, "entries": [{"id": "a", "tokens": b, "want": [0, 7]}], "end": ["a"]}]
    r = subprocess.run([sys.executable, str(ROOT / "bin" / "trace_run"), "--model", str(model), "--dtype", "float32", "--device",
                        "cpu", "--out", str(tmp_path / "out"), "--max-tokens", "40", "--page-size", "4"],
                       input="".join(json.dumps(s) + "\n" for s in steps), capture_output=True, text=True, timeout=300)
    assert r.returncode == 0, r.stderr[-2000:]
    assert [l for l in r.stdout.splitlines() if l.startswith("done")] == [f"done {i}" for i in range(5)]
    la, lb = orc.forward(cfg, t, a), orc.forward(cfg, t, b)
    want = {0: la[[10, 2]], 2: torch.stack([la[13], lb[7]]), 3: la[[18]], 4: lb[[0, 7]]}
    for s, w in want.items():
        got = torch.from_numpy(np.fromfile(tmp_path / "out" / f"{s}.f32", dtype="<f4")).reshape(w.shape)
        assert cases.error(got, w) < TOL, s
    assert not (tmp_path / "out" / "1.f32").exists()


def test_command_line_generates_text_with_a_stack(tmp_path):
    from cosmos_b200.scripts import inference
    spec = tmp_path / "specs.jsonl"
    spec.write_text("\n".join(json.dumps({"model_mode": "reasoner", "name": n, "prompt": p, "max_new_tokens": k, "do_sample": False})
                              for n, p, k in (("a", "hello", 6), ("b", "a longer question about nothing", 3))))
    load_stack("lederax-tiny", torch.float32, n_layers=1).save(tmp_path / "ckpt")
    for model in ("lederax-tiny", str(tmp_path / "ckpt")):
        out = tmp_path / f"out{len(model)}"
        assert inference.main(["-i", str(spec), "-o", str(out), "--checkpoint-path", model, "--device", "cpu", "--benchmark"]) == 0
        assert (out / "a" / "reasoner_text.txt").exists() and (out / "b" / "reasoner_text.txt").exists()
        bench = json.loads((out / "benchmark.json").read_text())
        assert [r["completion_tokens"] <= k for r, k in zip(bench["samples"], (6, 3))] == [True, True]
    spec.write_text(json.dumps({"model_mode": "text2video", "name": "v", "prompt": "x", "resolution": "256"}))
    assert inference.main(["-i", str(spec), "-o", str(tmp_path / "o2"), "--checkpoint-path", "lederax-tiny", "--device", "cpu"]) == 2


def test_server_answers_chat_requests_with_a_stack():
    from types import SimpleNamespace

    from cosmos_b200.serve.server import stack_server
    srv = stack_server(SimpleNamespace(model="lederax-tiny", max_num_seqs=2, max_model_len=128), None, torch.float32)
    try:
        body = {"messages": [{"role": "user", "content": "hi there"}], "max_tokens": 7, "temperature": 0}
        a, b = srv.chat_completions(dict(body)), srv.chat_completions(dict(body, seed=3))
        assert a["choices"][0]["message"]["content"] == b["choices"][0]["message"]["content"]
        assert a["usage"]["completion_tokens"] <= 7 and a["choices"][0]["finish_reason"] in ("stop", "length")
        with pytest.raises(Exception, match="text only"):
            srv.chat_completions({"messages": [{"role": "user", "content": [{"type": "image_url", "image_url": {"url": "x"}}]}]})
    finally:
        srv.batch_engine.close()
