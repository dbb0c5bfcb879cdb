"""Small Mererax models for the tests: configurations as config.json dictionaries with sizes that all differ, and random weights
whose mechanisms show in the logits (peaky attention, distinct slopes, gates on both sides of zero, slow and fast decays)."""
import json

from safetensors.torch import save_file

from tests import oracle_mererax as orc


def par(heads=4, kv=2, dim=12, temp=(0.4, 8), scale=0.9, mem=3, mdim=10, mvdim=22, cap=7.0, ff=26, of=None):
    left = {"heads": heads, "kv_heads": kv, "dim": dim, "vdim": dim, "scale": scale}
    if temp:
        left["q_temp"] = {"coef": temp[0], "every": temp[1]}
    entry = {"type": "parallel", "mixer": {"left": left, "right": {"heads": mem, "dim": mdim, "vdim": mvdim, "gate_cap": cap}},
             "mlp": None if ff is None else {"kind": "dense", "ff": ff}}
    return entry if of is None else dict(entry, weights_of=of)


def scan(inner=44, state=5, rank=3, conv=3, ff=30, of=None):
    entry = {"type": "mamba1", "mixer": {"inner": inner, "state": state, "dt_rank": rank, "conv": conv},
             "mlp": None if ff is None else {"kind": "dense", "ff": ff}}
    return entry if of is None else dict(entry, weights_of=of)


def config(layers, vocab=53, width=36, eps=1e-5, scale=3.0):
    return {"architecture": "Mererax", "vocab": vocab, "width": width, "embedding": {"scale": scale}, "norm": {"eps": eps},
            "layers": layers}


CONFIGS = {
    # attention first and last, shared weights with caches and states of their own
    "mixed": config([par(), scan(), par(heads=6, kv=3, dim=10, temp=(0.7, 5), mem=2, mdim=7, mvdim=40, cap=3.0, ff=19), par(of=0),
                     scan(of=1)]),
    # layers without a feed-forward, no temperature, one head of everything, one tap, one state
    "bare": config([scan(inner=24, state=1, rank=1, conv=1, ff=None), par(heads=1, kv=1, dim=16, temp=None, mem=1, mdim=16, mvdim=9, ff=None),
                    scan(inner=17, state=9, rank=5, conv=2, ff=11), par(heads=5, kv=1, dim=6, scale=1.3, mem=4, mdim=3, mvdim=33, ff=None)],
                   width=30, vocab=61, eps=1e-3),
    # weights taken from a later layer, and through another layer
    "chain": config([scan(inner=40, state=18, rank=9, conv=6, of=2), par(of=3), scan(inner=40, state=18, rank=9, conv=6), par(of=4), par()],
                    width=40, scale=2.0),
    # shapes that the tensor-core kernels take (with bf16 on a GPU)
    "tc": config([scan(inner=208, state=16, rank=24, conv=4, ff=72), par(heads=8, kv=2, dim=64, scale=0.2, temp=(0.3, 40), mem=2, mdim=64,
                                                                       mvdim=128, cap=9.0, ff=144),
                  par(heads=2, kv=2, dim=128, scale=0.15, temp=(0.2, 64), mem=3, mdim=128, mvdim=64, cap=15.0, ff=None), scan(of=0, inner=208,
                  state=16, rank=24, conv=4, ff=72)], vocab=200, width=192),
    # products long enough that a few rows split K: the kernels behind them add up partial sums
    "wide": config([scan(inner=536, state=12, rank=20, conv=4, ff=528), par(heads=6, kv=2, dim=88, scale=0.1, temp=(0.3, 16), mem=2, mdim=64, mvdim=288,
                                                                       cap=8.0, ff=544)], vocab=150, width=520),
}


def weights(cfg, seed=0):
    return orc.random_tensors(cfg, seed)


def write(cfg, tensors, path):
    path.mkdir(parents=True, exist_ok=True)
    (path / "config.json").write_text(json.dumps(cfg))
    save_file({k: v.contiguous() for k, v in tensors.items()}, str(path / "model.safetensors"))
    return path
