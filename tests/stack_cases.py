"""Small Lederax models for the tests: configurations as config.json dictionaries and random weights whose mechanisms show
in the logits (peaky scores, biases, distinct mixing factors), written to a directory that the product's loader reads."""
import json

import torch
from safetensors.torch import save_file


def layer(heads=4, kv=2, dim=12, vdim=20, window=9, v_mix=True, ff=28, experts=5, top=2, scale=None):
    return {"type": "attention",
            "mixer": {"heads": heads, "kv_heads": kv, "dim": dim, "vdim": vdim, "scale": scale or dim ** -0.5,
                      "mask": {"size": window}, "v_mix": v_mix},
            "mlp": None if ff is None else {"kind": "moe", "expert": {"ff": ff}, "router": {"experts": experts, "top": top}}}


def config(layers, vocab=53, width=36, groups=3, eps=1e-5, scale=0.7):
    return {"architecture": "Lederax", "vocab": vocab, "width": width, "embedding": {"scale": scale},
            "norm": {"eps": eps, "groups": groups}, "layers": layers}


CONFIGS = {
    # every size differs from its neighbours; windows around the page sizes of the tests
    "mixed": config([layer(), layer(heads=6, kv=2, dim=10, vdim=20, window=4, experts=3, top=1), layer(window=17, ff=33, top=3)]),
    # the first layer does not mix, the second gives the values, one layer has no feed-forward
    "late_mix": config([layer(v_mix=False, heads=2, kv=1, dim=16, vdim=8), layer(heads=3, kv=3, vdim=14), layer(heads=6, kv=3, vdim=14, ff=None),
                        layer(heads=3, kv=3, vdim=14, window=1)], width=40, groups=1),
    "no_mix": config([layer(v_mix=False, window=6), layer(v_mix=False, window=300, heads=5, kv=1, dim=9, vdim=11)], vocab=61, width=30, groups=5),
    # one expert that everybody uses; all experts used by everybody
    "all_experts": config([layer(experts=1, top=1, ff=8), layer(experts=4, top=4, ff=16)], width=32, groups=8, scale=1.0),
    # shapes that the tensor-core kernels take (with bf16 on a GPU)
    "tc": config([layer(heads=4, kv=2, dim=64, vdim=64, window=40), layer(heads=16, kv=2, dim=40, vdim=64, window=90, experts=7, top=2, ff=72),
                  layer(heads=2, kv=2, dim=128, vdim=64, window=33)], vocab=200, width=192, groups=2),
}


def weights(cfg, seed=0, loud=2.2):
    """bf16 tensors by checkpoint name."""
    g = torch.Generator().manual_seed(seed)
    d, t = cfg["width"], {}

    def mat(rows, cols, gain=1.0):
        return torch.randn(rows, cols, generator=g) * gain * cols ** -0.5

    t["embed"] = torch.randn(cfg["vocab"], d, generator=g)
    ints = {}
    for i, entry in enumerate(cfg["layers"]):
        m, f, p = entry["mixer"], entry["mlp"], f"l{i}."
        h, kv, dim, vdim = m["heads"], m["kv_heads"], m["dim"], m["vdim"]
        for n, rows, gain in (("q", h * dim, loud), ("k", kv * dim, loud), ("v", kv * vdim, 1.0)):
            t[f"{p}mix.{n}"] = mat(rows, d, gain)
            t[f"{p}mix.{n}.b"] = torch.randn(rows, generator=g) * 0.4
        t[p + "mix.vmix"] = torch.tensor(0.2 + 0.15 * i)
        t[p + "mix.r1"] = torch.rand(h, generator=g) * 2 + 0.02
        t[p + "mix.r2"] = torch.rand(h, generator=g) * 0.5 + 0.05
        t[p + "mix.o"] = mat(d, h * vdim)
        t[p + "norm1"] = 1 + 0.3 * torch.randn(d, generator=g)
        if f is not None:
            e, top, ff = f["router"]["experts"], f["router"]["top"], f["expert"]["ff"]
            t[p + "norm2"] = 1 + 0.3 * torch.randn(d, generator=g)
            for k in range(e):
                t[f"{p}mlp.e{k}.up"], t[f"{p}mlp.e{k}.down"] = mat(ff, d, 1.5), mat(d, ff, 1.5)
            ints[p + "mlp.table"] = torch.rand(cfg["vocab"], e, generator=g).argsort(1)[:, :top].to(torch.int32).contiguous()
    t["final.norm"] = 1 + 0.3 * torch.randn(d, generator=g)
    t["head"] = mat(cfg["vocab"], d)
    return {**{k: v.to(torch.bfloat16).contiguous() for k, v in t.items()}, **ints}


def write(cfg, tensors, path):
    path.mkdir(parents=True, exist_ok=True)
    (path / "config.json").write_text(json.dumps(cfg))
    save_file(tensors, str(path / "model.safetensors"))
    return path


def tokens(cfg, n, seed=0):
    return torch.randint(0, cfg["vocab"], (n,), generator=torch.Generator().manual_seed(seed)).tolist()


def error(got, want):
    """Root mean square difference per row with the mean taken off, over the spread of the expected logits; the worst row."""
    d = got.double().cpu() - want.double()
    d = d - d.mean(-1, keepdim=True)
    return float((d.pow(2).mean(-1).sqrt() / want.double().std()).max())


def decoder(path, dtype, device, page_size=4, max_len=400, max_batch=4):
    from cosmos_b200.models.stack import load_stack
    from cosmos_b200.serve.decoder import StackDecoder

    return StackDecoder(load_stack(path, dtype, device), page_size, max_batch=max_batch, max_len=max_len)


def feed(dec, seq, ids, cuts, have=0):
    """Runs ids in portions of the given sizes (cycled) and returns the logits of every position."""
    out, o, i = [], 0, 0
    while o < len(ids):
        n = min(cuts[i % len(cuts)], len(ids) - o)
        assert dec.cache.reserve(seq, n)
        out.append(dec.run_portions([(seq, ids[o:o + n], have + o, list(range(n)))]).float().cpu())
        o += n
        i += 1
    return torch.cat(out)
