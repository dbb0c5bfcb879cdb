"""Plain, slow Lederax in float64 (or float32), one function per mechanism, written from the equations. Nothing here
is shared with the product: the tests compare the framework's kernels, cache and scheduler with it.

A model is a config dictionary (the keys of config.json) and a dictionary of tensors by checkpoint name. Notation:
x[t] residual stream of token t, h normed input, i a query's position, j a key's position."""
import math

import torch


def grouped_rms_norm(x, w, eps, groups):
    """RMS norm over blocks of the last axis: x viewed as [.., groups, d / groups], normed along the last of these, times w."""
    parts = x.reshape(*x.shape[:-1], groups, x.shape[-1] // groups)
    parts = parts / torch.sqrt((parts * parts).mean(-1, keepdim=True) + eps)
    return parts.reshape(x.shape) * w


def linear(x, w, b=None):
    y = x @ w.t()
    return y if b is None else y + b


def value_norm(v, eps):
    """v [tokens, kv heads, vdim], each head divided by its root mean square, no weight."""
    return v / torch.sqrt((v * v).mean(-1, keepdim=True) + eps)


def value_mix(v, v_first, lam):
    return (1.0 - lam) * v + lam * v_first


def distance_bias(r1, r2, dist):
    """What is taken off the score of a head at distance dist >= 0."""
    return r1 * torch.log1p(r2 * dist)


def windowed_attention(q, k, v, scale, window, r1, r2):
    """q [n, H, dim], k [n, G, dim], v [n, G, vdim] of one whole sequence; query i sees 0 <= i - j < window."""
    n, heads, _ = q.shape
    per = heads // k.shape[1]
    out = q.new_zeros(n, heads, v.shape[-1])
    for h in range(heads):
        kh, vh = k[:, h // per], v[:, h // per]
        for i in range(n):
            lo = max(0, i - window + 1)
            dist = torch.arange(i - lo, -1, -1, dtype=q.dtype)
            s = kh[lo:i + 1] @ q[i, h] * scale - distance_bias(r1[h], r2[h], dist)
            p = torch.exp(s - s.max())
            out[i, h] = (p / p.sum()) @ vh[lo:i + 1]
    return out


def gelu_erf(z):
    return 0.5 * z * (1.0 + torch.erf(z / math.sqrt(2.0)))


def table_moe(h, ids, table, experts):
    """experts: list of (up, down). Token t goes to the experts table[ids[t]], each with weight 1 / top."""
    out = torch.zeros_like(h)
    top = table.shape[1]
    for t in range(h.shape[0]):
        for e in table[ids[t]].tolist():
            up, down = experts[e]
            out[t] += linear(gelu_erf(linear(h[t], up)), down) / top
    return out


def forward(cfg, tensors, ids, dtype=torch.float64, layers_out=None, values_out=None):
    """Whole-sequence logits [n, vocab]. `layers_out` (a list) receives the residual stream after every layer."""
    w = {k: (t if t.dtype in (torch.int32, torch.int64) else t.to(dtype)) for k, t in tensors.items()}
    ids = torch.as_tensor(ids, dtype=torch.long)
    eps, groups = cfg["norm"]["eps"], cfg["norm"].get("groups", 1)
    x = w["embed"][ids] * cfg["embedding"]["scale"]
    v_first = None
    for li, layer in enumerate(cfg["layers"]):
        m, pre = layer["mixer"], f"l{li}."
        h = grouped_rms_norm(x, w[pre + "norm1"], eps, groups)
        n = h.shape[0]
        q = linear(h, w[pre + "mix.q"], w[pre + "mix.q.b"]).reshape(n, m["heads"], m["dim"])
        k = linear(h, w[pre + "mix.k"], w[pre + "mix.k.b"]).reshape(n, m["kv_heads"], m["dim"])
        v = linear(h, w[pre + "mix.v"], w[pre + "mix.v.b"]).reshape(n, m["kv_heads"], m["vdim"])
        v = value_norm(v, eps)
        if m.get("v_mix"):
            if v_first is None:
                v_first = v
            else:
                v = value_mix(v, v_first, w[pre + "mix.vmix"])
        if values_out is not None:
            values_out.append(v)
        o = windowed_attention(q, k, v, m["scale"], m["mask"]["size"], w[pre + "mix.r1"], w[pre + "mix.r2"])
        x = x + linear(o.reshape(n, -1), w[pre + "mix.o"])
        if layer["mlp"] is not None:
            h = grouped_rms_norm(x, w[pre + "norm2"], eps, groups)
            ne = layer["mlp"]["router"]["experts"]
            experts = [(w[f"{pre}mlp.e{e}.up"], w[f"{pre}mlp.e{e}.down"]) for e in range(ne)]
            x = x + table_moe(h, ids, w[pre + "mlp.table"], experts)
        if layers_out is not None:
            layers_out.append(x)
    return linear(grouped_rms_norm(x, w["final.norm"], eps, groups), w["head"])
