"""Plain, slow Mererax in float64 (or float32), one function per mechanism, written from the equations. Nothing here is
shared with the product: the tests compare the framework's kernels, cache, state and scheduler with it.

A model is a config dictionary (the keys of config.json) and a dictionary of tensors by checkpoint name. Notation:
x[t] residual stream of token t, h normed input, i a query's position, j a key's position, S a recurrent state."""
import math

import torch


def linear(x, w):
    return x @ w.t()


def unit_rms(x, eps):
    """x divided by its root mean square along the last axis."""
    return x / torch.sqrt((x * x).mean(-1, keepdim=True) + eps)


def one_plus_norm(x, w, eps):
    return unit_rms(x, eps) * (1.0 + w)


def sinusoid(positions, width):
    """[tokens, width] in float64: sin at even entries, cos at odd ones, one frequency a pair."""
    out = torch.zeros(len(positions), width, dtype=torch.float64)
    for e in range(width):
        angle = positions.double() * 10000.0 ** (-(e - e % 2) / width)
        out[:, e] = torch.cos(angle) if e % 2 else torch.sin(angle)
    return out


def temperature(p, coef, every):
    return 1.0 + coef * math.log((p + 1) // every + 1)


def slope(h, heads):
    return 2.0 ** (-8.0 * (h + 1) / heads)


def biased_attention(q, k, v, scale, first=0):
    """q [n, H, dim], k [n, G, dim], v [n, G, vdim] of one whole sequence; every query sees itself and all before it. Only
    the rows from `first` on are computed."""
    n, heads, _ = q.shape
    per = heads // k.shape[1]
    out = q.new_zeros(n, heads, v.shape[-1])
    for h in range(heads):
        kh, vh = k[:, h // per], v[:, h // per]
        for i in range(first, n):
            dist = torch.arange(i, -1, -1, dtype=q.dtype)
            s = kh[:i + 1] @ q[i, h] * scale - slope(h, heads) * dist
            p = torch.exp(s - s.max())
            out[i, h] = (p / p.sum()) @ vh[:i + 1]
    return out


def attention_branch(m, t, p, h, eps, first=0):
    n, heads, groups, dim = h.shape[0], m["heads"], m["kv_heads"], m["dim"]
    k_raw = linear(h, t[p + "k"])
    q = unit_rms(linear(h, t[p + "q"]), eps) * t[p + "q.norm"]
    k = unit_rms(k_raw, eps) * t[p + "k.norm"]
    if m.get("q_temp"):
        q = q * torch.tensor([temperature(i, m["q_temp"]["coef"], m["q_temp"]["every"]) for i in range(n)], dtype=h.dtype)[:, None]
    o = biased_attention(q.reshape(n, heads, dim), k.reshape(n, groups, dim), k_raw.reshape(n, groups, dim), m["scale"], first)
    return linear(o.reshape(n, -1), t[p + "o"])


def mlstm(q, k, v, i, f):
    """q, k [n, H, dim] (q already scaled), v [n, H, vdim], i, f [n, H] log gates -> [n, H, vdim]."""
    n, heads, dim = q.shape
    out = q.new_zeros(n, heads, v.shape[-1])
    for h in range(heads):
        s, z, m = q.new_zeros(dim, v.shape[-1]), q.new_zeros(dim), q.new_zeros(())
        for t in range(n):
            m_new = torch.maximum(f[t, h] + m, i[t, h])
            keep, take = torch.exp(f[t, h] + m - m_new), torch.exp(i[t, h] - m_new)
            s = keep * s + take * torch.outer(k[t, h], v[t, h])
            z = keep * z + take * k[t, h]
            m = m_new
            out[t, h] = (s.t() @ q[t, h]) / (torch.maximum((z @ q[t, h]).abs(), torch.exp(-m)) + 1e-6)
    return out


def mlstm_gates(raw_i, raw_f, cap):
    i = cap * torch.tanh(raw_i / cap)
    f = -torch.nn.functional.softplus(-cap * torch.tanh(raw_f / cap))
    return i, f


def mlstm_branch(m, t, p, h, eps):
    n, heads, dim, vdim = h.shape[0], m["heads"], m["dim"], m["vdim"]
    q = linear(h, t[p + "q"]).reshape(n, heads, dim) * dim ** -0.5
    k = linear(h, t[p + "k"]).reshape(n, heads, dim)
    v = linear(h, t[p + "v"]).reshape(n, heads, vdim)
    i, f = mlstm_gates(linear(h, t[p + "i"]) + t[p + "i.b"], linear(h, t[p + "f"]) + t[p + "f.b"], m["gate_cap"])
    o = unit_rms(mlstm(q, k, v, i, f), eps).reshape(n, -1) * t[p + "norm"] * torch.sigmoid(linear(h, t[p + "g"]))
    return linear(o, t[p + "o"])


def parallel_mixer(m, t, p, h, eps, first=0):
    left = attention_branch(m["left"], t, p + "left.", h, eps, first)
    right = mlstm_branch(m["right"], t, p + "right.", h, eps)
    return 0.5 * (unit_rms(left, eps) * t[p + "left.out"] + unit_rms(right, eps) * t[p + "right.out"])


def causal_conv(x, w, b):
    """x [n, channels], w [channels, taps] (last column: the current token)."""
    n, taps = x.shape[0], w.shape[1]
    out = b.expand(n, -1).clone()
    for t in range(n):
        for j in range(taps):
            s = t - (taps - 1 - j)
            if s >= 0:
                out[t] = out[t] + w[:, j] * x[s]
    return out


def silu(z):
    return z * torch.sigmoid(z)


def selective_scan(u, dt, a, b, c, d):
    """u, dt [n, inner], a [inner, state] (negative), b, c [n, state], d [inner] -> y [n, inner]."""
    s = torch.zeros_like(a)
    out = torch.zeros_like(u)
    for t in range(u.shape[0]):
        s = torch.exp(dt[t][:, None] * a) * s + (dt[t] * u[t])[:, None] * b[t][None]
        out[t] = s @ c[t] + d * u[t]
    return out


def mamba_mixer(m, t, p, h):
    inner, rank, state = m["inner"], m["dt_rank"], m["state"]
    xz = linear(h, t[p + "in"])
    u, z = silu(causal_conv(xz[:, :inner], t[p + "conv"], t[p + "conv.b"])), xz[:, inner:]
    dbc = linear(u, t[p + "x"])
    dt = torch.nn.functional.softplus(linear(dbc[:, :rank], t[p + "dt"]) + t[p + "dt.b"])
    y = selective_scan(u, dt, -torch.exp(t[p + "A_log"]), dbc[:, rank:rank + state], dbc[:, rank + state:], t[p + "D"])
    return linear(y * silu(z), t[p + "o"])


def dense(t, p, h):
    return linear(silu(linear(h, t[p + "gate"])) * linear(h, t[p + "up"]), t[p + "down"])


def source_layer(cfg, i):
    """The layer whose tensors layer i uses."""
    while cfg["layers"][i].get("weights_of") is not None:
        i = cfg["layers"][i]["weights_of"]
    return i


def forward(cfg, tensors, tokens, dtype=torch.float64, layers_out=None, first=0):
    """Logits [len(tokens), vocab] of one sequence from its start. `first`: attention rows before it are left out (only right
    when no later layer needs them, for tests that look at the last rows of a one-attention-layer model)."""
    t = {k: v.to(dtype) if v.is_floating_point() else v for k, v in tensors.items()}
    tok = torch.as_tensor(tokens, dtype=torch.long)
    eps = cfg["norm"]["eps"]
    x = t["embed"][tok] * cfg["embedding"]["scale"] + sinusoid(torch.arange(len(tok)), cfg["width"]).to(dtype)
    for i, layer in enumerate(cfg["layers"]):
        p = f"l{source_layer(cfg, i)}."
        h = one_plus_norm(x, t[p + "norm1"], eps)
        if layer["type"] == "mamba1":
            y = mamba_mixer(layer["mixer"], t, p + "mix.", h)
        else:
            y = parallel_mixer(layer["mixer"], t, p + "mix.", h, eps, first)
        if layer.get("mlp") is not None:
            y = y + dense(t, p + "mlp.", one_plus_norm(x, t[p + "norm2"], eps))
        x = x + y
        if layers_out is not None:
            layers_out.append(x.clone())
    return linear(one_plus_norm(x, t["final.norm"], eps), t["embed"])


def random_tensors(cfg, seed, std=None):
    """Random weights (bf16-representable) for a config dictionary, by checkpoint name. Spread so that every mechanism shows:
    decays from slow to fast, gates on both sides of zero, norm weights away from their neutral values."""
    g = torch.Generator().manual_seed(seed)

    def rnd(*s, scale=1.0):
        return torch.randn(*s, generator=g) * scale

    d, out = cfg["width"], {}
    mat = lambda o, i, f=1.0: rnd(o, i, scale=(std or f / math.sqrt(i)))  # noqa: E731
    out["embed"] = rnd(cfg["vocab"], d, scale=0.3)
    out["final.norm"] = rnd(d, scale=0.2)
    for i, layer in enumerate(cfg["layers"]):
        if layer.get("weights_of") is not None:
            continue
        p, m = f"l{i}.", layer["mixer"]
        out[p + "norm1"] = rnd(d, scale=0.2)
        if layer["type"] == "mamba1":
            inner, rank, state, taps = m["inner"], m["dt_rank"], m["state"], m["conv"]
            out[p + "mix.in"] = mat(2 * inner, d)
            out[p + "mix.conv"], out[p + "mix.conv.b"] = rnd(inner, taps, scale=0.5), rnd(inner, scale=0.2)
            out[p + "mix.x"] = mat(rank + 2 * state, inner, 2.0)
            out[p + "mix.dt"] = mat(inner, rank)
            out[p + "mix.dt.b"] = rnd(inner) - 2.0
            out[p + "mix.A_log"] = torch.rand(inner, state, generator=g) * 3.0 - 1.5
            out[p + "mix.D"] = rnd(inner)
            out[p + "mix.o"] = mat(d, inner)
        else:
            a, r = m["left"], m["right"]
            q, k = a["heads"] * a["dim"], a["kv_heads"] * a["dim"]
            out[p + "mix.left.q"], out[p + "mix.left.k"] = mat(q, d), mat(k, d)
            out[p + "mix.left.q.norm"], out[p + "mix.left.k.norm"] = 1 + rnd(q, scale=0.2), 1 + rnd(k, scale=0.2)
            out[p + "mix.left.o"] = mat(d, a["heads"] * a["vdim"])
            hd, hv = r["heads"] * r["dim"], r["heads"] * r["vdim"]
            # queries and keys lean the same way: a q . k near zero flips the sign of a young memory's normed output, and
            # 16-bit rounding would then decide it
            out[p + "mix.right.q"] = mat(hd, d)
            out[p + "mix.right.k"] = 0.85 * out[p + "mix.right.q"] + mat(hd, d, 0.5)
            out[p + "mix.right.v"], out[p + "mix.right.g"] = mat(hv, d), mat(hv, d)
            out[p + "mix.right.o"], out[p + "mix.right.norm"] = mat(d, hv), 1 + rnd(hv, scale=0.2)
            out[p + "mix.right.i"], out[p + "mix.right.f"] = mat(r["heads"], d), mat(r["heads"], d)
            out[p + "mix.right.i.b"], out[p + "mix.right.f.b"] = rnd(r["heads"]) - 2.0, rnd(r["heads"]) + 2.0
            out[p + "mix.left.out"], out[p + "mix.right.out"] = 1 + rnd(d, scale=0.2), 1 + rnd(d, scale=0.2)
        if layer.get("mlp") is not None:
            ff = layer["mlp"]["ff"]
            out[p + "norm2"] = rnd(d, scale=0.2)
            out[p + "mlp.gate"], out[p + "mlp.up"], out[p + "mlp.down"] = mat(ff, d), mat(ff, d), mat(d, ff)
    return {k: v.to(torch.bfloat16) for k, v in out.items()}
