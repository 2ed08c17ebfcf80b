"""Plain restatement of the Ninisun decoder, one function per mechanism, in one floating-point type.

Nothing here comes from the package: the tests compare the framework with it. A model is a ``dict`` configuration and
a ``dict`` of weights by checkpoint name; ``forward`` runs one whole sequence and returns logits (and, on request, the
residual stream after every layer). Wrong variants for tests that must notice a mistake are planted here (``mutate``),
never on the device.
"""

from __future__ import annotations

import math

import torch


def rms_norm(x, weight, eps):
    return x / torch.sqrt((x * x).mean(-1, keepdim=True) + eps) * weight


def sigmoid(z):
    return 1.0 / (1.0 + torch.exp(-z))


def gelu_tanh(z):
    return 0.5 * z * (1.0 + torch.tanh(math.sqrt(2.0 / math.pi) * (z + 0.044715 * z * z * z)))


def frequency(base, dims, i, scaling=None, mutate=None):
    """Turn rate of pair i: ``base^(-2i / dims)``; with ``scaling`` (YaRN) pairs that turn fewer than ``slow`` times in
    ``original`` positions are slowed down by ``factor``, those above ``fast`` are left alone, with a ramp over the pair
    index in between."""
    f = float(base) ** (-2.0 * i / dims)
    if not scaling or mutate == "no_scaling":
        return f

    def index_of(turns):
        return dims * math.log(scaling["original"] / (2.0 * math.pi * turns)) / (2.0 * math.log(base))

    lo = max(math.floor(index_of(scaling["fast"])), 0)
    hi = min(math.ceil(index_of(scaling["slow"])), dims - 1)
    ramp = min(max((i - lo) / max(hi - lo, 0.001), 0.0), 1.0)
    return f / scaling["factor"] * ramp + f * (1.0 - ramp)


def rotate(x, positions, rot, mutate=None):
    """x [T, ..., n]: elements 2i and 2i + 1 of the first ``dims`` form a pair that turns with the position."""
    if mutate == "no_rotation" or not rot:
        return x
    dims, out, scaling = rot["dims"], x.clone(), rot.get("scaling")
    grow = 0.1 * math.log(scaling["factor"]) + 1.0 if scaling and mutate != "no_magnitude" else 1.0
    for i in range(dims // 2):
        a = positions.to(torch.float64) * frequency(rot["base"], dims, i, scaling, mutate)
        c, s = (torch.cos(a) * grow).to(x.dtype), (torch.sin(a) * grow).to(x.dtype)
        c, s = (t.view(-1, *[1] * (x.dim() - 2)) for t in (c, s))
        u, v = x[..., 2 * i], x[..., 2 * i + 1]
        out[..., 2 * i], out[..., 2 * i + 1] = u * c - v * s, v * c + u * s
    return out


def visible(n, size=None, keep_first=0):
    """[n, n] mask: which keys (columns) each position sees: the last ``size`` and the first ``keep_first``."""
    i, j = torch.arange(n)[:, None], torch.arange(n)[None]
    ok = j <= i
    return ok if not size else ok & ((i - j < size) | (j < keep_first))


def scores(q, k, scale):
    """[H, T, T] products of the heads' queries with their group's keys. q [T, H, D], k [T, G, D]."""
    k = k.repeat_interleave(q.shape[1] // k.shape[1], 1)
    return torch.einsum("ihd,jhd->hij", q, k) * scale


def weighted(p, v):
    """Weights [H, T, T] over values [T, G, V] -> [T, H, V]."""
    return torch.einsum("hij,jhd->ihd", p, v.repeat_interleave(p.shape[0] // v.shape[1], 1))


def softmax_heads(q, k, v, scale, size=None, keep_first=0):
    s = scores(q, k, scale).masked_fill(~visible(q.shape[0], size, keep_first).to(q.device), float("-inf"))
    e = torch.exp(s - s.amax(-1, keepdim=True))
    return weighted(e / e.sum(-1, keepdim=True), v)


def sigmoid_heads(q, k, v, scale, bias, size=None, keep_first=0):
    p = sigmoid(scores(q, k, scale) + bias[:, None, None])
    return weighted(p * visible(q.shape[0], size, keep_first).to(p), v)


def attention(h, w, n, m, first_v, mutate=None):
    """Windowed layer; ``first_v``: the values that later layers mix in (None in the first such layer)."""
    T = h.shape[0]
    pos = torch.arange(T, device=h.device)
    heads = lambda t, k: (h @ w[f"{n}.{t}"].t()).view(T, k, -1)  # noqa: E731
    q, k, v = heads("q", m["heads"]), heads("k", m["kv_heads"]), heads("v", m["kv_heads"])
    q, k = rotate(q, pos, m["rot"], mutate), rotate(k, pos, m["rot"], mutate)
    if m.get("v_mix"):
        if first_v is None:
            first_v = v
        elif mutate != "no_mixing":
            lam = w[f"{n}.vmix"]
            v = (1.0 - lam) * v + lam * first_v
    mask = m.get("mask") or {}
    size, keep = mask.get("size"), mask.get("keep_first", 0)
    if size and mutate in ("wide_window", "narrow_window"):
        size += 1 if mutate == "wide_window" else -1
    if mutate in ("keep_more", "keep_fewer"):
        keep = max(0, keep + (1 if mutate == "keep_more" else -1))
    return softmax_heads(q, k, v, m["scale"], size, keep).reshape(T, -1) @ w[f"{n}.o"].t(), first_v


def gated_sigmoid_attention(h, w, n, m, mutate=None):
    T = h.shape[0]
    pos = torch.arange(T, device=h.device)

    def heads(t, k):
        b = 0.0 if mutate == "no_bias" else w[f"{n}.{t}.b"]
        return (h @ w[f"{n}.{t}"].t() + b).view(T, k, -1)

    q, k, v = heads("q", m["heads"]), heads("k", m["kv_heads"]), heads("v", m["kv_heads"])
    q, k = rotate(q, pos, m["rot"], mutate), rotate(k, pos, m["rot"], mutate)
    bias = w[f"{n}.pb"] * (0.0 if mutate == "no_score_bias" else 1.0)
    o = softmax_heads(q, k, v, m["scale"]) if mutate == "softmax" else sigmoid_heads(q, k, v, m["scale"], bias)
    if mutate != "no_gate":
        o = o * sigmoid(h @ w[f"{n}.g"].t())[..., None]
    return o.reshape(T, -1) @ w[f"{n}.o"].t()


def delta_step(S, r, w, k, a, v, mutate=None):
    """One token of the generalized delta rule: S [H, D, V]; r, w, k, a [H, D]; v [H, V]."""
    u = k / torch.sqrt((k * k).sum(-1, keepdim=True) + 1e-6)
    seen = torch.einsum("hd,hdv->hv", u, S)
    S = (S if mutate == "no_decay" else w[..., None] * S)
    if mutate != "no_removal":
        S = S - (a * u)[..., None] * seen[:, None]
    S = S + k[..., None] * v[:, None]
    return S, torch.einsum("hd,hdv->hv", r, S)


def delta_rule(r, w, k, a, v, S=None, mutate=None):
    """r, w, k, a [T, H, D], v [T, H, V] -> (o [T, H, V], state after the last token)."""
    S = r.new_zeros(*k.shape[1:], v.shape[-1]) if S is None else S
    out = []
    for t in range(r.shape[0]):
        S, o = delta_step(S, r[t], w[t], k[t], a[t], v[t], mutate)
        out.append(o)
    return torch.stack(out), S


def delta_mixer(h, w, n, m, eps, mutate=None):
    T, H = h.shape[0], m["heads"]
    heads = lambda t: (h @ w[f"{n}.{t}"].t()).view(T, H, -1)  # noqa: E731
    z = torch.tanh(h @ w[f"{n}.w1"].t()) @ w[f"{n}.w2"].t() + w[f"{n}.w0"]
    decay = torch.exp(-math.exp(-0.5) * sigmoid(z)).view(T, H, -1)
    rate = sigmoid(h @ w[f"{n}.a"].t() + w[f"{n}.a.b"]).view(T, H, -1)
    o, _ = delta_rule(heads("r"), decay, heads("k"), rate, heads("v"), mutate=mutate)
    o = o / torch.sqrt((o * o).mean(-1, keepdim=True) + eps)
    return (o.reshape(T, -1) * w[f"{n}.norm"] * sigmoid(h @ w[f"{n}.g"].t())) @ w[f"{n}.o"].t()


def parallel_mixer(h, w, n, m, eps, mutate=None):
    left = gated_sigmoid_attention(h, w, f"{n}.left", m["left"], mutate)
    right = delta_mixer(h, w, f"{n}.right", m["right"], eps, mutate)
    return m["left_scale"] * left + m["right_scale"] * right


def feed_forward(h, w, n):
    return (gelu_tanh(h @ w[f"{n}.gate"].t()) * (h @ w[f"{n}.up"].t())) @ w[f"{n}.down"].t()


def forward(cfg, weights, tokens, dtype=torch.float64, layers=None, mutate=None):
    """tokens: list of ids -> logits [T, vocab]. ``layers``: a list that receives the stream after every layer."""
    w = {k: v.to(dtype) for k, v in weights.items()}
    eps = cfg["norm"]["eps"]
    x = w["embed"][torch.as_tensor(tokens, device=w["embed"].device)]
    first_v = None
    for i, entry in enumerate(cfg["layers"]):
        n, m = f"l{i}", entry["mixer"]

        def add(x, branch, which):
            b = rms_norm(branch, w[f"{n}.norm{which}b"], eps)
            return x + (b if mutate == "no_layer_scale" else b * w[f"{n}.ls{which}"])

        h = rms_norm(x, w[f"{n}.norm1"], eps)
        if entry["type"] == "attention":
            o, first_v = attention(h, w, f"{n}.mix", m, first_v, mutate)
        else:
            o = parallel_mixer(h, w, f"{n}.mix", m, eps, mutate)
        x = add(x, o, 1)
        if entry.get("mlp") is not None:
            x = add(x, feed_forward(rms_norm(x, w[f"{n}.norm2"], eps), w, f"{n}.mlp"), 2)
        if layers is not None:
            layers.append(x.clone())
    return rms_norm(x, w["final.norm"], eps) @ w["embed"].t()


# ------------------------------------------------------------------------------------------------ small models
def windowed(heads, kv_heads, dim, vdim, scale, size, keep_first=0, base=1000.0, dims=None, v_mix=True, mlp=None):
    return {"type": "attention", "mlp": mlp,
            "mixer": {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "scale": scale, "v_mix": v_mix,
                      "mask": {"size": size, "keep_first": keep_first},
                      "rot": {"base": base, "dims": dim if dims is None else dims}}}


def parallel(left, right, scales=(1.0, 1.0), mlp=None):
    """left: (heads, kv_heads, dim, vdim, scale, dims, base, scaling); right: (heads, dim)."""
    H, G, D, V, scale, dims, base, scaling = left
    rot = {"base": base, "dims": dims, **({"scaling": scaling} if scaling else {})}
    return {"type": "parallel", "mlp": mlp,
            "mixer": {"left": {"heads": H, "kv_heads": G, "dim": D, "vdim": V, "scale": scale, "rot": rot},
                      "left_scale": scales[0], "right": {"heads": right[0], "dim": right[1]}, "right_scale": scales[1]}}


def dense(ff):
    return {"kind": "dense", "ff": ff}


def random_config(layers, width, vocab, eps=1e-5):
    return {"architecture": "Ninisun", "layers": layers, "norm": {"eps": eps}, "vocab": vocab, "width": width}


def random_weights(cfg, seed=0, dtype=torch.bfloat16, rank=8):
    g = torch.Generator().manual_seed(seed)
    W = cfg["width"]
    out = {}

    def lin(name, o, i, gain=1.0):
        out[name] = (torch.randn(o, i, generator=g) * gain * i ** -0.5).to(dtype)

    def vec(name, n, mean=1.0, std=0.2):
        out[name] = (mean + std * torch.randn(n, generator=g)).to(dtype)

    out["embed"] = torch.randn(cfg["vocab"], W, generator=g).to(dtype)
    for i, e in enumerate(cfg["layers"]):
        n, m = f"l{i}", e["mixer"]
        for k in ("norm1", "norm1b") + (("norm2", "norm2b") if e.get("mlp") else ()):
            vec(f"{n}.{k}", W)
        vec(f"{n}.ls1", W, 0.6, 0.2)
        if e["type"] == "attention":
            H, G, D, V = (m[k] for k in ("heads", "kv_heads", "dim", "vdim"))
            for k, o in (("q", H * D), ("k", G * D), ("v", G * V)):
                lin(f"{n}.mix.{k}", o, W, 1.5)
            lin(f"{n}.mix.o", W, H * V)
            out[f"{n}.mix.vmix"] = (0.3 + 0.4 * torch.rand((), generator=g)).to(dtype)
        else:
            a, r = m["left"], m["right"]
            H, G, D, V = (a[k] for k in ("heads", "kv_heads", "dim", "vdim"))
            for k, o in (("q", H * D), ("k", G * D), ("v", G * V)):
                lin(f"{n}.mix.left.{k}", o, W, 1.5)
                vec(f"{n}.mix.left.{k}.b", o, 0.0, 0.5)
            vec(f"{n}.mix.left.pb", H, -2.0, 0.7)
            lin(f"{n}.mix.left.g", H, W)
            lin(f"{n}.mix.left.o", W, H * V)
            H, D = r["heads"], r["dim"]
            for k in ("r", "k", "v", "g", "a"):
                lin(f"{n}.mix.right.{k}", H * D, W)
            vec(f"{n}.mix.right.a.b", H * D, 0.0, 0.5)
            lin(f"{n}.mix.right.w1", rank, W)
            lin(f"{n}.mix.right.w2", H * D, rank, 2.0)
            vec(f"{n}.mix.right.w0", H * D, -3.0, 1.5)
            vec(f"{n}.mix.right.norm", H * D)
            lin(f"{n}.mix.right.o", W, H * D)
        if e.get("mlp"):
            vec(f"{n}.ls2", W, 0.6, 0.2)
            F = e["mlp"]["ff"]
            lin(f"{n}.mlp.gate", F, W)
            lin(f"{n}.mlp.up", F, W)
            lin(f"{n}.mlp.down", W, F)
    vec("final.norm", W)
    return out
