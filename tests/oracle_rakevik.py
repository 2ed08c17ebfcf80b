"""Plain restatement of the Rakevik decoder, one function per mechanism, token by token and in one floating-point type.

Nothing here comes from the package: the tests compare the framework with it. A model is a ``dict`` configuration and
a ``dict`` of weights by checkpoint name; ``forward`` runs one whole sequence and returns logits (and, on request, the
residual stream after every layer run). Wrong variants for tests that must notice a mistake are planted here
(``mutate``), never on the device.
"""

from __future__ import annotations

import math

import torch


def rms_norm(x, weight, eps):
    return x / torch.sqrt((x * x).mean(-1, keepdim=True) + eps) * weight


def token_shift(h, mu):
    """h [T, W]: blend every row with the row before it (zeros before the first), element by element."""
    before = torch.cat([torch.zeros_like(h[:1]), h[:-1]])
    return h + (before - h) * mu


def sigmoid(z):
    return 1.0 / (1.0 + torch.exp(-z))


def softplus(z):
    return torch.log1p(torch.exp(-z.abs())) + torch.clamp(z, min=0.0)


def xielu(z, act):
    """Two-branch activation with the raw parameters ``act = (p, q)``."""
    a_pos, a_neg = softplus(act[0]), 0.5 + softplus(act[1])
    neg = a_neg * (torch.expm1(torch.clamp(z, max=0.0)) - z) + 0.5 * z
    return torch.where(z > 0, a_pos * z * z + 0.5 * z, neg)


def hgrn2_scan(q, f, v, state=None):
    """q, f [T, H, D], v [T, H, V] -> (o [T, H, V], state [H, D, V])."""
    T, H, D = q.shape
    s = torch.zeros(H, D, v.shape[-1], dtype=q.dtype) if state is None else state.clone()
    out = torch.empty(T, H, v.shape[-1], dtype=q.dtype)
    for t in range(T):
        s = f[t][:, :, None] * s + (1.0 - f[t])[:, :, None] * v[t][:, None, :]
        out[t] = (s * q[t][:, :, None]).sum(1)
    return out, s


def forget_gate(z, bias, lower):
    return lower + (1.0 - lower) * sigmoid(z + bias)


def hgrn2_mixer(h, w, name, m, eps):
    T = h.shape[0]
    H, D, V = m["heads"], m["dim"], m["vdim"]
    q = h @ w[name + ".q"].T
    q = (q * sigmoid(q)).view(T, H, D)
    f = forget_gate(h @ w[name + ".f"].T, w[name + ".f.b"], w[name + ".lower"]).view(T, H, D)
    v = (h @ w[name + ".v"].T).view(T, H, V)
    o, _ = hgrn2_scan(q, f, v)
    o = rms_norm(o, w[name + ".norm"], eps)
    return o.reshape(T, H * V) @ w[name + ".o"].T


def query_temperature(positions, coef, every):
    return 1.0 + coef * torch.log(torch.floor((positions + 1.0) / every) + 1.0)


def sink_attention(q, k, v, scale, sink=None, mutate=None):
    """q [T, H, D], k [T, G, D], v [T, G, V], causal; ``sink`` [H] joins every denominator once."""
    T, H, _ = q.shape
    G = k.shape[1]
    out = torch.empty(T, H, v.shape[-1], dtype=q.dtype)
    for h in range(H):
        g = h // (H // G) if mutate != "kv_head" else h % G
        s = (q[:, h] @ k[:, g].T) * scale
        s = s.masked_fill(torch.ones(T, T, dtype=torch.bool).triu(1), -math.inf)
        top = s.max(-1, keepdim=True).values
        if sink is not None and mutate != "no_sink":
            top = torch.maximum(top, sink[h])
        p = torch.exp(s - top)
        den = p.sum(-1, keepdim=True)
        if sink is not None and mutate != "no_sink":
            den = den + torch.exp(sink[h] - top)
        out[:, h] = (p / den) @ v[:, g]
    return out


def attention_mixer(h, w, name, m, eps, mutate=None):
    T = h.shape[0]
    H, G, D, V = m["heads"], m["kv_heads"], m["dim"], m["vdim"]
    q = rms_norm((h @ w[name + ".q"].T).view(T, H, D), w[name + ".q.norm"], eps)
    k = rms_norm((h @ w[name + ".k"].T).view(T, G, D), w[name + ".k.norm"], eps)
    v = (h @ w[name + ".v"].T).view(T, G, V)
    temp = m.get("q_temp")
    if temp and mutate != "no_q_temp":
        q = q * query_temperature(torch.arange(T, dtype=h.dtype), temp["coef"], temp["every"])[:, None, None]
    o = sink_attention(q, k, v, m["scale"], w[name + ".sink"], mutate)
    return o.reshape(T, H * V) @ w[name + ".o"].T


MIXERS = {"hgrn2": hgrn2_mixer, "attention": attention_mixer}


def layer(x, w, i, spec, eps, mutate=None):
    L = f"l{i}"
    h = rms_norm(x, w[L + ".norm1"], eps)
    if mutate != "no_shift":
        h = token_shift(h, w[L + ".shift"])
    if spec["type"] == "attention":
        x = x + attention_mixer(h, w, L + ".mix", spec["mixer"], eps, mutate)
    else:
        x = x + hgrn2_mixer(h, w, L + ".mix", spec["mixer"], eps)
    if spec.get("mlp"):
        z = rms_norm(x, w[L + ".norm2"], eps) @ w[L + ".mlp.up"].T
        x = x + xielu(z, w[L + ".mlp.act"]) @ w[L + ".mlp.down"].T
    return x


def forward(cfg, w, tokens, dtype=torch.float64, mutate=None, residuals=None):
    """Logits [T, vocab] of one sequence; the residual stream after every layer run is appended to ``residuals``."""
    w = {k: t.to(dtype) for k, t in w.items()}
    eps = cfg["norm"]["eps"]
    x0 = w["embed"][torch.as_tensor(tokens, dtype=torch.long)]
    x = x0
    layers = cfg["layers"]
    loop = cfg.get("loop")
    lo, hi, times = (loop["start"], loop["stop"], loop["times"]) if loop else (0, 0, 0)

    def run(i):
        nonlocal x
        x = layer(x, w, i, layers[i], eps, mutate)
        if residuals is not None:
            residuals.append(x)

    for i in range(lo):
        run(i)
    for t in range(times):
        x = torch.cat([x, x0], -1) @ w["loop.in"].T
        if mutate != "no_loop_step":
            x = x + w["loop.step"][t]
        for i in range(lo, hi):
            run(i)
    for i in range(hi, len(layers)):
        run(i)
    return rms_norm(x, w["final.norm"], eps) @ w["head"].T


def random_config(layers, width, vocab, loop=None, eps=1e-6):
    return {"architecture": "Rakevik", "layers": layers, "loop": loop, "norm": {"eps": eps}, "vocab": vocab,
            "width": width}


def random_weights(cfg, seed=0, dtype=torch.bfloat16):
    """Weights of the right shapes with spreads that keep every mechanism visible in the logits."""
    g = torch.Generator().manual_seed(seed)
    W, V = cfg["width"], cfg["vocab"]
    out = {}

    def mat(name, o, i, gain=1.0):
        out[name] = (torch.randn(o, i, generator=g) * gain / math.sqrt(i)).to(dtype)

    def vec(name, n, mean=0.0, std=0.1):
        out[name] = (mean + std * torch.randn(n, generator=g)).to(dtype)

    out["embed"] = torch.randn(V, W, generator=g).to(dtype)
    if cfg.get("loop"):
        mat("loop.in", W, 2 * W)
        out["loop.step"] = (0.5 * torch.randn(cfg["loop"]["times"], W, generator=g)).to(dtype)
    for i, spec in enumerate(cfg["layers"]):
        m, L = spec["mixer"], f"l{i}"
        vec(L + ".norm1", W, 1.0)
        out[L + ".shift"] = torch.rand(W, generator=g).to(dtype)
        H, D, U = m["heads"], m["dim"], m["vdim"]
        if spec["type"] == "hgrn2":
            mat(L + ".mix.q", H * D, W)
            mat(L + ".mix.f", H * D, W, 1.5)
            vec(L + ".mix.f.b", H * D, 2.0, 1.0)
            out[L + ".mix.lower"] = (0.9 * torch.rand(H * D, generator=g)).to(dtype)
            mat(L + ".mix.v", H * U, W)
            vec(L + ".mix.norm", U, 1.0)
        else:
            G = m["kv_heads"]
            mat(L + ".mix.q", H * D, W)
            mat(L + ".mix.k", G * D, W)
            mat(L + ".mix.v", G * U, W)
            vec(L + ".mix.q.norm", D, 1.5)
            vec(L + ".mix.k.norm", D, 1.5)
            vec(L + ".mix.sink", H, 1.0, 1.0)
        mat(L + ".mix.o", W, H * U)
        if spec.get("mlp"):
            vec(L + ".norm2", W, 1.0)
            mat(L + ".mlp.up", spec["mlp"]["ff"], W)
            mat(L + ".mlp.down", W, spec["mlp"]["ff"])
            vec(L + ".mlp.act", 2, 0.3, 0.5)
    vec("final.norm", W, 1.0)
    mat("head", V, W)
    return out
