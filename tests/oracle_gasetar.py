"""Plain restatement of the Gasetar decoder, one function per mechanism, in one floating-point type.

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


def silu(z):
    return z * sigmoid(z)


def soft_cap(z, cap):
    return cap * torch.tanh(z / cap) if cap else z


def frequency(base, dims, i, scaling=None, mutate=None):
    """Turn rate of pair i: ``base^(-2i / dims)``; with ``scaling``, slow pairs (long wavelengths) are slowed down by
    ``factor``, fast ones are left alone, and in between the two are blended."""
    f = float(base) ** (-2.0 * i / dims)
    if not scaling or mutate == "no_scaling":
        return f
    wave = 2.0 * math.pi / f
    if wave < scaling["original"] / scaling["high"]:
        return f
    if wave > scaling["original"] / scaling["low"]:
        return f / scaling["factor"]
    s = (scaling["original"] / wave - scaling["low"]) / (scaling["high"] - scaling["low"])
    return (1.0 - s) * f / scaling["factor"] + s * f


def rotate_half(x, positions, rot, mutate=None):
    """x [T, ..., n]: elements i and i + dims / 2 of the first ``dims`` form a pair that turns with the position."""
    if mutate == "no_rotation":
        return x
    dims, out = rot["dims"], x.clone()
    for i in range(dims // 2):
        a = positions.to(torch.float64) * frequency(rot["base"], dims, i, rot.get("scaling"), mutate)
        c, s = torch.cos(a).to(x.dtype), torch.sin(a).to(x.dtype)
        while c.dim() < x.dim() - 1:
            c, s = c[..., None], s[..., None]
        j, k = (2 * i, 2 * i + 1) if mutate == "neighbour_pairs" else (i, i + dims // 2)
        u, v = x[..., j], x[..., k]
        out[..., j] = u * c - v * s
        out[..., k] = v * c + u * s
    return out


def visible(T, window):
    """[T, T] of the keys j a query i sees: ``0 <= i - j < window`` (no window: all of the past)."""
    d = torch.arange(T)[:, None] - torch.arange(T)[None]
    return (d >= 0) & ((d < window) if window else (d >= 0))


def sink_softmax(s, sink):
    """Rows of scores -> weights; ``exp(sink)`` joins the denominator (None: no sink)."""
    top = s.max(-1, keepdim=True).values
    if sink is not None:
        top = torch.maximum(top, sink)
    p = torch.exp(s - top)
    den = p.sum(-1, keepdim=True)
    if sink is not None:
        den = den + torch.exp(sink - top)
    return p / den


# ------------------------------------------------------------------------------------------------ windowed attention
def windowed_heads(q, k, v, scale, window, cap, mutate=None):
    """q [T, H, D], k [T, G, D], v [T, G, V] -> [T, H, V]: scaled scores, soft-capped, softmax over the window."""
    T, H, _ = q.shape
    G = k.shape[1]
    if mutate in ("window_plus", "window_minus"):
        window = window + (1 if mutate == "window_plus" else -1)
    ok = visible(T, window).to(q.device)
    out = []
    for h in range(H):
        g = h % G if mutate == "wrong_groups" else h // (H // G)
        s = q[:, h] @ k[:, g].T * scale
        if mutate != "no_score_cap":
            s = soft_cap(s, cap)
        out.append(sink_softmax(s.masked_fill(~ok, -math.inf), None) @ v[:, g])
    return torch.stack(out, 1)


def attention(h, w, name, m, eps, mutate=None):
    T = h.shape[0]
    H, G, D, V = m["heads"], m["kv_heads"], m["dim"], m["vdim"]
    pos = torch.arange(T)
    q, k = h @ w[name + ".q"].T, h @ w[name + ".k"].T
    if mutate == "head_norms":
        q = rms_norm(q.view(T, H, D), w[name + ".q.norm"].view(H, D), eps)
        k = rms_norm(k.view(T, G, D), w[name + ".k.norm"].view(G, D), eps)
    else:                # over all heads of the projection at once
        q, k = rms_norm(q, w[name + ".q.norm"], eps), rms_norm(k, w[name + ".k.norm"], eps)
    q, k = q.reshape(T, H, D), k.reshape(T, G, D)
    v = (h @ w[name + ".v"].T).view(T, G, V)
    q, k = rotate_half(q, pos, m["rot"], mutate), rotate_half(k, pos, m["rot"], mutate)
    o = windowed_heads(q, k, v, m["scale"], (m.get("mask") or {}).get("size"), m.get("softcap"), mutate)
    return o.reshape(T, H * V) @ w[name + ".o"].T


# ------------------------------------------------------------------------------------------------ latent attention
def latent_heads(q, c, kr, uk, uv, dim, scale, sink, mutate=None):
    """q [T, H, dim + rot] and the shared key part kr [T, rot] (both rotated), latents c [T, L], per-head up-projections
    uk [H, dim, L] and uv [H, V, L] -> [T, H, V]."""
    T, H, _ = q.shape
    ok = visible(T, None)
    out = []
    for h in range(H):
        k = c @ uk[h].T
        s = (q[:, h, :dim] @ k.T + q[:, h, dim:] @ kr.T) * scale
        s = s.masked_fill(~ok, -math.inf)
        p = sink_softmax(s, None if mutate == "no_sink" else sink[h] * (scale if mutate == "scaled_sink" else 1.0))
        out.append(p @ (c @ uv[h].T))
    return torch.stack(out, 1)


def latent_attention(h, w, name, m, eps, mutate=None):
    T = h.shape[0]
    H, D, R, V, L = m["heads"], m["dim"], m["rot_dim"], m["vdim"], m["kv_rank"]
    pos = torch.arange(T)
    q = (h @ w[name + ".q"].T).view(T, H, D + R)
    down = h @ w[name + ".dkv"].T
    c = rms_norm(down[:, :L], w[name + ".dkv.norm"], eps)
    q = torch.cat([q[..., :D], rotate_half(q[..., D:], pos, m["rot"], mutate)], -1)
    kr = rotate_half(down[:, L:], pos, m["rot"], mutate)
    o = latent_heads(q, c, kr, w[name + ".uk"].view(H, D, L), w[name + ".uv"].view(H, V, L), D, m["scale"],
                     w[name + ".sink"], mutate).reshape(T, H * V)
    if mutate != "no_gate":
        o = o * sigmoid(h @ w[name + ".g"].T)
    return o @ w[name + ".o"].T


# ------------------------------------------------------------------------------------------------ feed-forward
def gated_unit(h, w, name):
    return (silu(h @ w[name + ".gate"].T) * (h @ w[name + ".up"].T)) @ w[name + ".down"].T


def route(z, top, mutate=None):
    """Router logits [T, E] -> (chosen experts [T, top], their weights: a softmax over the chosen logits)."""
    val, idx = z.topk(top, -1)
    if mutate == "softmax_over_all":
        return idx, torch.softmax(z, -1).gather(-1, idx)
    return idx, torch.softmax(val, -1)


def moe(h, w, name, spec, mutate=None):
    r = spec["router"]
    z = h @ w[name + ".router"].T
    if mutate != "no_router_bias":
        z = z + w[name + ".router.b"]
    idx, ws = route(z, r["top"], mutate)
    out = torch.zeros_like(h)
    for e in range(r["experts"]):
        t, k = (idx == e).nonzero(as_tuple=True)
        if len(t):
            out[t] += ws[t, k][:, None] * gated_unit(h[t], w, f"{name}.e{e}")
    if spec.get("shared") and mutate != "no_shared":
        out = out + gated_unit(h, w, name + ".shared")
    return out


def feed_forward(h, w, name, spec, mutate=None):
    return moe(h, w, name, spec, mutate) if spec["kind"] == "moe" else gated_unit(h, w, name)


# ------------------------------------------------------------------------------------------------ the model
def layer(x, w, i, spec, mult, eps, mutate=None):
    """Both branches read one norm of the stream and are added to it together."""
    L = f"l{i}"
    h = rms_norm(x, w[L + ".norm1"], eps)
    mixer = attention if spec["type"] == "attention" else latent_attention
    y = mixer(h, w, L + ".mix", spec["mixer"], eps, mutate)
    if spec.get("mlp"):
        if mutate == "one_after_the_other":
            h = rms_norm(x + mult * y, w[L + ".norm1"], eps)
        y = y + feed_forward(h, w, L + ".mlp", spec["mlp"], mutate)
    return x + (1.0 if mutate == "no_residual_mult" else mult) * y


def forward(cfg, weights, tokens, dtype=torch.float64, residuals=None, mutate=None):
    """Logits [T, vocab] of one sequence; ``residuals`` (a list) receives the stream after every layer."""
    w = {k: v.to(dtype) for k, v in weights.items()}
    eps = cfg["norm"]["eps"]
    x = w["embed"][torch.as_tensor(tokens, dtype=torch.long)] * cfg["embedding"]["scale"]
    for i, spec in enumerate(cfg["layers"]):
        x = layer(x, w, i, spec, cfg["residual_mult"], eps, mutate)
        if residuals is not None:
            residuals.append(x)
    z = rms_norm(x, w["final.norm"], eps) @ w["embed"].T
    z = z * (1.0 if mutate == "no_logit_scale" else cfg["logit_scale"])
    return z if mutate == "no_logit_cap" else soft_cap(z, cfg["logit_softcap"])


# ------------------------------------------------------------------------------------------------ random models
def windowed(heads, kv_heads, dim, vdim, scale, window, cap, base=1e4, dims=None, scaling=None, mlp=None):
    """``scaling``: (factor, low, high, original)."""
    rot = {"base": base, "dims": dim if dims is None else dims}
    if scaling:
        rot["scaling"] = dict(zip(("factor", "low", "high", "original"), scaling))
    return {"type": "attention", "mlp": mlp,
            "mixer": {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "scale": scale, "softcap": cap,
                      "mask": {"size": window}, "rot": rot}}


def latent(heads, dim, rot_dim, vdim, kv_rank, scale, base=1e4, mlp=None):
    return {"type": "latent_attention", "mlp": mlp,
            "mixer": {"heads": heads, "dim": dim, "rot_dim": rot_dim, "vdim": vdim, "kv_rank": kv_rank, "scale": scale,
                      "rot": {"base": base, "dims": rot_dim}}}


def dense(ff):
    return {"kind": "dense", "ff": ff}


def experts(n, top, ff, shared=None):
    out = {"kind": "moe", "router": {"experts": n, "top": top}, "expert": {"ff": ff}}
    return {**out, "shared": {"ff": shared}} if shared else out


def random_config(layers, width, vocab, mult=0.6, eps=1e-6, embed_scale=2.5, logit_scale=0.3, logit_cap=7.0):
    return {"architecture": "Gasetar", "layers": layers, "norm": {"eps": eps}, "residual_mult": mult, "vocab": vocab,
            "width": width, "embedding": {"scale": embed_scale}, "logit_scale": logit_scale, "logit_softcap": logit_cap}


def random_weights(cfg, seed=0, dtype=torch.bfloat16):
    """Random weights; sinks, router biases and norms are large enough to matter, scores reach the soft-cap's bend."""
    g = torch.Generator().manual_seed(seed)

    def r(*s, std=None):
        return torch.randn(*s, generator=g) * (std if std is not None else s[-1] ** -0.5)

    W = cfg["width"]
    w = {"embed": r(cfg["vocab"], W, std=1.0), "final.norm": 1 + r(W, std=0.2)}

    def unit(name, ff):
        w.update({name + ".gate": r(ff, W) * 2, name + ".up": r(ff, W) * 2, name + ".down": r(W, ff) * 2})

    for i, e in enumerate(cfg["layers"]):
        L, m, f = f"l{i}", e["mixer"], e.get("mlp")
        X, F = L + ".mix", L + ".mlp"
        w[L + ".norm1"] = 1 + r(W, std=0.2)
        if e["type"] == "attention":
            H, G, D, V = m["heads"], m["kv_heads"], m["dim"], m["vdim"]
            w.update({X + ".q": r(H * D, W), X + ".k": r(G * D, W), X + ".v": r(G * V, W),
                      X + ".q.norm": 1.5 + r(H * D, std=0.5), X + ".k.norm": 1.5 + r(G * D, std=0.5),
                      X + ".o": r(W, H * V) * 2})
        else:
            H, D, R, V, K = m["heads"], m["dim"], m["rot_dim"], m["vdim"], m["kv_rank"]
            w.update({X + ".q": r(H * (D + R), W) * 2, X + ".dkv": r(K + R, W) * 2, X + ".dkv.norm": 1 + r(K, std=0.2),
                      X + ".uk": r(H * D, K), X + ".uv": r(H * V, K), X + ".sink": r(H, std=1.5), X + ".g": r(H * V, W) * 2,
                      X + ".o": r(W, H * V) * 2})
        if not f:
            continue
        if f["kind"] == "dense":
            unit(F, f["ff"])
            continue
        n = f["router"]["experts"]
        w.update({F + ".router": r(n, W), F + ".router.b": r(n, std=0.5)})
        for x in range(n):
            unit(f"{F}.e{x}", f["expert"]["ff"])
        if f.get("shared"):
            unit(F + ".shared", f["shared"]["ff"])
    return {k: v.to(dtype) for k, v in w.items()}
