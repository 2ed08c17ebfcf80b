"""Plain restatement of the Disunex decoder, one function per mechanism, in one floating-point type.

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


def norm_after_sum(x, branch, alpha, weight, eps):
    """``rms_norm(alpha x + branch)`` with a weight stored around zero."""
    return rms_norm(alpha * x + branch, 1.0 + weight, eps)


def sigmoid(z):
    return 1.0 / (1.0 + torch.exp(-z))


def gelu_erf(z):
    return 0.5 * z * (1.0 + torch.erf(z / math.sqrt(2.0)))


def rotate_pairs(x, positions, base, dims):
    """x [T, ..., n]: neighbours (2i, 2i + 1) of the first ``dims`` turn by ``position * base^(-2i / dims)``."""
    out = x.clone()
    for i in range(dims // 2):
        a = positions.to(torch.float64) * float(base) ** (-2.0 * i / dims)
        c, s = torch.cos(a).to(x.dtype), torch.sin(a).to(x.dtype)
        while c.dim() < x.dim() - 1:
            c, s = c[..., None], s[..., None]
        u, v = x[..., 2 * i], x[..., 2 * i + 1]
        out[..., 2 * i] = u * c - v * s
        out[..., 2 * i + 1] = v * c + u * s
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


def latent_heads(q, c, kr, uk, uv, dim, scale, window, sink, mutate=None):
    """q [T, H, dim + rot] and the shared key part kr [T, rot] (both rotated), latents c [T, L], per-head up-projections
    uk [H, dim, L] and uv [H, V, L] -> [T, H, V]."""
    T, H, _ = q.shape
    if window is None:
        pass
    elif mutate == "window_plus":
        window = window + 1
    elif mutate == "window_minus":
        window = window - 1
    ok = visible(T, window)
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
    kr = down[:, L:]
    if mutate != "no_rotation":
        rot = m["rot"]
        q = torch.cat([q[..., :D], rotate_pairs(q[..., D:], pos, rot["base"], rot["dims"])], -1)
        kr = rotate_pairs(kr, pos, rot["base"], rot["dims"])
    o = latent_heads(q, c, kr, w[name + ".uk"].view(H, D, L), w[name + ".uv"].view(H, V, L), D, m["scale"],
                     m["mask"]["size"] if m.get("mask") else None, w[name + ".sink"], mutate)
    o = o.reshape(T, H * V)
    if mutate != "no_gate":
        o = o * sigmoid(h @ w[name + ".g"].T)
    return o @ w[name + ".o"].T


def clamped_expert(h, w, name, limit):
    g = torch.clamp(h @ w[name + ".gate"].T, max=limit)
    u = torch.clamp(h @ w[name + ".up"].T, -limit, limit)
    return (g * sigmoid(1.702 * g) * (u + 1.0)) @ w[name + ".down"].T


def route(z, correction, top, mutate=None):
    """Router logits [T, E] -> (chosen experts [T, top], their weights)."""
    s = sigmoid(z)
    choice = s if mutate == "no_correction" else s + correction
    idx = choice.topk(top, -1).indices
    ws = (choice if mutate == "corrected_weights" else s).gather(-1, idx)
    return idx, ws / (ws.sum(-1, keepdim=True) + 1e-20)


def moe(h, w, name, spec, mutate=None):
    r, limit = spec["router"], spec["expert"]["limit"]
    idx, ws = route(h @ w[name + ".router"].T, w[name + ".correction"], r["top"], mutate)
    out = torch.zeros_like(h)
    for e in range(r["experts"]):
        t, k = (idx == e).nonzero(as_tuple=True)
        if len(t):
            out[t] += ws[t, k][:, None] * clamped_expert(h[t], w, f"{name}.e{e}", limit)
    return out


def feed_forward(h, w, name, spec, mutate=None):
    if spec["kind"] == "moe":
        return moe(h, w, name, spec, mutate)
    return gelu_erf(h @ w[name + ".up"].T) @ w[name + ".down"].T


def layer(x, w, i, spec, alpha, eps, mutate=None):
    L = f"l{i}"
    if mutate == "no_alpha":
        alpha = 1.0
    x = norm_after_sum(x, latent_attention(x, w, L + ".mix", spec["mixer"], eps, mutate), alpha, w[L + ".norm1"], eps)
    if spec.get("mlp"):
        x = norm_after_sum(x, feed_forward(x, w, L + ".mlp", spec["mlp"], mutate), alpha, w[L + ".norm2"], eps)
    return x


def forward(cfg, weights, tokens, dtype=torch.float64, residuals=None, mutate=None):
    """Logits [T, vocab] of one sequence; ``residuals`` (a list) receives the stream after every layer."""
    w = {k: v.to(dtype) for k, v in weights.items()}
    eps, alpha = cfg["norm"]["eps"], cfg["postln_alpha"]
    x = w["embed"][torch.as_tensor(tokens, dtype=torch.long)]
    for i, spec in enumerate(cfg["layers"]):
        j = i if mutate == "no_sharing" and f"l{i}.norm1" in w else spec.get("weights_of", i)
        x = layer(x, w, j, spec, alpha, eps, mutate)
        if residuals is not None:
            residuals.append(x)
    return rms_norm(x, 1.0 + w["final.norm"], eps) @ w["embed"].T


# ------------------------------------------------------------------------------------------------ random models
def latent(heads, dim, rot_dim, vdim, kv_rank, scale, base=1e4, window=None, mlp=None, dims=None):
    m = {"heads": heads, "dim": dim, "rot_dim": rot_dim, "vdim": vdim, "kv_rank": kv_rank, "scale": scale,
         "rot": {"base": base, "dims": dims or rot_dim}}
    if window:
        m["mask"] = {"size": window}
    return {"type": "latent_attention", "mixer": m, "mlp": mlp}


def dense(ff):
    return {"kind": "dense", "ff": ff}


def experts(n, top, ff, limit):
    return {"kind": "moe", "router": {"experts": n, "top": top}, "expert": {"ff": ff, "limit": limit}}


def again(layers, j):
    """An entry that runs layer ``j``'s weights once more."""
    return {**layers[j], "weights_of": j}


def random_config(layers, width, vocab, alpha=1.7, eps=1e-6):
    return {"architecture": "Disunex", "layers": layers, "norm": {"eps": eps}, "postln_alpha": alpha, "vocab": vocab,
            "width": width}


def random_weights(cfg, seed=0, dtype=torch.bfloat16):
    """Random weights; sinks and corrections are large enough to matter, query and key products to stand out."""
    g = torch.Generator().manual_seed(seed)

    def r(*s, std=None):
        return torch.randn(*s, generator=g) * (std if std is not None else s[-1] ** -0.5)

    W = cfg["width"]
    w = {"embed": r(cfg["vocab"], W, std=1.0), "final.norm": r(W, std=0.2)}
    for i, e in enumerate(cfg["layers"]):
        if e.get("weights_of") is not None:
            continue
        L, m, f = f"l{i}", e["mixer"], e.get("mlp")
        H, D, R, V, K = m["heads"], m["dim"], m["rot_dim"], m["vdim"], m["kv_rank"]
        w[L + ".norm1"] = r(W, std=0.2)
        X = L + ".mix"
        w.update({X + ".q": r(H * (D + R), W) * 2, X + ".dkv": r(K + R, W) * 2, X + ".dkv.norm": 1 + r(K, std=0.2),
                  X + ".uk": r(H * D, K), X + ".uv": r(H * V, K), X + ".sink": r(H, std=1.5), X + ".g": r(H * V, W) * 2,
                  X + ".o": r(W, H * V) * 2})
        if not f:
            continue
        w[L + ".norm2"] = r(W, std=0.2)
        F = L + ".mlp"
        if f["kind"] == "dense":
            w.update({F + ".up": r(f["ff"], W), F + ".down": r(W, f["ff"]) * 2})
            continue
        n, ff = f["router"]["experts"], f["expert"]["ff"]
        w.update({F + ".router": r(n, W), F + ".correction": r(n, std=0.3)})
        for x in range(n):
            w.update({f"{F}.e{x}.gate": r(ff, W) * 2, f"{F}.e{x}.up": r(ff, W) * 2, f"{F}.e{x}.down": r(W, ff) * 2})
    return {k: v.to(dtype) for k, v in w.items()}
