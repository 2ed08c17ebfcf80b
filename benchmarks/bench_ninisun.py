"""Speed of the Ninisun family beside the framework's closest models: ``python bench.py --model ninisun`` (or
``python -m benchmarks.bench_ninisun``).

Two parts, each a list of JSON lines. *Kernels*: every kernel of the family at the sizes of a real model's layers, with
the share of its roofline (the measured copy bandwidth or cuBLAS rate, whichever bounds it), and beside it the kernel
that does the like job in an existing model; ``distance_ratio`` is how much farther from its roofline ours is (below 1:
nearer). *Models*: prefill and decode throughput of the serving engine for a Ninisun stack (three windowed layers to one
twin layer), a Gated-DeltaNet hybrid (``qwen3_5_text``), a recurrence-and-attention hybrid (``rakevik``) and a windowed
attention stack (``gemma3_text``) of equal width, depth, heads and feed-forward. Random weights; CUDA events; L2 flushed
between timed launches.
"""

from __future__ import annotations

import argparse
import json
import math

import torch

from benchmarks.bench_rakevik import BF, VOCAB, Table, _engine_speed, _pages, _rand

#: width, query / key-value heads (128 wide), heads of the delta rule and their size, rank of its decay, feed-forward, window,
#: kept first tokens
SIZES = ((2048, 16, 4, 32, 64, 64, 6144, 1024, 4), (4096, 32, 8, 64, 64, 128, 12288, 4096, 4))


# ------------------------------------------------------------------------------------------------ kernels
def bench_rows(t: Table, T: int, size) -> None:
    from easydel_b200.ops import kernels as K, rotation, stream

    W, H, G, HD, D, rank, F, *_ = size
    name = f"rows {T}, width {W}"
    x, y = _rand(T, W, dtype=torch.float32), _rand(T, W, dtype=torch.float32)
    w = torch.ones(W, device="cuda")
    xb, wb, rb = _rand(T, W), _rand(W), _rand(T, W)
    branch = stream.NormedBranch(y, w, 1e-6, w)
    t.add("norm and scale of a branch, sum, norm", name, (lambda: stream.add_norm(x, branch, 1.0, w, 1e-6, BF), T * W * 14),
          "sum of the branches and norm", (lambda: stream.add_norm(x, y, 0.7, w, 1e-6, BF), T * W * 14))
    t.add("norm and scale of a branch, sum, norm", name, (lambda: stream.add_norm(x, branch, 1.0, w, 1e-6, BF), T * W * 14),
          "rmsnorm with residual add", (lambda: K.rmsnorm_fwd(xb, wb, 1e-6, residual=rb, want_rstd=False), T * W * 8))
    sl, p = torch.arange(T, device="cuda", dtype=torch.int32) + 128, torch.arange(T, dtype=torch.int32, device="cuda")
    wide = _rand(T, (H + 2 * G) * 128 + 5 * HD * D)
    qkv, packed = wide[:, :(H + 2 * G) * 128], _rand(T, (H + 2 * G) * 128)
    kp, vp, _ = _pages(1, max(T, 128), G, 128, 128)
    hw = torch.ones(128, device="cuda")
    nb, heads = 4 * T * (H + 2 * G) * 128, (H, G, 128, 128)
    bias, first = torch.zeros((H + 2 * G) * 128, device="cuda"), _rand(T, G, 128)
    lam = torch.tensor(0.4, device="cuda")
    for what, rows, kw, more in (("rotate, blend, append", packed, dict(first=first, lam=lam), 2 * T * G * 128),
                                 ("biases, rotate, append", qkv, dict(bias=bias), 0)):
        for dims in (128, 32):
            f = rotation.pair_frequencies(1e6, dims, "cuda")
            t.add(f"attention prologue ({what})", f"{name}, {H}/{G} heads, {dims} rotated",
                  (lambda: stream.qkv_rotary_prologue(rows, heads, None, None, 0.0, p, f, sl, kp, vp, "neighbours", **kw),
                   nb + more),
                  "attention prologue (norms per head, no rotation, append)",
                  (lambda: stream.qkv_prologue(packed, heads, hw, hw, 1e-6, p, None, sl, kp, vp), nb))
    n_in = (H + 2 * G) * 128 + 5 * HD * D + rank + H
    for what, n, kk in (("packed projection of a windowed layer", (H + 2 * G) * 128, W),
                        ("packed projection of both mixers", n_in, W),
                        ("out projection of both mixers, fp32 result", W, H * 128 + HD * D),
                        ("low-rank product, fp32 result", HD * D, rank),
                        ("gate and up projections", 2 * F, W), ("down projection, fp32 result", W, F)):
        a, b = _rand(T, kk), _rand(n, kk, scale=1 / math.sqrt(kk))
        f32 = "fp32" in what
        yb = torch.empty(T, n, dtype=BF, device="cuda")
        t.add(what, f"{T} x {n} x {kk}",
              (lambda: stream.linear(a, b, out_dtype=torch.float32 if f32 else None),
               2 * (T * kk + n * kk) + (4 if f32 else 2) * T * n, 2 * T * n * kk),
              "same product, bf16 output", (lambda: K.gemm(a, b, out=yb), 2 * (T * kk + n * kk + T * n), 2 * T * n * kk))
    gu = _rand(T, 2 * F)
    t.add("gated gelu", f"rows {T}, ff {F}", (lambda: stream.gated_unit(gu, "gelu_tanh"), 6 * T * F), "gated silu",
          (lambda: K.gated_act_fwd(gu, "silu"), 6 * T * F))


def bench_recurrence(t: Table, B: int, L: int, size, D: int | None = None) -> None:
    """The generalised delta rule against the gated delta rule, ``B`` sequences of ``L`` tokens (L = 1: a decode step)."""
    from easydel_b200.ops import ssm

    H, rank = size[3] * size[4] // (D or size[4]), size[5]
    D, T = D or size[4], B * L
    widths = (H * D,) * 5 + (rank,)
    cols = ssm.DeltaColumns(*torch.split(_rand(T, sum(widths)), widths, -1))
    z = lambda: torch.zeros(H * D, device="cuda")  # noqa: E731
    wt = ssm.DeltaWeights(_rand(H * D, rank, scale=rank ** -0.5), z(), z(), torch.ones(H * D, device="cuda"), math.exp(-0.5), 1e-6,
                          1e-6)
    cu = torch.arange(0, T + 1, L, dtype=torch.int32, device="cuda")
    slots = torch.arange(B, dtype=torch.int32, device="cuda")
    st, st2 = torch.zeros(B, H, D, D, device="cuda"), torch.zeros(B, H, D, D, device="cuda")
    out = torch.empty(T, H * D, dtype=BF, device="cuda")
    q, k, v = _rand(T, H, D, scale=D ** -0.5), _rand(T, H, D, scale=D ** -0.5), _rand(T, H, D)
    g, beta = -torch.rand(T, H, D, device="cuda"), torch.rand(T, H, device="cuda").to(BF)
    nb = 2 * T * H * 6 * D + 2 * T * rank + 2 * H * D * rank + 8 * B * H * D * D
    t.add("generalised delta rule, decode" if L == 1 else "generalised delta rule (decay, rows, scan, norm, gate)",
          f"{B} x {L} tokens, {H} heads {D} x {D}",
          (lambda: ssm.generalized_delta_rule(cols, (H, D, D), wt, cu, L, slots, st, 1.1, out), nb),
          "delta rule with a decay per channel (no decay product, norm, gate)",
          (lambda: ssm.gated_delta_rule(q, k, v, g, beta, None, cu, st2), T * H * (8 * D + 4 * D + 2) + 8 * B * H * D * D))


def bench_attention(t: Table, B: int, new: int, ctx: int, size) -> None:
    """Kept first tokens and sigmoid weights against the plain window and the softmax."""
    from easydel_b200.ops import serving as S

    H, G, window, keep = size[1], size[2], size[7], size[8]
    lens = torch.full((B,), ctx, dtype=torch.int32, device="cuda")
    cu = torch.arange(0, B * new + 1, new, dtype=torch.int32, device="cuda")
    k, v, table = _pages(B, ctx, G, 128, 128)
    q, gate = _rand(B * new, H, 128), _rand(B * new, H)
    sig = S.SigmoidWeights(torch.full((H,), -3.0, device="cuda"), gate, 1.2)
    out = torch.empty(B * new, 2 * H, 128, dtype=BF, device="cuda")[:, :H]
    units = B * G
    sms = torch.cuda.get_device_properties(0).multi_processor_count

    def case(win, first, sigmoid):
        seen = min(win or ctx, ctx)
        pairs = B * H * sum(min(i + 1, seen + first) for i in range(ctx - new, ctx))
        nb = 4 * B * (min(ctx, seen + new - 1 + first) * G + new * H) * 128
        kw = dict(scale=128 ** -0.5, window=win or 0, keep_first=first, sigmoid=sigmoid, out=out if sigmoid else None)
        if new == 1:
            n = 1 if units * 2 > sms else int(min(8, ctx // 128 // 4, max(1, sms // units)))
            n = S.decode_splits(max(1, n), win, first)
            return lambda: S.decode_attention(q, k, v, lens, table, num_splits=n, **kw), nb, 4 * pairs * 128
        return lambda: S.paged_attention(q, k, v, cu, lens, table, new, **kw), nb, 4 * pairs * 128

    what = "decode" if new == 1 else "prefill"
    size_ = f"{B} x {new} tokens over {ctx} keys, {H}/{G} heads"
    t.add(f"{what} attention, window with kept first tokens", f"{size_}, window {window} + {keep}", case(window, keep, None),
          "window", case(window, 0, None))
    t.add(f"{what} attention, sigmoid weights, gate", size_, case(None, 0, sig), "softmax", case(None, 0, None))


def bench_kernels() -> list[dict]:
    t = Table()
    with torch.no_grad():
        for size in SIZES:
            for T in (8192, 64):
                bench_rows(t, T, size)
            for B, L in ((1, 8192), (8, 1024), (8, 1), (64, 1), (256, 1)):
                bench_recurrence(t, B, L, size)
            for B, L in ((1, 8192), (64, 1)):
                bench_recurrence(t, B, L, size, 128)
            bench_attention(t, 1, 8192, 8192, size)
            for B, ctx in ((64, 1024), (64, 8192), (8, 8192), (256, 1024)):
                bench_attention(t, B, 1, ctx, size)
    return t.rows


# ------------------------------------------------------------------------------------------------ models
def _models(size, layers: int):
    """(name, constructor) of stacks with equal width, depth, heads and feed-forward."""
    from easydel_b200.infra.factory import TaskType, _ensure_models_imported, registry

    _ensure_models_imported()
    W, H, G, HD, D, rank, F, window, keep = size

    def build(mtype, **kw):
        reg = registry.get_module_registration(TaskType.CAUSAL_LM, mtype)
        return reg.module.sequential_init(reg.config(**kw), dtype=BF, param_dtype=BF, device="cuda", seed=1).eval()

    mlp = {"kind": "dense", "ff": F}
    win = {"heads": H, "kv_heads": G, "dim": 128, "vdim": 128, "scale": 128 ** -0.5, "v_mix": True,
           "mask": {"size": window, "keep_first": keep}, "rot": {"base": 1e6, "dims": 128}}
    twin = {"left": {"heads": H, "kv_heads": G, "dim": 128, "vdim": 128, "scale": 128 ** -0.5,
                     "rot": {"base": 5e5, "dims": 128, "scaling": {"factor": 4.0, "original": 8192, "fast": 32.0, "slow": 1.0}}},
            "left_scale": 1.0, "right": {"heads": HD, "dim": D, "rank": rank}, "right_scale": 1.0}
    yield "ninisun", lambda: build(
        "ninisun", vocab=VOCAB, width=W,
        layers=[{"type": "parallel", "mixer": twin, "mlp": mlp} if i % 4 == 3 else
                {"type": "attention", "mixer": win, "mlp": mlp} for i in range(layers)])
    common = dict(vocab_size=VOCAB, hidden_size=W, intermediate_size=F, num_hidden_layers=layers, num_attention_heads=H,
                  num_key_value_heads=G, head_dim=128, tie_word_embeddings=True)
    yield "qwen3_5_text", lambda: build("qwen3_5_text", linear_key_head_dim=128, linear_value_head_dim=128,
                                        linear_num_key_heads=H, linear_num_value_heads=H, **common)
    plain = {"kind": "dense", "ff": F * 3 // 2}      # two matrices instead of three
    att = {"heads": H, "kv_heads": G, "dim": 128, "vdim": 128, "scale": 128 ** -0.5}
    yield "rakevik", lambda: build(
        "rakevik", vocab=VOCAB, width=W, loop=None,
        layers=[{"type": "hgrn2", "mixer": {"heads": H, "dim": 128, "vdim": 128}, "mlp": plain} if i % 4 == 3 else
                {"type": "attention", "mixer": att, "mlp": plain} for i in range(layers)])
    yield "gemma3_text", lambda: build(
        "gemma3_text", query_pre_attn_scalar=128, sliding_window=window, max_position_embeddings=16384,
        layer_types=["full_attention" if i % 4 == 3 else "sliding_attention" for i in range(layers)], **common)


def bench_models() -> list[dict]:
    rows = []
    for size, layers in zip(SIZES, (8, 8)):
        for name, build in _models(size, layers):
            model = build()
            n = sum(p.numel() for p in model.parameters())
            for batch in (8, 64):
                row = {"model": name, "width": size[0], "layers": layers, "window": size[7], "parameters": n,
                       **_engine_speed(model, 8192, batch, 1024)}
                rows.append(row)
                print(json.dumps(row), flush=True)
            del model
            torch.cuda.empty_cache()
    return rows


def main(argv=None) -> None:
    ap = argparse.ArgumentParser(description=__doc__)
    ap.add_argument("what", nargs="?", choices=("all", "kernels", "models"), default="all")
    a = ap.parse_args(argv)
    if a.what in ("all", "kernels"):
        bench_kernels()
    if a.what in ("all", "models"):
        bench_models()


if __name__ == "__main__":
    main()
