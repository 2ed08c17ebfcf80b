"""Speed of the Gasetar family beside the framework's closest models: ``python bench.py --model gasetar`` (or
``python -m benchmarks.bench_gasetar``).

Two parts, each a list of JSON lines. *Kernels*: every kernel of the family at the sizes of a real model's layers, with
the share of its roofline (the measured copy bandwidth or cuBLAS rate, whichever bounds it), and beside it the kernel
that does the like job in an existing model; ``distance_ratio`` is how much farther from its roofline ours is (below 1:
nearer). *Models*: prefill and decode throughput of the serving engine for a Gasetar stack (three windowed layers to one
latent layer, experts with a shared one), the latent stacks ``disunex`` and ``deepseek_v3`` of equal width, depth, heads,
latents and experts, and a ``gemma2`` stack (windows and capped scores) whose dense feed-forward is as wide as the experts
of a token together. Random weights; CUDA events; L2 flushed between timed launches.
"""

from __future__ import annotations

import argparse
import json
import math

import torch

from benchmarks.bench_rakevik import BF, VOCAB, Table, _engine_speed, _pages, _rand

#: width, query / key-value heads of windowed layers (128 wide), latent heads, unrotated / rotary / value size, latent,
#: experts, choices, expert (and shared) feed-forward, dense feed-forward, window
SIZES = ((2048, 16, 4, 16, 128, 64, 128, 512, 64, 6, 1408, 5632, 1024),
         (4096, 32, 8, 32, 128, 64, 128, 512, 64, 8, 2048, 14336, 4096))
CAP = 50.0


# ------------------------------------------------------------------------------------------------ kernels
def bench_rows(t: Table, T: int, size) -> None:
    from easydel_b200.ops import _lib, kernels as K, latent, rotation, stream
    from easydel_b200.ops.moe_kernels import ExpertRows

    W, H, G, HL, D, R, V, L, E, k, F, ff, _ = size
    name = f"rows {T}, width {W}"
    x, y = _rand(T, W, dtype=torch.float32), _rand(T, W, dtype=torch.float32)
    w = torch.ones(W, device="cuda")
    xb, wb, rb = _rand(T, W), _rand(W), _rand(T, W)
    t.add("sum of the branches and norm", name, (lambda: stream.add_norm(x, y, 0.7, w, 1e-6, BF), T * W * 14),
          "rmsnorm with residual add", (lambda: K.rmsnorm_fwd(xb, wb, 1e-6, residual=rb, want_rstd=False), T * W * 8))
    ys, wts = _rand(T * k, W), torch.rand(T, k, device="cuda")
    pos = torch.randperm(T * k, device="cuda").to(torch.int32)
    rows, out = ExpertRows(ys, wts, pos, y), torch.empty(T, W, dtype=BF, device="cuda")
    t.add(f"sum of the branches with {k} experts, norm", name,
          (lambda: stream.add_norm(x, rows, 0.7, w, 1e-6, BF), T * W * (14 + 2 * k)), "moe combine (no norm)",
          (lambda: _lib.call("edl_moe_combine", ys.data_ptr(), wts.data_ptr(), pos.data_ptr(), out.data_ptr(), T, k, W, 0,
                             _lib.stream_ptr()), T * W * (2 + 2 * k)))
    sl, p = torch.arange(T, device="cuda", dtype=torch.int32) + 128, torch.arange(T, dtype=torch.int32, device="cuda")
    qkv = _rand(T, (H + 2 * G) * 128)
    kp, vp, _ = _pages(1, max(T, 128), G, 128, 128)
    qw, kw, hw = torch.ones(H * 128, device="cuda"), torch.ones(G * 128, device="cuda"), torch.ones(128, device="cuda")
    nb, heads = 4 * T * (H + 2 * G) * 128, (H, G, 128, 128)
    for dims in (128, 64):
        f = rotation.pair_frequencies(1e4, dims, "cuda")
        t.add("attention prologue (full-width norms, rotate, append)", f"{name}, {H}/{G} heads, {dims} rotated",
              (lambda: stream.qkv_rotary_prologue(qkv, heads, qw, kw, 1e-6, p, f, sl, kp, vp), nb),
              "attention prologue (norms per head, no rotation, append)",
              (lambda: stream.qkv_prologue(qkv, heads, hw, hw, 1e-6, p, None, sl, kp, vp), nb))
    proj = _rand(T, HL * (D + R) + L + R + HL * V)
    pages = torch.zeros(T // 128 + 2, 128, 1, L + R, dtype=BF, device="cuda")
    nw, freq, lh = torch.ones(L, device="cuda"), rotation.pair_frequencies(1e4, R, "cuda"), (HL, D, R, L)
    t.add("latent prologue, halves", f"{name}, {HL} heads",
          (lambda: latent.prologue(proj, lh, nw, 1e-6, freq, p, sl, pages, "halves"), 4 * T * (HL * R + L + R)),
          "latent prologue, neighbours",
          (lambda: latent.prologue(proj, lh, nw, 1e-6, freq, p, sl, pages), 4 * T * (HL * R + L + R)))
    for what, n, kk, base in (("packed projection", qkv.shape[1], W, False), ("out projection, fp32 result", W, H * 128, False),
                              ("gate and up projections", 2 * ff, W, False), ("down projection onto fp32 rows", W, ff, True),
                              ("shared down projection onto fp32 rows", W, F, True), ("router, fp32 result", E, W, False)):
        a, b = _rand(T, kk), _rand(n, kk, scale=1 / math.sqrt(kk))
        f32 = "fp32" in what
        yb, acc = torch.empty(T, n, dtype=BF, device="cuda"), torch.zeros(T, n, device="cuda") if base else None
        run = (lambda: stream.branch_product(a, b, acc)) if base else \
            (lambda: stream.linear(a, b, out_dtype=torch.float32 if f32 else None))
        t.add(what, f"{T} x {n} x {kk}", (run, 2 * (T * kk + n * kk) + (8 if base else 4 if f32 else 2) * T * n, 2 * T * n * kk),
              "same product, bf16 output", (lambda: K.gemm(a, b, out=yb), 2 * (T * kk + n * kk + T * n), 2 * T * n * kk))
    ids, table = torch.randint(0, VOCAB, (T,), device="cuda"), _rand(VOCAB, W)
    t.add("scaled embedding rows", name, (lambda: stream.embed(table, ids, None, 45.0), T * W * 6), "embedding rows",
          (lambda: K.embed_fwd(table, ids), T * W * 4))
    if T <= 256:
        z = _rand(T, VOCAB, dtype=torch.float32)
        t.add("scaled and capped logits", f"{T} x {VOCAB}", (lambda: stream.scale_cap(z, 0.25, 30.0), 8 * z.numel()),
              "the same in tensor operations", (lambda: torch.tanh((z * 0.25) / 30.0).mul_(30.0), 8 * z.numel()))


def bench_experts(t: Table, T: int, size) -> None:
    from easydel_b200.ops import kernels as K, moe_kernels as MK, stream

    W, E, k, F = size[0], size[8], size[9], size[10]
    h, wr = _rand(T, W), _rand(E, W, scale=W ** -0.5)
    logits = stream.linear(h, wr, None, torch.float32)
    nb = T * E * 4 + T * k * 12
    t.add("softmax routing and expert tables", f"rows {T}, {k} of {E}", (lambda: MK.SoftmaxRouting(logits, k), nb),
          "sigmoid routing and expert tables", (lambda: MK.SigmoidRouting(logits, None, k), nb))
    gu, dn = _rand(E, 2 * F, W, scale=W ** -0.5), _rand(E, W, F, scale=F ** -0.5)
    r = MK.SoftmaxRouting(logits, k)
    val, idx = logits.topk(k, -1)
    w = torch.softmax(val, -1)
    used = min(E, T * k)
    nb, fl = 2 * used * 3 * F * W + 4 * T * W + 8 * T * k * F, 6 * T * k * W * F
    t.add("silu experts (gather, products, unit)", f"rows {T}, {k} of {E}, {W} x {F}",
          (lambda: MK.stream_experts(h, r, gu, dn), nb, fl), "routed silu experts (with tables and combine)",
          (lambda: MK.moe_ffn(h, gu, dn, w, idx, "silu"), nb, fl))
    x2 = _rand(r.max_rows, 2 * F)
    t.add("gated unit of rows in use", f"rows {T * k} of {r.max_rows}, ff {F}", (lambda: MK.expert_unit(x2, r), 6 * T * k * F),
          "gated silu over all rows", (lambda: K.gated_act_fwd(x2, "silu"), 6 * T * k * F))


def bench_decode(t: Table, B: int, ctx: int, size) -> None:
    from easydel_b200.ops import kernels as K, latent, serving as S

    W, H, G, HL, D, R, V, L, *_, window = size
    k, v, table = _pages(B, ctx, G, 128, 128)
    lens = torch.full((B,), ctx, dtype=torch.int32, device="cuda")
    seen = min(window, ctx)
    short = torch.full((B,), seen, dtype=torch.int32, device="cuda")
    q = _rand(B, H, 128)
    nb = 4 * B * (seen * G * 128 + H * 128)
    n = S.decode_splits(max(1, min(8, K.sm_count(q.device) // max(1, B))) if B * 2 <= K.sm_count(q.device) else 1, window)
    t.add("decode attention, window and capped scores", f"{B} rows over {ctx} keys, window {window}, {H}/{G} heads, {n} splits",
          (lambda: S.decode_attention(q, k, v, lens, table, scale=0.09, window=window, softcap=CAP, num_splits=n), nb),
          "decode attention of as many keys, no cap",
          (lambda: S.decode_attention(q, k, v, short, table, scale=0.09, num_splits=n), nb))
    pages = _rand(B * (ctx // 128) + 1, 128, 1, L + R)
    ql, sinks = _rand(B, HL, L + R), torch.ones(HL, device="cuda")
    n = latent.decode_splits(B, HL, 0, ctx, K.sm_count(q.device))
    nb, fl = 2 * B * (ctx * (L + R) + HL * (2 * L + R)), 2 * B * HL * ctx * (2 * L + R)
    t.add("latent decode, sinks", f"{B} rows over {ctx} keys, {HL} heads, {n} splits",
          (lambda: S.latent_decode(ql[..., :L], ql[..., L:], pages, lens, table, scale=0.07, sinks=sinks, num_splits=n), nb, fl),
          "latent decode, no sinks (512 + 64)",
          (lambda: S.mla_decode_attention(ql, pages, lens, table, scale=0.07, num_splits=n), nb, fl))


def bench_prefill(t: Table, T: int, size) -> None:
    from easydel_b200.ops import serving as S

    H, G, window = size[1], size[2], size[-1]
    k, v, table = _pages(1, T, G, 128, 128)
    lens = torch.full((1,), T, dtype=torch.int32, device="cuda")
    cu = torch.tensor([0, T], dtype=torch.int32, device="cuda")
    nb = 4 * T * (H + G) * 128
    for win in (window, 0):
        s = min(T, win or T)
        fl = 4 * H * (s * (s + 1) / 2 + (T - s) * s) * 128
        for what, size_ in (("scores far below the cap", 1.0), ("scores up to the cap", 6.0)):
            q = _rand(T, H, 128, scale=size_)

            def case(cap):
                return (lambda: S.paged_attention(q, k, v, cu, lens, table, T, scale=128 ** -0.5, window=win, softcap=cap), nb,
                        fl)

            t.add(f"prefill attention, capped, {what}", f"{T} tokens, window {win or 'none'}, {H}/{G} heads", case(CAP),
                  "no cap", case(0.0))


def bench_kernels() -> list[dict]:
    t = Table()
    with torch.no_grad():
        for size in SIZES:
            for T in (8192, 64):
                bench_rows(t, T, size)
                bench_experts(t, T, size)
            for B, ctx in ((64, 1024), (64, 8192), (8, 8192), (256, 1024)):
                bench_decode(t, B, ctx, size)
            bench_prefill(t, 8192, size)
    return t.rows


# ------------------------------------------------------------------------------------------------ models
def _models(size, layers: int):
    """(name, constructor) of stacks with equal width, depth, heads, latents and experts."""
    from easydel_b200.infra.factory import TaskType, _ensure_models_imported, registry

    _ensure_models_imported()
    W, H, G, HL, D, R, V, L, E, k, F, ff, window = size

    def build(mtype, **kw):
        reg = registry.get_module_registration(TaskType.CAUSAL_LM, mtype)
        return reg.module.sequential_init(reg.config(**kw), dtype=BF, param_dtype=BF, device="cuda", seed=1).eval()

    lat = {"heads": HL, "dim": D, "rot_dim": R, "vdim": V, "kv_rank": L, "scale": (D + R) ** -0.5,
           "rot": {"base": 1e4, "dims": R}}
    win = {"heads": H, "kv_heads": G, "dim": 128, "vdim": 128, "scale": 128 ** -0.5, "softcap": CAP, "mask": {"size": window},
           "rot": {"base": 1e4, "dims": 128, "scaling": {"factor": 8.0, "low": 1.0, "high": 4.0, "original": 8192}}}
    moe = {"kind": "moe", "router": {"experts": E, "top": k}, "expert": {"ff": F}, "shared": {"ff": F}}
    stack = [{"type": "latent_attention", "mixer": lat, "mlp": moe} if i % 4 == 1 else
             {"type": "attention", "mixer": win, "mlp": moe if i else {"kind": "dense", "ff": ff}} for i in range(layers)]
    yield "gasetar", lambda: build("gasetar", layers=stack, vocab=VOCAB, width=W, residual_mult=0.7, logit_scale=0.25,
                                   logit_softcap=30.0)
    clamped = {"kind": "moe", "router": {"experts": E, "top": k}, "expert": {"ff": F, "limit": 7.0}}
    yield "disunex", lambda: build(
        "disunex", vocab=VOCAB, width=W, postln_alpha=2.0,
        layers=[{"type": "latent_attention", "mixer": lat, "mlp": clamped if i else {"kind": "dense", "ff": ff}}
                for i in range(layers)])
    yield "deepseek_v3", lambda: build(
        "deepseek_v3", vocab_size=VOCAB, hidden_size=W, intermediate_size=ff, moe_intermediate_size=F,
        num_hidden_layers=layers, num_attention_heads=HL, num_key_value_heads=HL, n_shared_experts=1, n_routed_experts=E,
        kv_lora_rank=L, q_lora_rank=None, qk_rope_head_dim=R, v_head_dim=V, qk_nope_head_dim=D, num_experts_per_tok=k,
        first_k_dense_replace=1, n_group=1, topk_group=1, norm_topk_prob=True, routed_scaling_factor=1.0,
        max_position_embeddings=16384, tie_word_embeddings=True)
    yield "gemma2", lambda: build(
        "gemma2", vocab_size=VOCAB, hidden_size=W, intermediate_size=(k + 1) * F, num_hidden_layers=layers,
        num_attention_heads=H, num_key_value_heads=G, head_dim=128, query_pre_attn_scalar=128, sliding_window=window,
        layer_types=["full_attention" if i % 4 == 1 else "sliding_attention" for i in range(layers)],
        max_position_embeddings=16384)


def bench_models() -> list[dict]:
    rows = []
    for size, layers in zip(SIZES, (8, 4)):
        for name, build in _models(size, layers):
            model = build()
            n = sum(p.numel() for p in model.parameters())
            for batch in (8, 64):
                try:
                    speed = _engine_speed(model, 8192, batch, 1024)
                except torch.OutOfMemoryError:      # scores of padded rows as one tensor: smaller steps fit
                    torch.cuda.empty_cache()
                    speed = _engine_speed(model, 2048, batch, 1024)
                row = {"model": name, "width": size[0], "layers": layers, "window": size[-1], "parameters": n, **speed}
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
