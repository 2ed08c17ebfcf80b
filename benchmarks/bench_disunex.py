"""Speed of the Disunex family beside the framework's closest model: ``python bench.py --model disunex`` (or
``python -m benchmarks.bench_disunex``).

Two parts, each a list of JSON lines. *Kernels*: every kernel of the family at the sizes of a real model's layers, with
the share of its roofline (the measured copy bandwidth or cuBLAS rate, whichever bounds it), and beside it the kernel
that does the like job in an existing model; ``distance_ratio`` is how much farther from its roofline ours is (below 1:
nearer). *Models*: prefill and decode throughput of the serving engine for a Disunex stack and a ``deepseek_v3`` stack
(latent attention and sigmoid-scored experts, the closest model) of equal width, depth, heads and experts. Random
weights; CUDA events; L2 flushed between timed launches.
"""

from __future__ import annotations

import argparse
import json
import math

import torch

from benchmarks.bench_rakevik import BF, VOCAB, Table, _engine_speed, _pages, _rand

#: width, heads, unrotated / rotary / value size of a head, latent, experts, choices, expert and dense feed-forward, window
SIZES = ((2048, 16, 128, 64, 128, 512, 64, 6, 1408, 8192, 1024),
         (4096, 32, 128, 64, 128, 512, 64, 8, 2048, 14336, 4096))


# ------------------------------------------------------------------------------------------------ kernels
def bench_rows(t: Table, T: int, size) -> None:
    from easydel_b200.ops import kernels as K, latent, rotation, stream
    from easydel_b200.ops.moe_kernels import ExpertRows

    W, H, D, R, V, L, E, k, F, ff, _ = size
    name = f"rows {T}, width {W}"
    x, y, w = _rand(T, W, dtype=torch.float32), _rand(T, W, dtype=torch.float32), 0.1 * _rand(W, dtype=torch.float32)
    xb, wb, rb = _rand(T, W), _rand(W), _rand(T, W)
    add_norm = (lambda: K.rmsnorm_fwd(xb, wb, 1e-6, residual=rb, want_rstd=False), T * W * 8)
    t.add("norm after the sum", name, (lambda: stream.post_norm(x, y, 1.0, w, 1e-6, BF, 1.0), T * W * 14),
          "rmsnorm with residual add", add_norm)
    ys, wts = _rand(T * k, W), torch.rand(T, k, device="cuda")
    pos = torch.randperm(T * k, device="cuda").to(torch.int32)
    rows, out = ExpertRows(ys, wts, pos), torch.empty(T, W, dtype=BF, device="cuda")
    from easydel_b200.ops import _lib

    t.add(f"norm after the sum of {k} experts", name,
          (lambda: stream.post_norm(x, rows, 1.0, w, 1e-6, BF, 1.0), T * W * (10 + 2 * k)), "moe combine (no norm)",
          (lambda: _lib.call("edl_moe_combine", ys.data_ptr(), wts.data_ptr(), pos.data_ptr(), out.data_ptr(), T, k, W, 0,
                             _lib.stream_ptr()), T * W * (2 + 2 * k)))
    proj = _rand(T, H * (D + R) + L + R + H * V)
    pages = torch.zeros(T // 128 + 2, 128, 1, L + R, dtype=BF, device="cuda")
    sl, p = torch.arange(T, device="cuda", dtype=torch.int32) + 128, torch.arange(T, dtype=torch.int32, device="cuda")
    nw, freq = torch.ones(L, device="cuda"), rotation.pair_frequencies(1e4, R, "cuda")
    packed = _rand(T, (H + 1) * R)
    cos, moved = torch.rand(T, R // 2, device="cuda"), torch.empty_like(packed)
    t.add("latent prologue (rotate, norm, append)", f"{name}, {H} heads",
          (lambda: latent.prologue(proj, (H, D, R, L), nw, 1e-6, freq, p, sl, pages), 4 * T * (H * R + L + R)),
          "rope over the rotary parts alone, contiguous",
          (lambda: K.rope_copy(packed, moved, p, cos, cos, H + 1, R), 4 * T * (H + 1) * R))
    o, gated = _rand(T, H, V), torch.empty(T, H * V, dtype=BF, device="cuda")
    gate, gu = proj[:, -H * V:], _rand(T, 2 * H * V)
    t.add("head gate", f"rows {T}, {H} x {V}", (lambda: latent.head_gate(o, gate, gated), 6 * T * H * V), "gated silu",
          (lambda: K.gated_act_fwd(gu, "silu"), 6 * T * H * V))
    z, gz = _rand(T, ff), _rand(T, 2 * ff)
    t.add("gelu (erf)", f"rows {T}, ff {ff}", (lambda: stream.gelu_erf(z), 4 * T * ff), "gated silu",
          (lambda: K.gated_act_fwd(gz, "silu"), 6 * T * ff))
    for what, n, kk in (("packed projection", proj.shape[1], W), ("out projection, fp32 result", W, H * V),
                        ("down projection, fp32 result", W, ff)):
        a, b = _rand(T, kk), _rand(n, kk, scale=1 / math.sqrt(kk))
        f32 = "fp32" in what
        yb = torch.empty(T, n, dtype=BF, device="cuda")
        t.add(what, f"{T} x {n} x {kk}",
              (lambda: stream.linear(a, b, out_dtype=torch.float32 if f32 else None),
               2 * (T * kk + n * kk) + (4 if f32 else 2) * T * n, 2 * T * n * kk),
              "same product, bf16 output", (lambda: K.gemm(a, b, out=yb), 2 * (T * kk + n * kk + T * n), 2 * T * n * kk))


def bench_experts(t: Table, T: int, size) -> None:
    from easydel_b200.ops import kernels as K, moe_kernels as MK, stream

    W, H, D, R, V, L, E, k, F, ff, _ = size
    h, wr, corr = _rand(T, W), _rand(E, W, scale=W ** -0.5), 0.1 * _rand(E, dtype=torch.float32)
    logits = stream.linear(h, wr, None, torch.float32)

    def like_route():
        s = torch.sigmoid(logits)
        idx = (s + corr).topk(k, dim=-1).indices
        w = s.gather(-1, idx)
        return w / w.sum(-1, keepdim=True).clamp_min(1e-20), MK.Routing(idx, E)

    nb = T * E * 4 + T * k * 12
    t.add("routing and expert tables", f"rows {T}, {k} of {E}", (lambda: MK.SigmoidRouting(logits, corr, k), nb),
          "the same in tensor operations and bucket kernels", (like_route, nb))
    gu, dn = _rand(E, 2 * F, W, scale=W ** -0.5), _rand(E, W, F, scale=F ** -0.5)
    r = MK.SigmoidRouting(logits, corr, k)
    w, r2 = like_route()
    used = min(E, T * k)
    nb = 2 * used * 3 * F * W + 4 * T * W + 8 * T * k * F
    fl = 6 * T * k * W * F
    idx = torch.topk(torch.sigmoid(logits) + corr, k, dim=-1).indices
    t.add("clamped experts (gather, products, unit)", f"rows {T}, {k} of {E}, {W} x {F}",
          (lambda: MK.clamped_experts(h, r, gu, dn, 7.0), nb, fl), "routed silu experts (with tables and combine)",
          (lambda: MK.moe_ffn(h, gu, dn, w, idx, "silu"), nb, fl))
    act, x2 = torch.empty(r.max_rows, F, dtype=BF, device="cuda"), _rand(r.max_rows, 2 * F)
    from easydel_b200.ops import _lib

    t.add("clamped unit", f"rows {T * k} of {r.max_rows}, ff {F}",
          (lambda: _lib.call("edl_moe_glu", x2.data_ptr(), 0, r.row_token.data_ptr(), r.meta.data_ptr(), act.data_ptr(), F,
                             r.max_rows, 7.0, 1.702, _lib.stream_ptr()), 6 * T * k * F),
          "gated silu over all rows", (lambda: K.gated_act_fwd(x2, "silu"), 6 * T * k * F))


def bench_decode(t: Table, B: int, ctx: int, size, window: int) -> None:
    from easydel_b200.ops import kernels as K, latent, serving as S

    W, H, D, R, V, L = size[:6]
    per = ctx // 128
    pages = _rand(B * per + 1, 128, 1, L + R)
    table = (torch.randperm(B * per, device="cuda") + 1).to(torch.int32).view(B, per)
    lens = torch.full((B,), ctx, dtype=torch.int32, device="cuda")
    q, sinks = _rand(B, H, L + R), torch.ones(H, device="cuda")
    n = latent.decode_splits(B, H, window, ctx, K.sm_count(q.device))
    seen = min(ctx, window or ctx)
    lens2 = torch.full((B,), seen, dtype=torch.int32, device="cuda")
    nb = lambda s: 2 * B * (s * (L + R) + H * (2 * L + R))  # noqa: E731
    fl = lambda s: 2 * B * H * s * (2 * L + R)              # noqa: E731
    t.add("latent decode, window and sinks", f"{B} rows over {ctx} keys, window {window}, {H} heads, {n} splits",
          (lambda: S.latent_decode(q[..., :L], q[..., L:], pages, lens, table, scale=0.07, window=window, sinks=sinks,
                                   num_splits=n), nb(seen), fl(seen)),
          "latent decode of as many keys, no sinks (512 + 64)",
          (lambda: S.mla_decode_attention(q, pages, lens2, table, scale=0.07, num_splits=n), nb(seen), fl(seen)))
    qn, up = _rand(B, H, D), _rand(H, D, L)
    t.add("fold the key up-projection", f"{B} rows", (lambda: torch.bmm(qn.transpose(0, 1), up),
                                                      2 * (B * H * (D + L) + H * D * L), 2 * B * H * D * L),
          "the same as an einsum", (lambda: torch.einsum("thn,hnl->thl", qn, up), 2 * (B * H * (D + L) + H * D * L),
                                    2 * B * H * D * L))


def bench_prefill(t: Table, T: int, size) -> None:
    from easydel_b200.ops import _lib, kernels as K, latent, serving as S

    W, H, D, R, V, L, *_, window = size
    n = T // 128
    pages = _rand(n + 1, 128, 1, L + R)
    src = (torch.randperm(n, device="cuda") + 1).to(torch.int32)
    ctx = torch.empty(T, L + R, dtype=BF, device="cuda")
    t.add("gather the visible pages", f"{T} rows of {L + R}",
          (lambda: _lib.call("edl_gather_pages", pages.data_ptr(), src.data_ptr(), ctx.data_ptr(), n, 256 * (L + R),
                             _lib.stream_ptr()), 4 * T * (L + R)), "index_select",
          (lambda: torch.index_select(pages, 0, src), 4 * T * (L + R)))
    up = _rand(H * D + H * V, L, scale=L ** -0.5)
    wx = latent.expansion_weight(up, H, D, R, V, L)
    N = wx.shape[0]
    lat = _rand(T, L)
    t.add("expand keys and values", f"{T} x {N} x {L + R}",
          (lambda: K.gemm(ctx, wx), 2 * (T * (L + R) + N * (L + R) + T * N), 2 * T * N * (L + R)),
          "up-projection of the latents alone",
          (lambda: K.gemm(lat, up), 2 * (T * L + up.numel() + T * up.shape[0]), 2 * T * up.shape[0] * L))
    lens = torch.full((1,), T, dtype=torch.int32, device="cuda")
    cu = torch.tensor([0, T], dtype=torch.int32, device="cuda")
    sinks = torch.ones(H, device="cuda")

    def case(d, v, win, sink):
        k, vv, table = _pages(1, T, H, d, v)
        q = _rand(T, H, d)
        s = min(T, win or T)
        pairs = H * (s * (s + 1) / 2 + (T - s) * s)
        nb = 2 * T * H * 2 * (d + v)
        if d <= 128:
            return (lambda: S.paged_attention(q, k, vv, cu, lens, table, T, scale=d ** -0.5, sinks=sink, window=win), nb,
                    2 * pairs * (d + v))
        out = torch.empty(T, H, v, dtype=BF, device="cuda")
        return (lambda: _lib.call("edl_attn_paged", q.data_ptr(), k.data_ptr(), vv.data_ptr(), out.data_ptr(), q.stride(0),
                                  k.stride(1), vv.stride(1), H * v, cu.data_ptr(), lens.data_ptr(), table.data_ptr(),
                                  table.stride(0), 1, T, T, k.shape[0], H, H, d, v, float(d ** -0.5), 1, win, 0, 0.0,
                                  _lib.ptr(sink), _lib.status_word(q.device).data_ptr(), _lib.stream_ptr()), nb,
                2 * pairs * (d + v))

    for win in (window, 0):
        t.add("prefill attention over expanded keys, sinks", f"{T} tokens, window {win or 'none'}, {H} heads {D + R} / {V}",
              case(D + R, V, win, sinks), "128 / 128 without sinks", case(128, 128, win, None))
    t.add("prefill attention over expanded keys, sinks", f"{T} tokens, window {window}, {H} heads 96 / 96",
          case(96, 96, window, sinks), "128 / 128 without sinks", case(128, 128, window, None))


def bench_kernels() -> list[dict]:
    t = Table()
    with torch.no_grad():
        for size in SIZES:
            for T in (8192, 64):
                bench_rows(t, T, size)
                bench_experts(t, T, size)
            for B, ctx, window in ((64, 1024, 1024), (64, 8192, size[-1]), (8, 8192, size[-1]), (256, 1024, 1024)):
                bench_decode(t, B, ctx, size, window)
            bench_prefill(t, 8192, size)
    return t.rows


# ------------------------------------------------------------------------------------------------ models
def _models(size, layers: int):
    """(name, constructor) of stacks with equal width, depth, heads, latents and experts."""
    from easydel_b200.infra.factory import TaskType, _ensure_models_imported, registry

    _ensure_models_imported()
    W, H, D, R, V, L, E, k, F, ff, window = size

    def build(mtype, **kw):
        reg = registry.get_module_registration(TaskType.CAUSAL_LM, mtype)
        return reg.module.sequential_init(reg.config(**kw), dtype=BF, param_dtype=BF, device="cuda", seed=1).eval()

    def entry(mlp, win):
        mixer = {"heads": H, "dim": D, "rot_dim": R, "vdim": V, "kv_rank": L, "scale": (D + R) ** -0.5,
                 "rot": {"base": 1e4, "dims": R}}
        return {"type": "latent_attention", "mlp": mlp, "mixer": {**mixer, "mask": {"size": win}} if win else mixer}

    moe = {"kind": "moe", "router": {"experts": E, "top": k}, "expert": {"ff": F, "limit": 7.0}}
    gated = 2 * ff // 3 // 64 * 64
    for name, win in (("disunex", window), ("disunex, no window", None)):
        stack = [entry({"kind": "dense", "ff": ff}, win)] + [entry(moe, win)] * (layers - 1)
        yield name, lambda stack=stack: build("disunex", layers=stack, vocab=VOCAB, width=W, postln_alpha=2.0)
    yield "deepseek_v3", lambda: build(
        "deepseek_v3", vocab_size=VOCAB, hidden_size=W, intermediate_size=gated, moe_intermediate_size=F,
        num_hidden_layers=layers, num_attention_heads=H, num_key_value_heads=H, n_shared_experts=0, n_routed_experts=E,
        kv_lora_rank=L, q_lora_rank=None, qk_rope_head_dim=R, v_head_dim=V, qk_nope_head_dim=D, num_experts_per_tok=k,
        first_k_dense_replace=1, n_group=1, topk_group=1, norm_topk_prob=True, routed_scaling_factor=1.0,
        max_position_embeddings=16384, tie_word_embeddings=True)


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
