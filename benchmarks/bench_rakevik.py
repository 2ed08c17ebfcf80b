"""Speed of the Rakevik family beside the framework's closest models: ``python bench.py --model rakevik`` (or
``python -m benchmarks.bench_rakevik``).

Two parts, each a list of JSON lines. *Kernels*: every kernel of the family at the sizes of a real model's layers, with
the share of its roofline (the measured copy bandwidth or cuBLAS rate, whichever bounds it), and beside it the kernel
that does the like job in an existing model at the same sizes; ``distance_ratio`` is how much farther from its roofline
ours is (below 1: nearer). *Models*: prefill and decode throughput of the serving engine for a Rakevik stack, a
Gated-DeltaNet hybrid (``qwen3_5_text``, the closest model: three recurrent layers to one attention layer, dense MLP) and
an attention-only stack (``qwen3``) of equal width, depth and parameters. Random weights; CUDA events; L2 flushed
between timed launches.
"""

from __future__ import annotations

import argparse
import json
import math

import torch

from benchmarks.bench_kernels import _peaks, time_cuda

BF = torch.bfloat16


def _rand(*s, dtype=BF, scale=1.0):
    return (torch.randn(*s, device="cuda", dtype=torch.float32) * scale).to(dtype)


class Table:
    def __init__(self):
        self.pk = _peaks()
        self.flush = torch.empty(256 << 20, dtype=torch.uint8, device="cuda")
        self.rows = []

    def measure(self, fn, bytes_: float, flops: float = 0.0) -> dict:
        """Time and roofline share: the roofline time is the larger of bytes / copy bandwidth and FLOPs / cuBLAS rate."""
        ms = time_cuda(fn, iters=15, warmup=4, flush=self.flush)
        roof = max(bytes_ / (self.pk["hbm_gbs"] * 1e9), flops / (self.pk["tflops"] * 1e12)) * 1e3
        return {"us": round(ms * 1e3, 2), "roofline_us": round(roof * 1e3, 2), "of_measured_roofline": round(roof / ms, 4)}

    def add(self, name: str, size: str, ours, like_name: str, like):
        a, b = self.measure(*ours), self.measure(*like)
        row = {"kernel": name, "size": size, **a, "like": like_name, "like_us": b["us"],
               "like_of_measured_roofline": b["of_measured_roofline"],
               "distance_ratio": round(b["of_measured_roofline"] / max(a["of_measured_roofline"], 1e-9), 3)}
        self.rows.append(row)
        print(json.dumps(row), flush=True)


# ------------------------------------------------------------------------------------------------ kernels
def _pages(B, ctx, Hkv, D, Dv):
    per = -(-ctx // 128)
    k, v = _rand(B * per + 1, 128, Hkv, D), _rand(B * per + 1, 128, Hkv, Dv)
    table = (torch.randperm(B * per, device="cuda") + 1).to(torch.int32).view(B, per)
    return k, v, table


def bench_rows(t: Table, T: int, W: int, H: int, G: int, D: int, V: int, F: int) -> None:
    """Row kernels and products at ``T`` rows: norms, prologue, activation, projections."""
    from easydel_b200.ops import kernels as K, stream

    size = f"rows {T}, width {W}"
    x, w, mu = _rand(T, W, dtype=torch.float32), _rand(W, dtype=torch.float32), torch.rand(W, device="cuda")
    xb, wb, rb = _rand(T, W), _rand(W), _rand(T, W)
    nseq = T if T <= 256 else 4
    cu = torch.arange(0, T + 1, T // nseq, dtype=torch.int32, device="cuda")
    slots = torch.arange(nseq, dtype=torch.int32, device="cuda")
    state = torch.zeros(nseq, W, device="cuda")
    st = 8 * nseq * W if nseq == T else 0
    t.add("norm_shift", size, (lambda: stream.norm_shift(x, w, 1e-6, BF, mu, cu, slots, state), T * W * 6 + st),
          "rmsnorm with residual add", (lambda: K.rmsnorm_fwd(xb, wb, 1e-6, residual=rb, want_rstd=False), T * W * 8))
    qkv = _rand(T, H * D + G * (D + V))
    kp, vp, _ = _pages(1, max(T, 128), G, D, V)
    sl = (torch.arange(T, device="cuda", dtype=torch.int32) + 128)
    pos = torch.arange(T, dtype=torch.int32, device="cuda")
    qn = torch.ones(D, device="cuda")
    nb = 2 * T * (H * D + G * (D + V)) * 2
    heads = (H, G, D, V)
    packed = _rand(T, (H + 2 * G) * D)
    cos = torch.rand(T, D // 2, device="cuda")
    out = torch.empty_like(packed)
    t.add("qkv_prologue (norm q k, temperature, append)", size,
          (lambda: stream.qkv_prologue(qkv, heads, qn, qn, 1e-6, pos, (0.5, 1024.0), sl, kp, vp), nb),
          "rope over packed qkv (no norm, no append)",
          (lambda: K.rope_copy(packed, out, pos, cos, cos, H + G, D), 2 * T * (H + 2 * G) * D * 2))
    z, act, gu = _rand(T, F), torch.tensor([0.3, 0.3], device="cuda"), _rand(T, 2 * F)
    t.add("xielu", f"rows {T}, ff {F}", (lambda: stream.xielu(z, act), T * F * 4), "gated silu",
          (lambda: K.gated_act_fwd(gu, "silu"), T * F * 6))
    for name, n, k in (("out projection into the fp32 stream", W, H * V), ("down projection into the fp32 stream", W, F)):
        a, b = _rand(T, k), _rand(n, k, scale=1 / math.sqrt(k))
        y = torch.zeros(T, n, dtype=torch.float32, device="cuda")
        yb = torch.empty(T, n, dtype=BF, device="cuda")
        t.add(name, f"{T} x {n} x {k}",
              (lambda: stream.linear_add_(y, a, b), 2 * (T * k + n * k) + 8 * T * n, 2 * T * n * k),
              "same product, bf16 output", (lambda: K.gemm(a, b, out=yb), 2 * (T * k + n * k + T * n), 2 * T * n * k))
    cat, wl, bias = _rand(T, 2 * W), _rand(W, 2 * W, scale=0.02), _rand(W)
    yb = torch.empty(T, W, dtype=BF, device="cuda")
    t.add("loop input product", f"{T} x {W} x {2 * W}",
          (lambda: stream.linear(cat, wl, bias, torch.float32), 2 * (T * 2 * W + 2 * W * W) + 4 * T * W, 4 * T * W * W),
          "same product, bf16 output",
          (lambda: K.gemm(cat, wl, bias=bias, out=yb), 2 * (T * 2 * W + 2 * W * W + T * W), 4 * T * W * W))
    t.add("cast_rows", size, (lambda: stream.cast_rows(x, cat[:, :W]), T * W * 6), "rmsnorm with residual add",
          (lambda: K.rmsnorm_fwd(xb, wb, 1e-6, residual=rb, want_rstd=False), T * W * 8))
    o32, nw = _rand(T, H, V, dtype=torch.float32), torch.ones(V, device="cuda")
    t.add("head_norm", f"{T} x {H} x {V}", (lambda: stream.head_norm(o32, nw, 1e-6, BF), T * H * V * 6), "rmsnorm",
          (lambda: K.rmsnorm_fwd(xb, wb, 1e-6, want_rstd=False), T * W * 4))


def bench_recurrence(t: Table, B: int, L: int, H: int, D: int, V: int) -> None:
    """HGRN2 against the gated delta rule, ``B`` sequences of ``L`` tokens (L = 1: a decode step)."""
    from easydel_b200.ops import ssm

    T = B * L
    proj, bias, low = _rand(T, 2 * H * D + H * V), _rand(H * D, dtype=torch.float32), torch.rand(H * D, device="cuda")
    norm = torch.ones(V, device="cuda")
    cu = torch.arange(0, T + 1, L, dtype=torch.int32, device="cuda")
    slots = torch.arange(B, dtype=torch.int32, device="cuda")
    st = torch.zeros(B, H, D, V, device="cuda")
    q, k, v = _rand(T, H, D, scale=D ** -0.5), _rand(T, H, D, scale=D ** -0.5), _rand(T, H, V)
    g, beta = -torch.rand(T, H, device="cuda"), torch.rand(T, H, device="cuda").to(BF)
    st2 = torch.zeros(B, H, D, V, device="cuda")
    states = 8 * B * H * D * V
    t.add("hgrn2_decode" if L == 1 else "hgrn2_scan (+ output norm)", f"{B} x {L} tokens, {H} heads {D} x {V}",
          (lambda: ssm.hgrn2(proj, (H, D, V), bias, low, norm, 1e-6, cu, L, slots, st),
           2 * T * H * (2 * D + 2 * V) + states),
          "gated delta rule (no output norm)",
          (lambda: ssm.gated_delta_rule(q, k, v, g, beta, None, cu, st2), 2 * T * H * (2 * D + 2 * V) + 6 * T * H + states))


def bench_attention(t: Table, B: int, new: int, ctx: int, H: int, G: int, D: int, V: int) -> None:
    """Paged attention with value heads of their own size against the same kernel at 128 / 128."""
    from easydel_b200.ops import serving as S

    lens = torch.full((B,), ctx, dtype=torch.int32, device="cuda")
    cu = torch.arange(0, B * new + 1, new, dtype=torch.int32, device="cuda")
    sinks = torch.ones(H, device="cuda")
    pairs = B * H * (new * ctx - new * (new - 1) / 2)

    def case(d, v, sink):
        k, vv, table = _pages(B, ctx, G, d, v)
        q = _rand(B * new, H, d)
        nbytes = 2 * B * (ctx * G * (d + v) + new * H * (d + v))
        if new == 1:
            return (lambda: S.decode_attention(q, k, vv, lens, table, scale=d ** -0.5, sinks=sink), nbytes)
        return (lambda: S.paged_attention(q, k, vv, cu, lens, table, new, scale=d ** -0.5, sinks=sink), nbytes,
                2 * pairs * (d + v))

    t.add("decode attention with sinks" if new == 1 else "prefill attention with sinks",
          f"{B} x {new} tokens over {ctx} keys, {H}/{G} heads {D} / {V}", case(D, V, sinks), "128 / 128 without sinks",
          case(128, 128, None))


def bench_kernels() -> list[dict]:
    t = Table()
    with torch.no_grad():
        for W, H, G, F in ((2048, 16, 4, 8192), (4096, 32, 8, 14336)):
            for T in (8192, 64):
                bench_rows(t, T, W, H, G, 128, 128, F)
            bench_recurrence(t, 1, 8192, H, 128, 128)
            bench_recurrence(t, 8, 1024, H, 128, 128)
            for B in (8, 64, 256):
                bench_recurrence(t, B, 1, H, 128, 128)
        for D, V in ((128, 128), (64, 96), (96, 128)):
            bench_attention(t, 1, 8192, 8192, 32, 8, D, V)
            bench_attention(t, 64, 1, 2048, 32, 8, D, V)
    return t.rows


# ------------------------------------------------------------------------------------------------ models
VOCAB = 32768


def _models(W: int, H: int, G: int, F: int, layers: int):
    """(name, constructor) of stacks with equal width, depth and feed-forward parameters."""
    from easydel_b200.infra.factory import TaskType, _ensure_models_imported, registry

    _ensure_models_imported()

    def build(mtype, **kw):
        reg = registry.get_module_registration(TaskType.CAUSAL_LM, mtype)
        return reg.module.sequential_init(reg.config(**kw), dtype=BF, param_dtype=BF, device="cuda", seed=1).eval()

    mlp = {"kind": "dense", "ff": F}
    rec = {"type": "hgrn2", "mixer": {"heads": H, "dim": 128, "vdim": 128}, "mlp": mlp}
    att = {"type": "attention", "mlp": mlp,
           "mixer": {"heads": H, "kv_heads": G, "dim": 128, "vdim": 128, "scale": 128 ** -0.5,
                     "q_temp": {"coef": 0.5, "every": 1024}}}
    gated = 2 * F // 3 // 64 * 64
    common = dict(vocab_size=VOCAB, hidden_size=W, intermediate_size=gated, num_hidden_layers=layers,
                  num_attention_heads=H, num_key_value_heads=G, head_dim=128, tie_word_embeddings=False)
    yield "rakevik", lambda: build("rakevik", layers=[att if i % 4 == 3 else rec for i in range(layers)],
                                   loop={"start": 0, "stop": layers, "times": 1}, vocab=VOCAB, width=W)
    yield "qwen3_5_text", lambda: build("qwen3_5_text", linear_key_head_dim=128, linear_value_head_dim=128,
                                        linear_num_key_heads=H, linear_num_value_heads=H, **common)
    yield "qwen3", lambda: build("qwen3", **common)


def _engine_speed(model, prompt: int, batch: int, ctx: int) -> dict:
    from easydel_b200.inference import SamplingParams
    from easydel_b200.inference.esurge import eSurge

    eng = eSurge(model, max_model_len=max(prompt, ctx + 128) + 128, max_num_seqs=batch, max_num_batched_tokens=prompt,
                 num_pages=max(batch * (-(-(ctx + 128) // 128)), prompt // 128) + 8, enable_prefix_caching=False,
                 async_scheduling=True)
    g = torch.Generator().manual_seed(0)
    toks = lambda n: torch.randint(0, VOCAB, (n,), generator=g).tolist()  # noqa: E731
    ev = lambda: torch.cuda.Event(enable_timing=True)  # noqa: E731
    times = []
    for i in range(3 + 5):
        eng.add_request(toks(prompt), SamplingParams(max_tokens=1, temperature=0.0, ignore_eos=True))
        torch.cuda.synchronize()
        a, b = ev(), ev()
        a.record()
        eng.step()
        b.record()
        torch.cuda.synchronize()
        times.append(a.elapsed_time(b))
        while eng.step():
            pass
    pre = sorted(times[3:])[2]
    for _ in range(batch):
        eng.add_request(toks(ctx), SamplingParams(max_tokens=100, temperature=0.0, ignore_eos=True))
    while eng.scheduler.num_waiting or any(r.num_computed_tokens < r.num_prompt_tokens
                                           for r in eng.scheduler.running):
        eng.step()
    for _ in range(8):                      # warm-up and capture of the decode step
        eng.step()
    torch.cuda.synchronize()
    a, b = ev(), ev()
    a.record()
    for _ in range(32):
        eng.step()
    b.record()
    torch.cuda.synchronize()
    dec = a.elapsed_time(b) / 32
    graphs = bool(eng.runner.use_graphs)
    eng.close()
    return {"prefill_tokens": prompt, "prefill_ms": round(pre, 3), "prefill_tokens_per_s": round(prompt / pre * 1e3),
            "decode_batch": batch, "decode_context": ctx, "decode_ms_per_step": round(dec, 3),
            "decode_tokens_per_s": round(batch / dec * 1e3), "decode_graphs": graphs}


def bench_models() -> list[dict]:
    rows = []
    for W, H, G, F in ((2048, 16, 4, 6144), (4096, 32, 8, 12288)):
        for name, build in _models(W, H, G, F, 8):
            model = build()
            n = sum(p.numel() for p in model.parameters())
            for batch in (8, 64):
                row = {"model": name, "width": W, "layers": 8, "parameters": n, **_engine_speed(model, 8192, batch, 1024)}
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
