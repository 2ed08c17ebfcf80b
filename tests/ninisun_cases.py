"""Small Ninisun models, written to checkpoint folders, and engines over them: shared by the CPU and GPU tests."""

from __future__ import annotations

import oracle_ninisun as O
import torch

from rakevik_cases import error, load, replayer, run_cut, tokens, write_checkpoint  # noqa: F401

YARN = {"factor": 4.0, "original": 64, "fast": 8.0, "slow": 1.0}

CONFIGS = {
    # every kind of layer, several shapes and windows, layers without a feed-forward, values narrower and wider than keys,
    # partly rotated heads, a layer that keeps its own values between those that blend
    "mixed": O.random_config(
        [O.windowed(6, 2, 48, 24, 0.2, 33, 5, base=5e3, dims=32, mlp=O.dense(96)),
         O.parallel((4, 1, 32, 40, 0.15, 24, 300.0, YARN), (3, 16), (0.8, 1.3), O.dense(72)),
         O.windowed(4, 4, 16, 40, 0.3, 130, 0, v_mix=False),
         O.parallel((2, 2, 24, 16, 0.2, 24, 90.0, None), (2, 40), (1.5, 0.6)),
         O.windowed(2, 2, 64, 24, 0.2, 20, 40, dims=16, mlp=O.dense(40))], 96, 130),
    # sizes that are not multiples of 8, windows and kept heads of one token, the first layer has no window
    "odd": O.random_config(
        [O.parallel((3, 3, 10, 7, 0.3, 6, 40.0, {"factor": 3.0, "original": 30, "fast": 4.0, "slow": 0.5}), (5, 7), (0.7, 1.1),
                    O.dense(20)),
         O.windowed(3, 1, 20, 12, 0.3, 7, 1, base=99.0, dims=6, mlp=O.dense(11)),
         O.windowed(2, 1, 14, 12, 0.2, 1, 3, mlp=O.dense(20))], 60, 53, eps=1e-3),
    # the sizes of a large model's heads; a group of 17 queries; windows and kept tokens longer than a page
    "wide": O.random_config(
        [O.parallel((17, 1, 128, 128, 0.06, 128, 1e5, {"factor": 2.0, "original": 200, "fast": 32.0, "slow": 1.0}), (2, 64),
                    (0.3, 1.0), O.dense(64)),
         O.windowed(16, 2, 128, 64, 0.06, 260, 130, base=1e5, dims=64, mlp=O.dense(128)),
         O.parallel((8, 2, 64, 128, 0.09, 16, 1e4, YARN), (1, 128), (0.5, 0.8), O.dense(96)),
         O.windowed(34, 2, 64, 64, 0.09, 150, 7)], 128, 90),
    # attention heads that fit the tiles beside states, ranks and gates that do not; no feed-forward anywhere
    "uneven": O.random_config(
        [O.parallel((3, 1, 32, 40, 0.2, 10, 700.0, YARN), (3, 21), (1.2, 0.9)),
         O.windowed(5, 1, 40, 16, 0.2, 50, 2, dims=6, v_mix=False),
         O.parallel((7, 7, 16, 8, 0.3, 16, 700.0, None), (1, 50), (0.9, 1.4))], 68, 59),
    # one kind of layer only; factors of one
    "windowed": O.random_config([O.windowed(4, 2, 32, 32, 0.2, 64, 2, mlp=O.dense(64)),
                                 O.windowed(8, 2, 64, 32, 0.1, 20, 129, dims=2)], 72, 64),
    "twin": O.random_config([O.parallel((5, 5, 16, 24, 0.25, 16, 50.0, YARN), (4, 32), mlp=O.dense(48)),
                             O.parallel((2, 1, 64, 64, 0.125, 8, 50.0, None), (4, 32))], 64, 70),
}


def make(tmp_path, name, dtype, device, seed=0, cfg=None, weights=None):
    cfg = cfg or CONFIGS[name]
    w = weights or O.random_weights(cfg, seed, rank=5 if name in ("odd", "uneven") else 24 if name == "wide" else 8)
    return cfg, w, load(write_checkpoint(tmp_path / name, cfg, w), dtype, device)


def greedy(cfg, w, prompt, n):
    toks = list(prompt)
    for _ in range(n):
        toks.append(int(O.forward(cfg, w, toks)[-1].argmax()))
    return toks[len(prompt):]


def bf16_floor(cfg, w, toks):
    """Logits of the plain form with everything rounded to bf16: how far 16-bit rounding alone moves them."""
    return error(O.forward(cfg, w, toks, dtype=torch.bfloat16).float(), O.forward(cfg, w, toks))


def feed(rep, plan, seqs):
    """Runs a schedule ``[[(name, tokens), ...], ...]`` over ``seqs``; returns every sequence's logits."""
    got, at = {n: [] for n in seqs}, {n: 0 for n in seqs}
    for step in plan:
        entries, end = [], []
        for n, k in step:
            entries.append({"id": n, "tokens": seqs[n][at[n]:at[n] + k], "want": list(range(k))})
            at[n] += k
            if at[n] == len(seqs[n]):
                end.append(n)
        lg = rep.step(entries, end)
        for n, k in step:
            got[n].append(lg[:k])
            lg = lg[k:]
    assert all(at[n] == len(t) for n, t in seqs.items())
    return {n: torch.cat(v) for n, v in got.items()}
