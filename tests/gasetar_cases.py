"""Small Gasetar models, written to checkpoint folders, and engines over them: shared by the CPU and GPU tests."""

from __future__ import annotations

import oracle_gasetar as O
import torch

from rakevik_cases import error, load, replayer, run_cut, tokens, write_checkpoint  # noqa: F401

CONFIGS = {
    # every kind of layer and feed-forward, several shapes and windows, a layer without a feed-forward, values narrower and
    # wider than keys, partly rotated heads, all three bands of the frequency scaling
    "mixed": O.random_config(
        [O.windowed(6, 2, 48, 24, 0.2, 33, 4.0, base=5e3, dims=32, scaling=(3.0, 1.0, 4.0, 40), mlp=O.experts(8, 3, 40, 24)),
         O.latent(4, 32, 16, 48, 64, 0.2, base=800.0, mlp=O.dense(96)),
         O.windowed(4, 4, 16, 40, 0.3, 130, 9.0, mlp=None),
         O.latent(6, 24, 8, 32, 40, 0.25, base=60.0, mlp=O.experts(16, 1, 16))], 96, 130, eps=1e-5),
    # sizes that are not multiples of 8, a window of one token, as many choices as experts
    "odd": O.random_config(
        [O.windowed(3, 1, 20, 12, 0.3, 7, 2.5, base=99.0, dims=6, scaling=(2.0, 0.5, 8.0, 20), mlp=O.experts(5, 5, 11, 13)),
         O.latent(2, 10, 6, 30, 26, 0.2, mlp=O.dense(44)), O.windowed(2, 2, 14, 22, 0.2, 1, 3.0, mlp=O.dense(20))], 60, 53,
        mult=1.3, eps=1e-3, embed_scale=0.7, logit_scale=1.7, logit_cap=2.0),
    # the sizes of a large model's heads; a group of 17 queries; a window longer than a page
    "wide": O.random_config(
        [O.latent(17, 96, 64, 128, 512, 0.08, mlp=O.experts(64, 6, 24, 32)),
         O.windowed(16, 2, 128, 64, 0.06, 260, 20.0, base=1e5, dims=64, scaling=(8.0, 1.0, 4.0, 300), mlp=O.dense(128)),
         O.windowed(34, 2, 64, 128, 0.09, 150, 6.0, dims=0, mlp=O.experts(24, 4, 16, 8))], 128, 90, mult=0.4),
    # one kind of mixer only; factors of one and no caps
    "latent": O.random_config([O.latent(5, 16, 8, 24, 32, 0.3, mlp=O.experts(8, 2, 24)), O.latent(5, 16, 8, 24, 32, 0.3)], 64,
                              70, mult=1.0, embed_scale=1.0, logit_scale=1.0, logit_cap=0.0),
    "windowed": O.random_config([O.windowed(4, 2, 32, 32, 0.2, 64, 0.0, mlp=O.dense(64)),
                                 O.windowed(8, 8, 64, 16, 0.1, 20, 5.0, dims=2, mlp=O.experts(4, 2, 32, 64))], 72, 64),
}


def make(tmp_path, name, dtype, device, seed=0, cfg=None, weights=None):
    cfg = cfg or CONFIGS[name]
    w = weights or O.random_weights(cfg, seed)
    return cfg, w, load(write_checkpoint(tmp_path / name, cfg, w), dtype, device)


def greedy(cfg, w, prompt, n):
    toks = list(prompt)
    for _ in range(n):
        toks.append(int(O.forward(cfg, w, toks)[-1].argmax()))
    return toks[len(prompt):]


def bf16_floor(cfg, w, toks):
    """Logits of the plain form with every product's operands rounded to bf16: how far 16-bit rounding alone moves them."""
    return error(O.forward(cfg, w, toks, dtype=torch.bfloat16).float(), O.forward(cfg, w, toks))
