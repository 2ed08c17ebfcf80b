"""Small Disunex models, written to checkpoint folders, and engines over them: shared by the CPU and GPU tests."""

from __future__ import annotations

import oracle_disunex as O
import torch

from rakevik_cases import error, load, replayer, run_cut, tokens, write_checkpoint  # noqa: F401


def _shared():
    a = O.latent(4, 32, 16, 48, 64, 0.2, base=5e3, window=33, mlp=O.dense(96))
    b = O.latent(6, 24, 8, 32, 40, 0.25, base=800.0, window=130, mlp=O.experts(8, 3, 40, 0.9))
    c = O.latent(4, 32, 16, 48, 64, 0.2, base=5e3, window=33, mlp=None)
    layers = [a, b, c]
    return [*layers, O.again(layers, 1), O.again(layers, 0), O.again(layers, 2)]


CONFIGS = {
    # several shapes and windows, a layer without a feed-forward, every kind of layer used twice
    "shared": O.random_config(_shared(), 96, 130, alpha=2.3, eps=1e-5),
    # no shared weights, one expert per token, a window longer than a page, seven heads
    "plain": O.random_config([O.latent(7, 64, 32, 64, 128, 0.1, window=150, mlp=O.experts(4, 1, 64, 2.0)),
                              O.latent(7, 64, 32, 64, 128, 0.1, window=150, mlp=O.dense(160))], 72, 104, alpha=1.0),
    # sizes that are not multiples of 8, a window of one token, partly rotated rotary part, many experts
    "odd": O.random_config([O.latent(3, 20, 6, 12, 18, 0.3, base=99.0, window=7, mlp=O.experts(37, 5, 11, 0.5), dims=4),
                            O.latent(2, 10, 10, 30, 26, 0.2, window=1, mlp=O.dense(44))], 60, 53, alpha=0.6, eps=1e-3),
    # without a mask the whole past is visible; the sizes of a large model's heads
    "wide": O.random_config([O.latent(2, 128, 64, 128, 512, 0.06, mlp=O.dense(64)),
                             O.latent(17, 96, 64, 40, 200, 0.08, window=260, mlp=O.experts(64, 6, 24, 1.5))], 128, 90,
                            alpha=3.5),
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
