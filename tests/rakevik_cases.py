"""Small Rakevik models, written to checkpoint folders, and engines over them: shared by the CPU and GPU tests."""

from __future__ import annotations

import json

import oracle_rakevik as O
import torch

from easydel_b200.inference.esurge import eSurge
from easydel_b200.inference.esurge.replay import TraceReplayer, engine_limits


def hgrn2(heads, dim, vdim, ff=None):
    return {"type": "hgrn2", "mixer": {"heads": heads, "dim": dim, "vdim": vdim},
            "mlp": {"kind": "dense", "ff": ff} if ff else None}


def attention(heads, kv_heads, dim, vdim, scale, coef=None, every=50, ff=None):
    m = {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "scale": scale}
    if coef is not None:
        m["q_temp"] = {"coef": coef, "every": every}
    return {"type": "attention", "mixer": m, "mlp": {"kind": "dense", "ff": ff} if ff else None}


CONFIGS = {
    # grouped queries (a group of three), values narrower than keys, a loop in the middle, FF on a recurrent layer
    "looped": O.random_config(
        [attention(6, 2, 48, 24, 0.2, 0.5, 10, ff=96), hgrn2(3, 24, 40, ff=72), attention(4, 1, 16, 56, 0.3),
         hgrn2(2, 40, 16)], 96, 130, loop={"start": 1, "stop": 3, "times": 3}, eps=1e-5),
    # no loop, one kind of attention shape, wide values
    "plain": O.random_config(
        [hgrn2(2, 16, 32), attention(8, 4, 32, 96, 0.15, 1.1, 7, ff=64), hgrn2(1, 72, 48, ff=40)], 72, 101),
    # the loop covers everything and runs once; heads wider than a tensor-core tile; sizes that are not multiples of 8
    "odd": O.random_config(
        [attention(3, 3, 20, 12, 0.25, 0.2, 33), hgrn2(2, 12, 10, ff=44), attention(2, 1, 136, 144, 0.1, ff=20)],
        60, 53, loop={"start": 0, "stop": 3, "times": 1}, eps=1e-3),
    # recurrent layers only / attention layers only
    "recurrent": O.random_config([hgrn2(2, 32, 64, ff=64), hgrn2(4, 8, 8)], 64, 64,
                                 loop={"start": 1, "stop": 2, "times": 2}),
    "attention": O.random_config([attention(4, 2, 64, 64, 0.125, ff=128), attention(2, 2, 128, 64, 0.1, 0.3, 16)],
                                 128, 90),
}


def write_checkpoint(folder, cfg, weights) -> str:
    from safetensors.torch import save_file

    folder.mkdir(parents=True, exist_ok=True)
    (folder / "config.json").write_text(json.dumps(cfg))
    save_file({k: v.contiguous() for k, v in weights.items()}, str(folder / "model.safetensors"))
    return str(folder)


def load(folder, dtype, device):
    from easydel_b200.modules.auto import AutoEasyDeLModelForCausalLM

    return AutoEasyDeLModelForCausalLM.from_pretrained(folder, dtype=dtype, device=device)


def make(tmp_path, name, dtype, device, seed=0, cfg=None, weights=None):
    cfg = cfg or CONFIGS[name]
    w = weights or O.random_weights(cfg, seed)
    return cfg, w, load(write_checkpoint(tmp_path / name, cfg, w), dtype, device)


def replayer(model, max_tokens=1024, max_requests=4):
    eng = eSurge(model, async_scheduling=False, **engine_limits(max_tokens, max_requests, 128))
    return TraceReplayer(eng)


def tokens(n, vocab, seed=0):
    return torch.randint(0, vocab, (n,), generator=torch.Generator().manual_seed(seed)).tolist()


def run_cut(rep, rid, toks, cuts, end=True):
    """Feeds ``toks`` in portions of the given sizes (the last one repeats) and returns all logits [T, vocab]."""
    out, at, i = [], 0, 0
    while at < len(toks):
        n = min(cuts[min(i, len(cuts) - 1)], len(toks) - at)
        part = toks[at:at + n]
        at += n
        out.append(rep.step([{"id": rid, "tokens": part, "want": list(range(n))}],
                            [rid] if end and at == len(toks) else []))
        i += 1
    return torch.cat(out)


def error(got, want):
    """Largest root mean square of a row's difference, against the spread of the reference logits."""
    got, want = got.detach(), want.detach()
    d = got.double() - want.double()
    return float((d.pow(2).mean(-1).sqrt() / want.double().std()).max())
