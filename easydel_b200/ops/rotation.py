"""Rotary angles computed where they are used, for layers over an fp32 stream.

Frequencies are kept as fp32 leading parts followed by the fp32 remainders, so that the kernels' angles ``position *
frequency`` are as exact as 32-bit results can be at any position, without a table. A pair is either two neighbours
``(2i, 2i + 1)`` or the elements ``i`` and ``i + dims / 2`` of the rotated part."""

from __future__ import annotations

import math

import torch

#: which elements of the rotated part turn together
LAYOUTS = ("neighbours", "halves")


def llama3_scaling(f: torch.Tensor, factor: float, low: float, high: float, original: float) -> torch.Tensor:
    """Llama 3.1's frequency scaling: wavelengths below ``original / high`` stay, those above ``original / low`` grow by
    ``factor``, and the ones in between are blended. In ``f``'s type."""
    wave = 2 * math.pi / f
    s = (original / wave - low) / (high - low)
    out = torch.where(wave > original / low, f / factor, f)
    between = (wave >= original / high) & (wave <= original / low)
    return torch.where(between, (1 - s) * f / factor + s * f, out)


def yarn_scaling(f: torch.Tensor, base: float, dims: int, factor: float, original: float, fast: float,
                 slow: float) -> torch.Tensor:
    """YaRN's frequency scaling: pairs that turn at least ``fast`` times within ``original`` positions stay, those that turn
    at most ``slow`` times are slowed down by ``factor``, with a linear ramp over the pair index in between. In ``f``'s type."""
    def index_of(turns):
        return dims * math.log(original / (2 * math.pi * turns)) / (2 * math.log(base))

    lo, hi = max(math.floor(index_of(fast)), 0), min(math.ceil(index_of(slow)), dims - 1)
    ramp = ((torch.arange(f.numel(), dtype=f.dtype) - lo) / max(hi - lo, 0.001)).clamp(0, 1)
    return f / factor * ramp + f * (1 - ramp)


def magnitude(scaling: dict | None) -> float:
    """Factor of cosines and sines: ``0.1 ln(factor) + 1`` under :func:`yarn_scaling`, else 1."""
    return 0.1 * math.log(float(scaling["factor"])) + 1.0 if scaling and "fast" in scaling else 1.0


def pair_frequencies(base: float, dims: int, device=None, scaling: dict | None = None) -> torch.Tensor:
    """``base^(-2i / dims)`` for i < dims / 2, as leading parts and remainders. ``scaling``: the ``factor``, ``low``,
    ``high`` and ``original`` of :func:`llama3_scaling`, or the ``factor``, ``original``, ``fast`` and ``slow`` of
    :func:`yarn_scaling`."""
    f = float(base) ** (-torch.arange(0, dims, 2, dtype=torch.float64) / dims)
    if scaling and "fast" in scaling:
        f = yarn_scaling(f, float(base), dims, *(float(scaling[k]) for k in ("factor", "original", "fast", "slow")))
    elif scaling:
        f = llama3_scaling(f, *(float(scaling[k]) for k in ("factor", "low", "high", "original")))
    hi = f.float()
    return torch.cat([hi, (f - hi.double()).float()]).to(device)


def rotate(x: torch.Tensor, positions: torch.Tensor, freq: torch.Tensor, layout: str = "neighbours",
           mag: float = 1.0) -> torch.Tensor:
    """Tensor form: the pairs of the first ``2 * pairs`` elements of ``x [T, ..., R]`` turned by ``position *
    frequency`` and scaled by ``mag``; computed in fp32, cast back."""
    n = freq.numel() // 2
    a = positions.double()[:, None] * (freq[:n].double() + freq[n:].double())
    c, s = (torch.cos(a) * mag).float(), (torch.sin(a) * mag).float()
    c, s = (t.view(t.shape[0], *[1] * (x.dim() - 2), n) for t in (c, s))
    if layout == "halves":
        u, v = x[..., :n].float(), x[..., n:2 * n].float()
        r = torch.cat([u * c - v * s, v * c + u * s], -1)
    else:
        u, v = x[..., 0:2 * n:2].float(), x[..., 1:2 * n:2].float()
        r = torch.stack([u * c - v * s, v * c + u * s], -1).flatten(-2)
    return torch.cat([r.to(x.dtype), x[..., 2 * n:]], -1)


def check_rotation(dims: int, width: int, layout: str) -> None:
    if layout not in LAYOUTS:
        raise ValueError(f"rotation layout {layout!r} is none of {LAYOUTS}")
    if dims % 2 or not 0 <= dims <= width:
        raise ValueError(f"{dims} rotated channels of {width}")
