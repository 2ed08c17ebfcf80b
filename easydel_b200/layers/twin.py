"""Two mixers side by side: attention over pages and a recurrence with a state, both reading the same rows.

All projections of both are one product of the layer's input, and both write into one row ``[attention | recurrence]`` whose
output projection is one product too: the factors of the two sides are folded into what they write.
"""

from __future__ import annotations

import torch
from torch import nn

from ..ops import ssm, stream
from .attention import Attention
from .delta_rule import GeneralizedDeltaMixer
from .linears import ColumnParallelLinear, RowParallelLinear


class TwinMixer(nn.Module):
    """``left_scale * left(h) + right_scale * right(h)``; the sides come without projections of their own."""

    def __init__(self, hidden_size: int, left: Attention, right: GeneralizedDeltaMixer, scales: tuple[float, float],
                 dtype: torch.dtype = torch.float32, init_std: float = 0.02):
        super().__init__()
        self.left, self.right, self.scales = left, right, (float(scales[0]), float(scales[1]))
        *wide, gate = left.in_splits
        # whole heads first; the widths that may be no multiple of 8 (the rank of the decay, a number per head) come last
        self.twin_proj = ColumnParallelLinear(hidden_size, (*wide, *right.in_splits, gate), bias=False, dtype=dtype,
                                            init_std=init_std)
        self.o_proj = RowParallelLinear(left.out_width + right.out_width, hidden_size, bias=False, dtype=dtype,
                                        init_std=init_std)

    def mix_stream(self, h: torch.Tensor, step, view, state: torch.Tensor | None) -> torch.Tensor:
        """h ``[T, hidden]`` -> ``[T, left + right]`` before the output projection. ``view``: the layer's pages; ``state``: the
        recurrence's pool."""
        rows = stream.linear(h, self.twin_proj.weight)
        parts = torch.split(rows, self.twin_proj.out_splits, -1)
        qkv = rows[:, :sum(self.twin_proj.out_splits[:3])]
        r, k, v, a, g, x = parts[3:9]
        cols = ssm.DeltaColumns(r, k, v, a, g, x)
        n, (ls, rs) = self.left.out_width, self.scales
        if stream.on_kernels(h):
            width = n + self.right.out_width
            out = torch.empty(h.shape[0], (width + 7) // 8 * 8, dtype=h.dtype, device=h.device)[:, :width]   # aligned rows
            self.left.mix_rows(qkv, step, view, gate=parts[9], out=out[:, :n], out_scale=ls)
            self.right.mix_rows(cols, step, state, out[:, n:], rs)
            return out
        return torch.cat([self.left.mix_rows(qkv, step, view, gate=parts[9], out_scale=ls),
                          self.right.mix_rows(cols, step, state, None, rs)], -1)
