"""HGRN2 token mixer, a gated linear recurrence without keys: channels write with the complement of their forget gate
(``ops.ssm.hgrn2``).

Per head, with a ``[dim, vdim]`` state: ``q = silu(W_q h)``, ``v = W_v h``, ``f = lower + (1 - lower) sigmoid(W_f h + b)``,
``S <- diag(f) S + (1 - f) v^T``, ``o = S^T q``; each head's ``o`` is RMS-normed with a weight shared by the heads. The
three projections are one product; gates, state and norm are fp32. The output projection is applied by the decoder
layer, which accumulates it into its fp32 residual stream.
"""

from __future__ import annotations

import torch
from torch import nn

from ..ops import ssm, stream
from .linears import ColumnParallelLinear, RowParallelLinear


class HGRN2Mixer(nn.Module):
    def __init__(self, hidden_size: int, heads: int, dim: int, vdim: int, norm_eps: float = 1e-6, layer_idx: int = 0,
                 dtype: torch.dtype = torch.float32, init_std: float = 0.02):
        super().__init__()
        self.heads, self.dim, self.vdim, self.eps, self.layer_idx = heads, dim, vdim, norm_eps, layer_idx
        self.qfv_proj = ColumnParallelLinear(hidden_size, (heads * dim, heads * dim, heads * vdim), bias=False,
                                             dtype=dtype, init_std=init_std)
        self.o_proj = RowParallelLinear(heads * vdim, hidden_size, bias=False, dtype=dtype, init_std=init_std)
        self.f_bias = nn.Parameter(torch.zeros(heads * dim, dtype=torch.float32))
        self.lower = nn.Parameter(torch.zeros(heads * dim, dtype=torch.float32))
        self.norm = nn.Module()
        self.norm.weight = nn.Parameter(torch.ones(vdim, dtype=torch.float32))

    def forward(self, h: torch.Tensor, step, state: torch.Tensor | None) -> torch.Tensor:
        """h ``[T, hidden]`` -> ``[T, heads * vdim]`` before the output projection. ``step``: the running step's sequence
        bounds and slots (:class:`..modules._base.decoder.StreamStep`); ``state``: fp32 pool ``[slots, heads, dim, vdim]``."""
        proj = stream.linear(h, self.qfv_proj.weight)
        return ssm.hgrn2(proj, (self.heads, self.dim, self.vdim), self.f_bias, self.lower, self.norm.weight, self.eps,
                         step.cu, step.max_len, step.slots, state)
