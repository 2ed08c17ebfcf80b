"""Generalised delta rule as a token mixer without projections of its own (``ops.ssm.generalized_delta_rule``).

Per head, with a ``[dim, vdim]`` state: every key channel decays by ``w = exp(-rate sigmoid(W2 tanh(W1 h) + w0))``, what the
state holds along the unit key ``u`` is removed at the rate ``a = sigmoid(W_a h + a0)``, and ``k v^T`` is added: ``S <- diag(w)
S - (a u) (u^T S) + k v^T``, ``o = S^T r``. Each head's ``o`` is RMS-normed, times a weight over all heads, times ``sigmoid(W_g
h)``. The caller hands in the columns of one packed projection (:attr:`in_splits`) and applies the output projection.
"""

from __future__ import annotations

import math

import torch
from torch import nn

from ..ops import ssm
from .linears import ColumnParallelLinear


class GeneralizedDeltaMixer(nn.Module):
    def __init__(self, heads: int, dim: int, rank: int, vdim: int | None = None, rate: float = math.exp(-0.5),
                 unit_eps: float = 1e-6, norm_eps: float = 1e-6, dtype: torch.dtype = torch.float32, init_std: float = 0.02):
        super().__init__()
        self.heads, self.dim, self.vdim, self.rank = heads, dim, vdim or dim, rank
        self.rate, self.unit_eps, self.eps = rate, unit_eps, norm_eps
        self.decay_up = ColumnParallelLinear(rank, heads * dim, bias=False, dtype=dtype, init_std=init_std)
        self.decay_bias = nn.Parameter(torch.zeros(heads * dim, dtype=torch.float32))
        self.rate_bias = nn.Parameter(torch.zeros(heads * dim, dtype=torch.float32))
        self.norm = nn.Module()
        self.norm.weight = nn.Parameter(torch.ones(heads * self.vdim, dtype=torch.float32))

    @property
    def in_splits(self) -> tuple[int, ...]:
        """Widths of r, k, v, removal rate, gate and the input of the low-rank decay."""
        k, v = self.heads * self.dim, self.heads * self.vdim
        return k, k, v, k, v, self.rank

    @property
    def out_width(self) -> int:
        return self.heads * self.vdim

    def mix_rows(self, cols: ssm.DeltaColumns, step, state: torch.Tensor | None, out: torch.Tensor | None = None,
                 out_scale: float = 1.0) -> torch.Tensor:
        """``[T, heads * vdim]`` (into ``out`` if given), times ``out_scale``. ``step``: the running step's sequence bounds
        and slots (:class:`..modules._base.decoder.StreamStep`); ``state``: fp32 pool ``[slots, heads, dim, vdim]``."""
        wt = ssm.DeltaWeights(self.decay_up.weight, self.decay_bias, self.rate_bias, self.norm.weight, self.rate, self.unit_eps,
                              self.eps)
        return ssm.generalized_delta_rule(cols, (self.heads, self.dim, self.vdim), wt, step.cu, step.max_len, step.slots, state,
                                          out_scale, out)
