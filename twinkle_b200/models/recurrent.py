"""Recurrent mixers of layers that are listed one by one: the selective scan (``Mamba1``) and the matrix memory of xLSTM (``MatrixMemory``).
What a sequence carries from token to token lives in slots of the sampler's cache, in 32-bit.
"""
from __future__ import annotations

from typing import Optional

import torch
import torch.nn as nn

from .. import ops
from .config import Mamba1Spec, MatrixMemorySpec
from .layers import Linear, RMSNorm


class Mamba1(nn.Module):
    """Per channel c and state n, with step sizes ``δ = softplus(W_dt r + b)``, ``[x | z] = W_in h``, ``u = silu(conv(x))``, ``[r | B | C] = W_x u``:

        S_cn ← exp(−δ_c e^{A_cn}) S_cn + δ_c u_c B_n,     y_c = (Σ_n S_cn C_n + D_c u_c) silu(z_c),     result = W_o y

    Convolution with its activation is one kernel, everything behind ``δ``'s projection another.  ``lead``: projections of the same input that
    are not this block's, in the leading columns of its input product."""

    def __init__(self, width: int, spec: Mamba1Spec, eps: float, layer_idx: int, lead=(), table=None):
        super().__init__()
        self.spec, self.layer_idx, self.first = spec, layer_idx, sum(n for _, n in lead)
        n, parts = spec.inner, list(lead) + spec.in_parts()
        self.in_proj = Linear(width, sum(w for _, w in parts), parts=parts)
        self.conv_weight = nn.Parameter(torch.empty(n, spec.conv))
        self.conv_bias = nn.Parameter(torch.zeros(n))
        self.x_proj = Linear(n, spec.dt_rank + 2 * spec.state, name='x_proj')
        self.dt_proj = Linear(spec.dt_rank, n, name='dt_proj')
        self.dt_bias = nn.Parameter(torch.zeros(n))
        self.A_log = nn.Parameter(torch.zeros(n, spec.state))
        self.D = nn.Parameter(torch.ones(n))
        self.o_proj = Linear(n, width, name='o_proj')

    def forward(self, h: torch.Tensor, batch, held=None):
        """``(result [T, width], the input product)``."""
        sp, n, view = self.spec, self.spec.inner, batch.cache
        p = self.in_proj(h)
        u = ops.conv_silu(p, self.first, n, self.conv_weight, self.conv_bias, batch.position_ids, view, self.layer_idx)
        r = self.x_proj(u)
        dt = self.dt_proj(r[:, :sp.dt_rank])
        y = ops.selective_scan(u, dt, self.dt_bias, self.A_log, r, sp.dt_rank, sp.dt_rank + sp.state, self.D, p, self.first + n, batch.cu_seqlens, batch.max_seqlen, view, self.layer_idx)
        return self.o_proj(y), p


class MatrixMemory(nn.Module):
    """mLSTM: per head a matrix ``S [dim, vdim]`` and a normaliser ``n [dim]``, with log gates ``i = cap(W_i h + b)`` and ``f = log σ(cap(W_f h + b))``
    and a running maximum ``m`` that starts at 0:

        m' = max(f + m, i),   S ← e^{f + m − m'} S + e^{i − m'} k vᵀ,   n ← likewise with k,   o = Sᵀ q / (max(|n·q|, e^{−m'}) + 10⁻⁶)

    (``q`` scaled by ``dim^−½``); heads over their root mean square, times a weight, times ``σ(W_g h)``, then projected.  Everything between the two
    products is one kernel.  ``first``: see ``GroupedAttention``."""

    def __init__(self, width: int, spec: MatrixMemorySpec, eps: float, layer_idx: int, lead=(), table=None, first: Optional[int] = None):
        super().__init__()
        self.spec, self.eps, self.layer_idx = spec, eps, layer_idx
        parts = list(lead) + spec.in_parts()
        self.in_proj = Linear(width, sum(n for _, n in parts), parts=parts) if first is None else None
        self.first = sum(n for _, n in lead) if first is None else first
        self.i_bias = nn.Parameter(torch.zeros(spec.heads))
        self.f_bias = nn.Parameter(torch.zeros(spec.heads))
        self.out_norm = RMSNorm(spec.heads * spec.vdim, eps)        # its weight; the kernel norms head by head
        self.o_proj = Linear(spec.heads * spec.vdim, width, name='o_proj')

    def remember(self, p: torch.Tensor, batch) -> torch.Tensor:
        """The input product → the output projection's result."""
        sp = self.spec
        o = ops.matrix_memory(p, self.first, sp.heads, sp.dim, sp.vdim, self.i_bias, self.f_bias, sp.gate_cap, self.out_norm.weight, self.eps, batch.cu_seqlens,
                              batch.max_seqlen, batch.cache, self.layer_idx)
        return self.o_proj(o)

    def forward(self, h: torch.Tensor, batch, held=None):
        """``(result [T, width], the input product)``."""
        p = self.in_proj(h)
        return self.remember(p, batch), p
