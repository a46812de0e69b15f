"""Latent attention without positions: what the cache keeps of a token is one normed vector that all heads share.

    c_q = norm(W_dq h),  q = W_uq c_q                                 queries through a bottleneck
    c   = norm(W_dkv h),  k = W_uk c,  v = W_uv c                      one latent per token, expanded per head
    o_i = σ(g_i) · Σ_j v_j exp(s_ij) / (e^sink + Σ_j exp(s_ij)),  s_ij = scale · q_i · k_j  (j ≤ i)

Prompts expand keys and values once and run packed attention.  A step never expands the context: ``q_i · W_uk c_j = (W_ukᵀ q_i) · c_j``,
so the query is taken into latent space, attends over the cached latents as key and value at once, and the result goes through
``W_uv``.  A layer may read the latents of an earlier one (``LatentSpec.kv_from``): it then keeps nothing of its own.
"""
from __future__ import annotations

from typing import Dict, List, Optional, Tuple

import torch
import torch.nn as nn

from .. import ops
from .config import LatentSpec
from .layers import Linear, RMSNorm


class LatentAttention(nn.Module):
    """``lead``: projections of the same input that are not this block's, in the leading columns of its input product."""

    def __init__(self, width: int, spec: LatentSpec, eps: float, layer_idx: int, lead: List[Tuple[str, int]] = ()):
        super().__init__()
        self.spec, self.eps, self.layer_idx = spec, eps, layer_idx
        self.source = layer_idx if spec.kv_from is None else spec.kv_from
        parts = list(lead) + spec.in_parts()
        self.in_proj = Linear(width, sum(n for _, n in parts), parts=parts)
        self.first = sum(n for _, n in lead)
        self.q_norm = RMSNorm(spec.q_rank, eps)
        self.kv_norm = RMSNorm(spec.kv_rank, eps) if spec.kv_from is None else None
        self.q_up = Linear(spec.q_rank, spec.heads * spec.dim, name='q_up')
        # [W_uk | W_uv], used as one matrix by prompts and head by head by steps (hence no adapter of its own)
        self.kv_up = nn.Parameter(torch.empty(spec.heads * (spec.dim + spec.vdim), spec.kv_rank))
        self.sinks = nn.Parameter(torch.zeros(spec.heads))
        self.o_proj = Linear(spec.heads * spec.vdim, width, name='o_proj')

    def forward(self, h: torch.Tensor, batch, held: Dict[int, torch.Tensor]) -> Tuple[torch.Tensor, torch.Tensor]:
        """``(result [T, width], the input product)``; a latent formed here is left in ``held`` under this layer's index."""
        sp, view, T = self.spec, batch.cache, h.shape[0]
        H, d, e, R = sp.heads, sp.dim, sp.vdim, sp.kv_rank
        own = self.kv_norm is not None
        p = self.in_proj(h)
        g0 = self.first + sp.q_rank + (R if own else 0)
        gate = p[:, g0:g0 + H]
        cq, c = ops.latent_norms(p, self.first, sp.q_rank, self.q_norm.weight, self.first + sp.q_rank, R if own else 0,
                                 self.kv_norm.weight if own else None, self.eps, view, self.layer_idx)
        if own:
            held[self.layer_idx] = c
        q = self.q_up(cq).view(T, H, d)
        if view is not None and view.stepping:
            ql = ops.head_linear(q, self.kv_up[:H * d].view(H, d, R), transposed=True)
            o = ops.latent_decode(ql, view.cache.k[self.source], view.table, view.seq_lens, sp.scale, self.sinks, gate)
            o = ops.head_linear(o, self.kv_up[H * d:].view(H, e, R))
        else:
            kv = ops.linear(held[self.source][:, :R], self.kv_up)
            k, v = kv[:, :H * d].view(T, H, d), kv[:, H * d:].view(T, H, e)
            o = ops.attention_packed(q, k, v, batch.cu_seqlens, batch.max_seqlen, sp.scale, self.sinks, gate)
        return self.o_proj(o.reshape(T, H * e)), p
