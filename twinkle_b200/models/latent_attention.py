"""Latent attention: what the cache keeps of a token is one normed vector that all heads share, and a few rotated key dimensions.

    c_q = norm(W_dq h),  q = W_uq c_q     or     q = W_q h              queries through a bottleneck, or plain
    [c | r] = W_dkv h,  c ← norm(c)                                     one latent per token, and (with positions) a rotated key part
    k = [W_uk c | r],  v = W_uv c                                       expanded per head; the rotated part is the same for all
    o_i = σ(g_i) · Σ_j v_j exp(s_ij) / (e^sink + Σ_j exp(s_ij)),  s_ij = scale · q_i · k_j      (sink and gate where the layer has them)

Prompts expand keys and values once and run packed attention.  A step never expands the context: ``q_i · W_uk c_j = (W_ukᵀ q_i) · c_j``,
so the query is taken into latent space, attends over the cached rows, of which the latent is key and value at once, and the result goes
through ``W_uv``.  A layer may read the latents of an earlier one (``LatentSpec.kv_from``): it then keeps nothing of its own.
"""
from __future__ import annotations

from typing import Dict, List, Optional, Tuple

import torch
import torch.nn as nn

from .. import ops
from .config import LatentSpec
from .layers import Linear, RMSNorm


class LatentAttention(nn.Module):
    """``lead``: projections of the same input that are not this block's, in the leading columns of its input product.  ``table``: ``(first,
    number)`` of this layer's pairs in the stack's table of angles."""

    def __init__(self, width: int, spec: LatentSpec, eps: float, layer_idx: int, lead: List[Tuple[str, int]] = (), table: Optional[Tuple[int, int]] = None):
        super().__init__()
        self.spec, self.eps, self.layer_idx, self.table = spec, eps, layer_idx, table or (0, 0)
        self.source = layer_idx if spec.kv_from is None else spec.kv_from
        parts = list(lead) + spec.in_parts()
        self.in_proj = Linear(width, sum(n for _, n in parts), parts=parts)
        self.first = sum(n for _, n in lead)
        self.q_norm = RMSNorm(spec.q_rank, eps) if spec.q_rank else None
        self.kv_norm = RMSNorm(spec.kv_rank, eps) if spec.kv_from is None else None
        self.q_up = Linear(spec.q_rank, spec.heads * spec.dim, name='q_up') if spec.q_rank else None
        # [W_uk | W_uv], used as one matrix by prompts and head by head by steps (hence no adapter of its own)
        self.kv_up = nn.Parameter(torch.empty(spec.heads * (spec.dim + spec.vdim), spec.kv_rank))
        self.sinks = nn.Parameter(torch.zeros(spec.heads)) if spec.sinks else None
        self.o_proj = Linear(spec.heads * spec.vdim, width, name='o_proj')

    @staticmethod
    def from_columns(spec: LatentSpec, x: torch.Tensor) -> torch.Tensor:
        """Lent columns of the layer-boundary tensor → ``[latent | rotated key part]``."""
        return x

    @staticmethod
    def to_columns(spec: LatentSpec, held: torch.Tensor) -> torch.Tensor:
        return held[:, :spec.lent_columns()]

    def queries(self, p: torch.Tensor, batch):
        """The input product → ``(q [T, H, dim + rot_dim], [latent | rotated key part] of this layer or None, the rotated queries of a step at
        their place in latent space [T, H, kv_rank + rot_dim] or None)``; the cache is written."""
        sp, own, T = self.spec, self.kv_norm is not None, p.shape[0]
        R, wc = sp.kv_rank if own else 0, self.kv_norm.weight if own else None
        if self.q_up is None:
            return ops.latent_rotary(p, self.first, sp.heads, sp.dim, sp.rot_dim, self.first + sp.heads * sp.qk_width, R, wc, self.eps, batch.rotary, *self.table,
                                     sp.rotary.interleaved if sp.rotary else False, sp.kv_rank, batch.cache, self.layer_idx)
        cq, c = ops.latent_norms(p, self.first, sp.q_rank, self.q_norm.weight, self.first + sp.q_rank, R, wc, self.eps, batch.cache, self.layer_idx)
        return self.q_up(cq).view(T, sp.heads, sp.dim), c, None

    def forward(self, h: torch.Tensor, batch, held: Dict[int, torch.Tensor]) -> Tuple[torch.Tensor, torch.Tensor]:
        """``(result [T, width], the input product)``; a latent formed here is left in ``held`` under this layer's index."""
        sp, view, T = self.spec, batch.cache, h.shape[0]
        H, d, e, R, r = sp.heads, sp.dim, sp.vdim, sp.kv_rank, sp.rot_dim
        p = self.in_proj(h)
        g0 = self.first + sum(n for _, n in sp.in_parts()) - H
        gate = p[:, g0:g0 + H] if sp.head_gate else None
        q, kept, ql = self.queries(p, batch)
        if kept is not None:
            held[self.layer_idx] = kept
        if view is not None and view.stepping:
            ql = ops.head_linear(q[..., :d], self.kv_up[:H * d].view(H, d, R), transposed=True, out=ql)
            o = ops.latent_decode(ql, view.cache.k[self.source], view.table, view.seq_lens, sp.scale, self.sinks, gate, R, sp.window)
            o = ops.head_linear(o, self.kv_up[H * d:].view(H, e, R))
        else:
            kept = held[self.source]
            kv = ops.linear(kept[:, :R], self.kv_up)
            k, v = kv[:, :H * d].view(T, H, d), kv[:, H * d:].view(T, H, e)
            o = ops.attention_packed(q, k, v, batch.cu_seqlens, batch.max_seqlen, sp.scale, self.sinks, gate, sp.window, key_tail=kept[:, R:R + r] if r else None)
        return self.o_proj(o.reshape(T, H * e)), p
