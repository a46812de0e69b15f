"""Grouped-query attention of layers that are listed one by one: a rotation, a window or chunks, and the options of ``config.AttentionSpec``.

    [q | k | v | g] = W_in h                                    one product
    q, k, v ← + bias;  q, k ← rotated rms norm per head         one pass, which also writes the cache
    o_i = σ(g_i) · Σ_j v_j exp(s_ij) / (e^sink + Σ_j exp(s_ij)),   s_ij = scale · q_i · k_j

A layer may read the keys and values of an earlier one (``AttentionSpec.kv_from``), as that layer's cache holds them: it then has queries
only and keeps nothing of its own.
"""
from __future__ import annotations

from typing import Any, Dict, List, Optional, Tuple

import torch
import torch.nn as nn

from .. import ops
from .config import AttentionSpec
from .layers import Linear, RMSNorm


class GroupedAttention(nn.Module):
    """``lead``: projections of the same input that are not this block's, in the leading columns of its input product.  ``table``: ``(first,
    number)`` of this layer's pairs in the stack's table of angles."""

    def __init__(self, width: int, spec: AttentionSpec, eps: float, layer_idx: int, lead: List[Tuple[str, int]] = (), table: Optional[Tuple[int, int]] = None):
        super().__init__()
        self.spec, self.eps, self.layer_idx, self.table = spec, eps, layer_idx, table
        self.source = layer_idx if spec.kv_from is None else spec.kv_from
        parts = list(lead) + spec.in_parts()
        self.in_proj = Linear(width, sum(n for _, n in parts), parts=parts)
        self.first = sum(n for _, n in lead)
        own = spec.kv_from is None
        self.qkv_bias = nn.Parameter(torch.zeros(sum(spec.qkv_sizes))) if spec.bias else None
        self.head_q_norm = RMSNorm(spec.dim, eps) if spec.qk_norm else None
        self.head_k_norm = RMSNorm(spec.dim, eps) if spec.qk_norm and own else None
        self.sinks = nn.Parameter(torch.zeros(spec.heads)) if spec.sinks else None
        self.o_proj = Linear(spec.heads * spec.vdim, width, name='o_proj')

    @staticmethod
    def from_columns(spec: AttentionSpec, x: torch.Tensor) -> Tuple[torch.Tensor, torch.Tensor]:
        """Lent columns of the layer-boundary tensor → keys and values."""
        k, v = x.split([spec.kv_heads * spec.dim, spec.kv_heads * spec.vdim], -1)
        return k.reshape(-1, spec.kv_heads, spec.dim), v.reshape(-1, spec.kv_heads, spec.vdim)

    @staticmethod
    def to_columns(spec: AttentionSpec, held: Tuple[torch.Tensor, torch.Tensor]) -> torch.Tensor:
        return torch.cat([held[0][..., :spec.dim].flatten(1), held[1][..., :spec.vdim].flatten(1)], -1)

    def forward(self, h: torch.Tensor, batch, held: Dict[int, Any]) -> Tuple[torch.Tensor, torch.Tensor]:
        """``(result [T, width], the input product)``; keys and values formed here are left in ``held`` under this layer's index."""
        sp, view, T = self.spec, batch.cache, h.shape[0]
        own = sp.kv_from is None
        p = self.in_proj(h)
        g0 = self.first + sum(sp.qkv_sizes)
        gate = p[:, g0:g0 + sp.heads] if sp.head_gate else None
        q, k, v = ops.rotary_heads(p, self.first, self.qkv_bias, self.head_q_norm.weight if sp.qk_norm else None, self.head_k_norm.weight if sp.qk_norm and own else None,
                                   batch.rotary, *self.table, sp.rotary.interleaved, sp.heads, sp.kv_heads if own else 0, sp.dim, sp.vdim, self.eps, view, self.layer_idx)
        if view is not None and view.stepping:
            o = ops.paged_attention_decode(q, view.cache.k[self.source], view.cache.v[self.source], view.table, view.seq_lens, sp.scale, window=sp.window or None,
                                           sinks=self.sinks, chunk=sp.chunk, gate=gate)
        else:
            if own:
                held[self.layer_idx] = k, v
            o = ops.attention_packed(q, *held[self.source], batch.cu_seqlens, batch.max_seqlen, sp.scale, self.sinks, gate, sp.window, sp.chunk)
        if o.shape[-1] != sp.vdim:          # rows were filled up to whole vectors
            o = o[..., :sp.vdim]
        return self.o_proj(o.reshape(T, sp.heads * sp.vdim)), p
