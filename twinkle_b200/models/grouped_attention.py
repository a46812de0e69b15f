"""Grouped-query attention of layers that are listed one by one, with the options of ``config.AttentionSpec``: a rotation, or numbers added to
scores by distance; a window or chunks.

    [q | k | v | g] = W_in h                                    one product
    q, k, v ← + bias, normed, rotated                           one pass, which also writes the cache
    o_i = σ(g_i) · Σ_j v_j exp(s_ij) / (e^sink + Σ_j exp(s_ij)),   s_ij = cap(scale · temperature · q_i · k_j) + number(i − j)

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
    number)`` of this layer's pairs in the stack's table of angles.  ``first``: the block reads someone else's input product, from that column
    on, and has none of its own."""

    def __init__(self, width: int, spec: AttentionSpec, eps: float, layer_idx: int, lead: List[Tuple[str, int]] = (), table: Optional[Tuple[int, int]] = None,
                 first: Optional[int] = None):
        super().__init__()
        self.spec, self.eps, self.layer_idx, self.table = spec, eps, layer_idx, table
        self.source = layer_idx if spec.kv_from is None else spec.kv_from
        parts = list(lead) + spec.in_parts()
        self.in_proj = Linear(width, sum(n for _, n in parts), parts=parts) if first is None else None
        self.first = sum(n for _, n in lead) if first is None else first
        own, H = spec.kv_from is None, spec.heads
        rows = (H, spec.kv_heads) if spec.qk_norm == 'whole' else (1, 1)
        vector = lambda n: nn.Parameter(torch.zeros(n))  # noqa: E731
        self.qkv_bias = vector(sum(spec.qkv_sizes)) if spec.bias else None
        self.head_q_norm = RMSNorm(spec.dim * rows[0], eps) if spec.qk_norm else None
        self.head_k_norm = RMSNorm(spec.dim * rows[1], eps) if spec.qk_norm and own else None
        self.sinks = vector(H) if spec.sinks else None
        self.temperature = nn.Parameter(torch.ones(H)) if spec.temperature else None
        self.log_slope = nn.Parameter(torch.ones(H)) if spec.log_bias else None
        self.log_rate = nn.Parameter(torch.ones(H)) if spec.log_bias else None
        self.distance_table = nn.Parameter(torch.zeros(spec.buckets, H)) if spec.buckets else None
        self._buckets: Dict[torch.device, torch.Tensor] = {}
        self.o_proj = Linear(H * spec.vdim, width, name='o_proj')
        self.o_bias = vector(width) if spec.out_bias else None

    @staticmethod
    def from_columns(spec: AttentionSpec, x: torch.Tensor) -> Tuple[torch.Tensor, torch.Tensor]:
        """Lent columns of the layer-boundary tensor → keys and values."""
        k, v = x.split([spec.kv_heads * spec.dim, spec.kv_heads * spec.vdim], -1)
        return k.reshape(-1, spec.kv_heads, spec.dim), v.reshape(-1, spec.kv_heads, spec.vdim)

    @staticmethod
    def to_columns(spec: AttentionSpec, held: Tuple[torch.Tensor, torch.Tensor]) -> torch.Tensor:
        return torch.cat([held[0][..., :spec.dim].flatten(1), held[1][..., :spec.vdim].flatten(1)], -1)

    def terms(self, device: torch.device) -> Optional[ops.ScoreTerms]:
        """What happens to a score beyond its scale."""
        sp = self.spec
        if not (sp.softcap or sp.temperature or sp.log_bias or sp.buckets):
            return None
        bucket = None
        if sp.buckets:
            bucket = self._buckets.get(device)
            if bucket is None:      # kept per device; not a buffer, which would follow the model's dtype
                bucket = self._buckets[device] = torch.tensor(sp.distance_buckets(), dtype=torch.int32, device=device)
        return ops.ScoreTerms(sp.softcap, self.temperature, self.log_slope, self.log_rate, self.distance_table, bucket)

    def heads(self, p: torch.Tensor, batch):
        """The input product → queries, keys and values (None in single steps, which find them in the cache); the cache is written."""
        sp, view = self.spec, batch.cache
        own = sp.kv_from is None
        qw, kw = self.head_q_norm.weight if sp.qk_norm else None, self.head_k_norm.weight if sp.qk_norm and own else None
        sizes = sp.heads, sp.kv_heads if own else 0, sp.dim, sp.vdim, self.eps, view, self.layer_idx
        if sp.rotary is not None:
            return ops.rotary_heads(p, self.first, self.qkv_bias, qw, kw, batch.rotary, *self.table, sp.rotary.interleaved, *sizes)
        return ops.plain_heads(p, self.first, self.qkv_bias, qw, kw, sp.value_norm, sp.values_are_keys, *sizes)

    def attend(self, p: torch.Tensor, batch, held: Dict[int, Any]) -> torch.Tensor:
        """The input product → the output projection's result without its bias."""
        sp, view, T = self.spec, batch.cache, p.shape[0]
        g0 = self.first + sum(sp.qkv_sizes)
        gate = p[:, g0:g0 + sp.heads] if sp.head_gate else p[:, g0:g0 + sp.heads * sp.vdim] if sp.out_gate else None
        q, k, v = self.heads(p, batch)
        terms = self.terms(p.device)
        if view is not None and view.stepping:
            o = ops.paged_attention_decode(q, view.cache.k[self.source], view.cache.v[self.source], view.table, view.seq_lens, sp.scale, window=sp.window or None,
                                           sinks=self.sinks, chunk=sp.chunk, gate=gate, terms=terms)
        else:
            if sp.kv_from is None:
                held[self.layer_idx] = k, v
            o = ops.attention_packed(q, *held[self.source], batch.cu_seqlens, batch.max_seqlen, sp.scale, self.sinks, gate, sp.window, sp.chunk, terms=terms)
        if o.shape[-1] != sp.vdim:          # rows were filled up to whole vectors
            o = o[..., :sp.vdim]
        return self.o_proj(o.reshape(T, sp.heads * sp.vdim))

    def forward(self, h: torch.Tensor, batch, held: Dict[int, Any]) -> Tuple[torch.Tensor, torch.Tensor]:
        """``(result [T, width], the input product)``; keys and values formed here are left in ``held`` under this layer's index."""
        p = self.in_proj(h)
        y = self.attend(p, batch, held)
        return (y if self.o_bias is None else y + self.o_bias), p
