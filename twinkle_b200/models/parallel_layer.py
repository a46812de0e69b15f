"""Decoder layers whose mixer and feed-forward block stand side by side on one norm, with a 32-bit residual stream.

One layer of a stack whose layers are listed one by one (``DecoderConfig.layer_specs``; Pomelix checkpoints):

    h = rmsnorm(x)                                                  x: fp32 stream, h: compute dtype
    [q | k | v | gate | up] = W_in h                                one product: both sub-layers read the same h
    q, k, v = short convolution → q, k over their rms per head → query temperature, value mixing
    x ← x + m · (W_o attention(q, k, v) ⊙ s_mixer + W_down (silu(gate) · up) ⊙ s_mlp)

Positions enter through the convolution and the query temperature only (no rotary embedding).  The update of the stream is
left pending at the end of a layer and carried out by the kernel that forms the next layer's norm (``Stream``), so that a
forward without gradients passes over the stream once per layer.  With gradients the stream is one tensor
``[x | values of the first mixing layer]`` per layer boundary, which is what activation recompute keeps.
"""
from __future__ import annotations

from dataclasses import dataclass, field
from typing import Dict, List, Optional, Tuple

import torch
import torch.nn as nn

from .. import ops
from .config import DecoderConfig
from .layers import Linear, RMSNorm


@dataclass
class CacheView:
    """Where the tokens of one forward live in the sampler's cache (``sampler.engine.PagedKVCache``).  With ``table`` and
    ``seq_lens`` every row is the next token of a sequence that is already there; without them the rows are whole prompts,
    packed, and their keys, values and convolution history are only written."""
    cache: object
    rows: torch.Tensor                          # [T] int64: row of each token in the flat key / value pools
    slots: torch.Tensor                         # [T] int32: slot of the token's sequence in the history and state pools
    left: torch.Tensor                          # [T] int32: later tokens of the same sequence in this forward
    table: Optional[torch.Tensor] = None        # [B, blocks] int32
    seq_lens: Optional[torch.Tensor] = None     # [B] int32, the new token included

    @property
    def stepping(self) -> bool:
        return self.table is not None


@dataclass
class GatedResult:
    """A sub-layer's result on its way into the stream: ``norm(σ(gate + bias) ⊙ result)``.  ``result [T, W]``, or expert rows
    with the places ``row_of [T, k]`` and weights ``share [T, k]`` of every token's."""
    result: torch.Tensor
    gate: torch.Tensor                          # [T, ≥ W]: the gate's projection in the leading columns
    bias: torch.Tensor
    norm: RMSNorm
    row_of: Optional[torch.Tensor] = None
    share: Optional[torch.Tensor] = None


@dataclass
class PlainResult:
    """A sub-layer's result on its way into the stream as it is: ``result [T, W]``, or expert rows with the places ``row_of [T, k]`` and
    weights ``share [T, k]`` of every token's, plus ``beside [T, W]`` times ``open [T]`` (the shared expert)."""
    result: torch.Tensor
    row_of: Optional[torch.Tensor] = None
    share: Optional[torch.Tensor] = None
    beside: Optional[torch.Tensor] = None
    open: Optional[torch.Tensor] = None


@dataclass
class NormedResult:
    """A sub-layer's result on its way into the stream: ``norm(result + bias)``, or with a second one ``norm(½ (inner(result + bias) +
    beside_inner(beside)))``."""
    result: torch.Tensor
    norm: RMSNorm
    bias: Optional[torch.Tensor] = None
    inner: Optional[RMSNorm] = None
    beside: Optional[torch.Tensor] = None
    beside_inner: Optional[RMSNorm] = None


@dataclass
class Stream:
    """The residual stream between layers: ``x`` (fp32) plus sub-layer results that have not joined it yet (``adds`` times
    ``mult``, one gated and normed result, one plain or one normed result), and what later layers take from earlier ones (``held``: layer → tensor)."""
    x: torch.Tensor
    adds: List[Tuple[torch.Tensor, torch.Tensor]] = field(default_factory=list)
    held: Dict[int, torch.Tensor] = field(default_factory=dict)
    mult: float = 1.0
    gated: Optional[GatedResult] = None
    plain: Optional[PlainResult] = None
    normed: Optional[NormedResult] = None

    def enter(self, norm: Optional[RMSNorm], dtype: Optional[torch.dtype] = None) -> torch.Tensor:
        """What is pending joins the stream; returns its norm (None: the stream itself, in ``dtype``) in the compute dtype — one kernel."""
        if self.normed is not None:
            y, w = self.normed, lambda n: None if n is None else n.weight  # noqa: E731
            h, self.x = ops.stream_normed(self.x, w(norm), y.norm.eps, y.result, y.bias, y.norm.weight, w(y.inner), y.beside, w(y.beside_inner))
        elif norm is None and self.gated is self.plain is None and not self.adds:
            h = self.x.to(dtype)
        elif self.gated is not None:
            g = self.gated
            h, self.x = ops.stream_gated_rmsnorm(self.x, norm.weight, norm.eps, norm.offset, g.result, g.gate, g.bias, g.norm.weight, g.row_of, g.share)
        elif self.plain is not None:
            y = self.plain
            h, self.x = ops.stream_joined_rmsnorm(self.x, norm.weight, norm.eps, norm.offset, y.result, y.row_of, y.share, y.beside, y.open)
        else:
            h, self.x = ops.stream_rmsnorm(self.x, norm.weight, norm.eps, self.adds, self.mult, norm.offset)
        self.adds, self.gated, self.plain, self.normed = [], None, None, None
        return h


class ParallelLayer(nn.Module):
    is_linear = is_moe = False

    def __init__(self, cfg: DecoderConfig, layer_idx: int):
        super().__init__()
        sp = self.spec = cfg.layer_specs[layer_idx]
        self.layer_idx, self.eps, self.mult, self.width = layer_idx, cfg.rms_norm_eps, float(cfg.residual_multiplier), cfg.hidden_size
        q, k, v = sp.qkv_sizes
        self.values_of = cfg.first_mixing_layer
        self.gives_values = layer_idx == self.values_of
        self.takes_values = sp.v_mix and not self.gives_values
        self.input_layernorm = RMSNorm(cfg.hidden_size, cfg.rms_norm_eps)
        parts = [('q_proj', q), ('k_proj', k), ('v_proj', v)] + ([('gate_proj', sp.ff), ('up_proj', sp.ff)] if sp.ff else [])
        self.in_proj = Linear(cfg.hidden_size, sum(n for _, n in parts), parts=parts)
        self.conv_weight = nn.Parameter(torch.empty(q + k + v, sp.conv)) if sp.conv else None
        self.v_lambda = nn.Parameter(torch.full((1, ), 0.5)) if sp.v_mix else None      # unused in the layer that gives the values
        self.o_proj = Linear(sp.heads * sp.vdim, cfg.hidden_size, name='o_proj')
        self.mixer_scale = nn.Parameter(torch.ones(cfg.hidden_size))
        self.down_proj = Linear(sp.ff, cfg.hidden_size, name='down_proj') if sp.ff else None
        self.mlp_scale = nn.Parameter(torch.ones(cfg.hidden_size)) if sp.ff else None

    def sublayers(self, h: torch.Tensor, batch, v_first: Optional[torch.Tensor]):
        """Both sub-layers on the normalised stream: ``([(result, channel scale), …], values of this layer)``."""
        sp, view = self.spec, batch.cache
        p = self.in_proj(h)
        q, k, v = ops.conv_heads(p, self.conv_weight, batch.position_ids, sp.heads, sp.kv_heads, sp.dim, sp.vdim, self.eps, sp.temp_coef, sp.temp_every,
                                 v_first if self.takes_values else None, self.v_lambda if self.takes_values else None, view, self.layer_idx)
        if view is not None and view.stepping:
            o = ops.paged_attention_decode(q, view.cache.k[self.layer_idx], view.cache.v[self.layer_idx], view.table, view.seq_lens, sp.scale)
        else:
            o = ops.attention_packed(q, k, v, batch.cu_seqlens, batch.max_seqlen, sp.scale)
        if o.shape[-1] != sp.vdim:          # rows were filled up to whole vectors
            o = o[..., :sp.vdim]
        adds = [(self.o_proj(o.reshape(o.shape[0], -1)), self.mixer_scale)]
        if self.down_proj is not None:
            gate = sum(sp.qkv_sizes)
            adds.append((self.down_proj(ops.glu_columns(p, gate, gate + sp.ff, sp.ff)), self.mlp_scale))
        return adds, v

    def advance(self, st: Stream, batch) -> Stream:
        """One layer without gradients: pending results of the layer below join the stream in this layer's norm kernel."""
        h = st.enter(self.input_layernorm)
        st.adds, v = self.sublayers(h, batch, st.held.get(self.values_of))
        st.mult = self.mult
        if self.gives_values:
            st.held[self.layer_idx] = v
        return st

    def forward(self, x: torch.Tensor, cos, sin, batch, kv_sink=None) -> torch.Tensor:
        """``x [T, width + values]`` fp32 → the same after this layer (see the module's docstring)."""
        x, held = x[:, :self.width], x[:, self.width:]
        h, _ = ops.stream_rmsnorm(x.contiguous(), self.input_layernorm.weight, self.eps)
        sp = self.spec
        v_first = held.to(h.dtype).view(-1, sp.kv_heads, sp.vdim) if self.takes_values else None
        adds, v = self.sublayers(h, batch, v_first)
        if self.gives_values:
            held = v[..., :sp.vdim].reshape(v.shape[0], -1).float()
        return torch.cat([x + self.mult * sum(y.float() * sc.float() for y, sc in adds), held], -1)
