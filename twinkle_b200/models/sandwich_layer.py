"""Decoder layers with a norm in front of and behind each sub-layer, a gate on its result, and a 32-bit residual stream.

One layer of a stack whose layers are listed one by one (``DecoderConfig.layer_specs``; Moronex checkpoints):

    h = norm(x),   y = mixer(h),          x ← x + norm(σ(W_g h + b) ⊙ y)         mixer: latent attention or HGRN2
    h = norm(x),   y = feed_forward(h),   x ← x + norm(σ(W_g h + b) ⊙ y)         gated block, experts, or absent

The gate's projection rides in the sub-layer's input product.  Gate, norm and sum of a result are left pending and carried out by
the kernel that forms the next norm (``Stream.enter``), which also combines a token's expert rows: without gradients the stream
is passed over once per sub-layer.  With gradients the stream is one tensor ``[x | latents that later layers borrow]`` per layer
boundary, which is what activation recompute keeps.
"""
from __future__ import annotations

import torch
import torch.nn as nn

from .. import ops
from .config import DecoderConfig
from .latent_attention import LatentAttention
from .layers import Linear, RMSNorm
from .linear_attention import HGRN2
from .parallel_layer import GatedResult, Stream

MIXERS = {'latent_attention': LatentAttention, 'hgrn2': HGRN2}


class GatedFeedForward(nn.Module):
    """``W_down (silu(W_gate h) ⊙ W_up h)`` with other projections of ``h`` (``lead``) in front of gate and up in one product."""

    def __init__(self, width: int, ff: int, lead):
        super().__init__()
        self.ff, self.first = ff, sum(n for _, n in lead)
        self.in_proj = Linear(width, self.first + 2 * ff, parts=list(lead) + [('gate_proj', ff), ('up_proj', ff)])
        self.down_proj = Linear(ff, width, name='down_proj')

    def forward(self, h: torch.Tensor):
        p = self.in_proj(h)
        return self.down_proj(ops.glu_columns(p, self.first, self.first + self.ff, self.ff)), p


class SandwichLayer(nn.Module):
    is_linear = False

    def __init__(self, cfg: DecoderConfig, layer_idx: int):
        super().__init__()
        sp = self.spec = cfg.layer_specs[layer_idx]
        self.layer_idx, self.width, self.eps = layer_idx, cfg.hidden_size, cfg.rms_norm_eps
        self.is_moe = sp.is_moe
        self.moe_index = sum(s.is_moe for s in cfg.layer_specs[:layer_idx])      # place in recorded routing lists
        self.columns, at = {}, cfg.hidden_size                                   # lent latents in the layer-boundary tensor
        for j, n in cfg.held_columns():
            self.columns[j] = (at, at + n)
            at += n
        norm = lambda: RMSNorm(cfg.hidden_size, cfg.rms_norm_eps, cfg.rms_norm_offset)  # noqa: E731
        lead = [('res_gate', cfg.hidden_size)]
        self.input_layernorm, self.post_mixer_layernorm = norm(), norm()
        self.mixer = MIXERS[sp.mixer.kind](cfg.hidden_size, sp.mixer, cfg.rms_norm_eps, layer_idx, lead)
        self.mixer_gate_bias = nn.Parameter(torch.zeros(cfg.hidden_size))
        self.mlp = self.mlp_gate = None
        if sp.mlp is None:
            return
        self.pre_mlp_layernorm, self.post_mlp_layernorm = norm(), norm()
        self.mlp_gate_bias = nn.Parameter(torch.zeros(cfg.hidden_size))
        if self.is_moe:
            from .decoder import MoEBlock
            self.mlp_gate = Linear(cfg.hidden_size, cfg.hidden_size, name='res_gate')
            self.mlp = MoEBlock(DecoderConfig(hidden_size=cfg.hidden_size, num_experts=sp.mlp.experts, num_experts_per_tok=sp.mlp.top,
                                              moe_intermediate_size=sp.mlp.ff, router_scoring='topk_softmax', router_linear_bias=True,
                                              expert_act='relu2'), layer_idx)
        else:
            self.mlp = GatedFeedForward(cfg.hidden_size, sp.mlp.ff, lead)

    def _forced(self, batch):
        return batch.routed_experts[self.moe_index] if batch.routed_experts is not None else None

    def feed_forward(self, h: torch.Tensor, batch) -> GatedResult:
        if not self.is_moe:
            y, p = self.mlp(h)
            return GatedResult(y, p, self.mlp_gate_bias, self.post_mlp_layernorm)
        gate = self.mlp_gate(h)
        if self.mlp.moe_parallel is None and not torch.is_grad_enabled():
            y, row_of, share = self.mlp.rows(h, self._forced(batch))
            return GatedResult(y, gate, self.mlp_gate_bias, self.post_mlp_layernorm, row_of, share)
        return GatedResult(self.mlp(h, self._forced(batch)), gate, self.mlp_gate_bias, self.post_mlp_layernorm)

    def advance(self, st: Stream, batch) -> Stream:
        """One layer; the result of its last sub-layer stays pending in the stream."""
        y, p = self.mixer(st.enter(self.input_layernorm), batch, st.held)
        st.gated = GatedResult(y, p, self.mixer_gate_bias, self.post_mixer_layernorm)
        if self.mlp is not None:
            st.gated = self.feed_forward(st.enter(self.pre_mlp_layernorm), batch)
        return st

    def forward(self, x: torch.Tensor, cos, sin, batch, kv_sink=None) -> torch.Tensor:
        """``x [T, width + lent latents]`` fp32 → the same after this layer."""
        held = {j: x[:, a:b].to(self.input_layernorm.weight.dtype) for j, (a, b) in self.columns.items()}
        st = self.advance(Stream(x[:, :self.width].clone(), held=held), batch)
        st.enter(self.input_layernorm)          # the sum; the norm formed with it is the next layer's business
        lent = [x[:, a:b] if j != self.layer_idx else st.held[j][:, :b - a].float() for j, (a, b) in self.columns.items()]
        return torch.cat([st.x] + lent, -1)
