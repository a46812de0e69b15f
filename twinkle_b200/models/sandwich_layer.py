"""Decoder layers with a norm in front of and behind each sub-layer, a gate on its result, and a 32-bit residual stream.

One layer of a stack whose layers are listed one by one (``DecoderConfig.layer_specs``; Moronex checkpoints):

    h = norm(x),   y = mixer(h),          x ← x + norm(σ(W_g h + b) ⊙ y)         mixer: latent attention or HGRN2
    h = norm(x),   y = feed_forward(h),   x ← x + norm(σ(W_g h + b) ⊙ y)         gated block, experts, or absent

The gate's projection rides in the sub-layer's input product.  Gate, norm and sum of a result are left pending and carried out by
the kernel that forms the next norm (``Stream.enter``), which also combines a token's expert rows.
"""
from __future__ import annotations

import torch
import torch.nn as nn

from .config import DecoderConfig
from .layers import Linear
from .mixer_layer import GatedFeedForward, MixerLayer
from .parallel_layer import GatedResult, Stream


class SandwichLayer(MixerLayer):

    def __init__(self, cfg: DecoderConfig, layer_idx: int):
        lead = [('res_gate', cfg.hidden_size)]
        super().__init__(cfg, layer_idx, lead)
        sp = self.spec
        self.post_mixer_layernorm = self.norm(cfg)
        self.mixer_gate_bias = nn.Parameter(torch.zeros(cfg.hidden_size))
        self.mlp = self.mlp_gate = None
        if sp.mlp is None:
            return
        self.pre_mlp_layernorm, self.post_mlp_layernorm = self.norm(cfg), self.norm(cfg)
        self.mlp_gate_bias = nn.Parameter(torch.zeros(cfg.hidden_size))
        if self.is_moe:
            self.mlp_gate = Linear(cfg.hidden_size, cfg.hidden_size, name='res_gate')
            self.mlp = self.experts(cfg)
        else:
            self.mlp = GatedFeedForward(cfg.hidden_size, sp.mlp.ff, lead, sp.mlp.limit, sp.mlp.act)

    def feed_forward(self, h: torch.Tensor, batch) -> GatedResult:
        if not self.is_moe:
            y, p = self.mlp(h)
            return GatedResult(y, p, self.mlp_gate_bias, self.post_mlp_layernorm)
        gate = self.mlp_gate(h)
        if self.mlp.rows_apply() and self.mlp.shared_expert is None:
            y, row_of, share, _ = self.mlp.rows(h, self._forced(batch))
            return GatedResult(y, gate, self.mlp_gate_bias, self.post_mlp_layernorm, row_of, share)
        return GatedResult(self.mlp(h, self._forced(batch)), gate, self.mlp_gate_bias, self.post_mlp_layernorm)

    def advance(self, st: Stream, batch) -> Stream:
        y, p = self.mix(st, batch)
        st.gated = GatedResult(y, p, self.mixer_gate_bias, self.post_mixer_layernorm)
        if self.mlp is not None:
            st.gated = self.feed_forward(st.enter(self.pre_mlp_layernorm), batch)
        return st
