"""Decoder layers with a norm in front of each sub-layer and a 32-bit residual stream.

One layer of a stack whose layers are listed one by one (``DecoderConfig.layer_specs``; Nilepel checkpoints):

    x ← x + mixer(norm(x))                 grouped attention (window, chunk) or latent attention
    x ← x + feed_forward(norm(x))          gated block, experts beside a shared one, or absent

The sum is left pending and carried out by the kernel that forms the next norm (``Stream.enter``), which also combines a token's expert
rows and scales the shared expert's.
"""
from __future__ import annotations

import torch

from .config import DecoderConfig
from .mixer_layer import GatedFeedForward, MixerLayer
from .parallel_layer import PlainResult, Stream


class PreNormLayer(MixerLayer):

    def __init__(self, cfg: DecoderConfig, layer_idx: int):
        super().__init__(cfg, layer_idx)
        f, self.mlp = self.spec.mlp, None
        if f is None:
            return
        self.pre_mlp_layernorm = self.norm(cfg)
        self.mlp = self.experts(cfg) if self.is_moe else GatedFeedForward(cfg.hidden_size, f.ff, limit=f.limit, act=f.act)

    def feed_forward(self, h: torch.Tensor, batch) -> PlainResult:
        if not self.is_moe:
            return PlainResult(self.mlp(h)[0])
        if not self.mlp.rows_apply():
            return PlainResult(self.mlp(h, self._forced(batch)))
        y, row_of, share, open_ = self.mlp.rows(h, self._forced(batch))
        beside = self.mlp.shared_expert.serve(h) if open_ is not None else None
        return PlainResult(y, row_of, share, beside, open_)

    def advance(self, st: Stream, batch) -> Stream:
        st.plain = PlainResult(self.mix(st, batch)[0])
        if self.mlp is not None:
            st.plain = self.feed_forward(st.enter(self.pre_mlp_layernorm), batch)
        return st
