"""Decoder layers whose sub-layers read the 32-bit residual stream as it is, with a norm on each sub-layer's result.

One layer of a stack whose layers are listed one by one (``DecoderConfig.layer_specs``; Puzonex checkpoints):

    x ← x + norm(mixer(x))                 attention, a selective scan, or attention beside a matrix memory
    x ← x + norm(feed_forward(x))          gated block, or absent

Norm and sum are left pending and carried out by the kernel that forms the next sub-layer's input (``Stream.enter``), which also combines the
results of two mixers side by side.
"""
from __future__ import annotations

from .config import DecoderConfig
from .mixer_layer import GatedFeedForward, MixerLayer
from .parallel_layer import NormedResult, Stream


class PostNormLayer(MixerLayer):
    pre_norm = False

    def __init__(self, cfg: DecoderConfig, layer_idx: int):
        super().__init__(cfg, layer_idx)
        f, self.mlp = self.spec.mlp, None
        if self.is_moe:
            raise NotImplementedError('experts in layers without norms in front of their sub-layers')
        self.post_mixer_layernorm = self.norm(cfg)
        if f is not None:
            self.post_mlp_layernorm = self.norm(cfg)
            self.mlp = GatedFeedForward(cfg.hidden_size, f.ff, limit=f.limit, act=f.act)

    def advance(self, st: Stream, batch) -> Stream:
        y, _ = self.mix(st, batch)
        pending = getattr(self.mixer, 'pending', None)
        st.normed = pending(y, self.post_mixer_layernorm) if pending is not None else NormedResult(y, self.post_mixer_layernorm)
        if self.mlp is not None:
            st.normed = NormedResult(self.mlp(st.enter(None, self.dtype))[0], self.post_mlp_layernorm)
        return st
