"""Decoder layers that run a mixer and a feed-forward block one after the other on a 32-bit residual stream: what the kinds of such
layers (``sandwich_layer.py``, ``prenorm_layer.py``) have in common.

A sub-layer's result is left pending and carried out by the kernel that forms the next norm (``Stream.enter``): without gradients the
stream is passed over once per sub-layer.  With gradients the stream is one tensor ``[x | what later layers borrow]`` per layer boundary,
which is what activation recompute keeps.
"""
from __future__ import annotations

import torch
import torch.nn as nn

from .. import ops
from .config import DecoderConfig
from .grouped_attention import GroupedAttention
from .latent_attention import LatentAttention
from .layers import Linear, RMSNorm
from .linear_attention import HGRN2
from .parallel_layer import Stream
from .recurrent import Mamba1
from .side_by_side import SideBySide

MIXERS = {'latent_attention': LatentAttention, 'attention': GroupedAttention, 'hgrn2': HGRN2, 'mamba1': Mamba1, 'parallel': SideBySide}


class GatedFeedForward(nn.Module):
    """``W_down act(W_gate h, W_up h)`` with other projections of ``h`` (``lead``) in front of gate and up in one product; ``limit`` and ``act``:
    see ``config.FeedForwardSpec``."""

    def __init__(self, width: int, ff: int, lead=(), limit: float = 0.0, act: str = 'silu'):
        super().__init__()
        self.ff, self.first, self.limit, self.act = ff, sum(n for _, n in lead), limit, act
        self.in_proj = Linear(width, self.first + 2 * ff, parts=list(lead) + [('gate_proj', ff), ('up_proj', ff)])
        self.down_proj = Linear(ff, width, name='down_proj')

    def forward(self, h: torch.Tensor):
        p = self.in_proj(h)
        return self.down_proj(ops.glu_columns(p, self.first, self.first + self.ff, self.ff, self.limit, self.act)), p


class MixerLayer(nn.Module):
    is_linear = False
    pre_norm = True         # whether sub-layers read a norm of the stream (or the stream itself)

    def __init__(self, cfg: DecoderConfig, layer_idx: int, lead=()):
        super().__init__()
        sp = self.spec = cfg.layer_specs[layer_idx]
        self.layer_idx, self.width, self.eps = layer_idx, cfg.hidden_size, cfg.rms_norm_eps
        self.is_moe = sp.is_moe
        self.moe_index = sum(s.is_moe for s in cfg.layer_specs[:layer_idx])      # place in recorded routing lists
        self.columns, at = {}, cfg.hidden_size                                   # what is lent, in the layer-boundary tensor
        for j, n in cfg.held_columns():
            self.columns[j] = (at, at + n, cfg.layer_specs[j].mixer)
            at += n
        self.input_layernorm = self.norm(cfg) if self.pre_norm else None
        self.mixer = MIXERS[sp.mixer.kind](cfg.hidden_size, sp.mixer, cfg.rms_norm_eps, layer_idx, lead, cfg.rotary_columns(layer_idx))

    @staticmethod
    def norm(cfg: DecoderConfig) -> RMSNorm:
        return RMSNorm(cfg.hidden_size, cfg.rms_norm_eps, cfg.rms_norm_offset)

    def experts(self, cfg: DecoderConfig) -> nn.Module:
        from .decoder import MoEBlock
        f = self.spec.mlp
        return MoEBlock(DecoderConfig(hidden_size=cfg.hidden_size, num_experts=f.experts, num_experts_per_tok=f.top, moe_intermediate_size=f.ff,
                                      router_scoring=f.scoring, router_linear_bias=f.scoring == 'topk_softmax', expert_act='swiglu' if f.gated else 'relu2',
                                      n_group=f.groups, topk_group=f.keep, routed_scaling_factor=f.scale, norm_topk_prob=False,
                                      shared_expert_intermediate_size=f.shared), self.layer_idx)

    def _forced(self, batch):
        return batch.routed_experts[self.moe_index] if batch.routed_experts is not None else None

    def mix(self, st: Stream, batch):
        """The mixer on the stream's norm (or the stream): ``(result, the input product)``.  What it keeps stays in ``st.held`` if a later
        layer borrows it."""
        out = self.mixer(st.enter(self.input_layernorm, self.dtype), batch, st.held)
        if self.layer_idx not in self.columns:
            st.held.pop(self.layer_idx, None)
        return out

    @property
    def dtype(self) -> torch.dtype:
        """The compute dtype."""
        return self.mixer.in_proj.weight.dtype

    def advance(self, st: Stream, batch) -> Stream:
        """One layer; the result of its last sub-layer stays pending in the stream."""
        raise NotImplementedError

    def forward(self, x: torch.Tensor, cos, sin, batch, kv_sink=None) -> torch.Tensor:
        """``x [T, width + lent columns]`` fp32 → the same after this layer."""
        dt = self.dtype
        held = {j: MIXERS[m.kind].from_columns(m, x[:, a:b].to(dt)) for j, (a, b, m) in self.columns.items()}
        st = self.advance(Stream(x[:, :self.width].clone(), held=held), batch)
        st.enter(self.input_layernorm, dt)      # the sum; the norm formed with it is the next layer's business
        lent = [x[:, a:b] if j != self.layer_idx else MIXERS[m.kind].to_columns(m, st.held[j]).float() for j, (a, b, m) in self.columns.items()]
        return torch.cat([st.x] + lent, -1)
