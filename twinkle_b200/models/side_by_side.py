"""Two mixers on the same input, attention and a matrix memory: one input product for both, and half the sum of their normed results.
"""
from __future__ import annotations

from typing import Any, Dict

import torch
import torch.nn as nn

from .config import SideBySideSpec
from .grouped_attention import GroupedAttention
from .layers import Linear, RMSNorm
from .parallel_layer import NormedResult
from .recurrent import MatrixMemory


class SideBySide(nn.Module):
    """``lead`` and ``table``: see ``GroupedAttention``."""

    def __init__(self, width: int, spec: SideBySideSpec, eps: float, layer_idx: int, lead=(), table=None):
        super().__init__()
        self.spec = spec
        parts, at = list(lead) + spec.in_parts(), sum(n for _, n in lead)
        self.in_proj = Linear(width, sum(n for _, n in parts), parts=parts)
        self.left = GroupedAttention(width, spec.left, eps, layer_idx, table=table, first=at)
        self.right = MatrixMemory(width, spec.right, eps, layer_idx, first=at + sum(n for _, n in spec.left.in_parts()))
        self.left_norm, self.right_norm = RMSNorm(width, eps), RMSNorm(width, eps)

    def pending(self, y, norm: RMSNorm) -> NormedResult:
        """Both results on their way into the stream, whose kernel norms and adds them."""
        return NormedResult(y[0], norm, self.left.o_bias, self.left_norm, y[1], self.right_norm)

    def forward(self, h: torch.Tensor, batch, held: Dict[int, Any]):
        """``((result of the left, without its bias, result of the right), the input product)``."""
        p = self.in_proj(h)
        return (self.left.attend(p, batch, held), self.right.remember(p, batch)), p
