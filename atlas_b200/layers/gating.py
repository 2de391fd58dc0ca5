"""Sigmoid gate on a sublayer's result, computed from what the sublayer reads: ``y * sigmoid(W h + b)``.

The product is this block's; the sigmoid and the multiplication are part of the residual kernel (``ops.NormDelta.gate``).
"""
from __future__ import annotations

from typing import Optional

import torch

from .. import ops
from ..ops import Act, LinearWeight
from .common import make_weight, randn_weight


class SublayerGate:
    def __init__(self, width: int, quant_kind: str):
        self.width, self.quant_kind = width, quant_kind
        self.w: Optional[LinearWeight] = None

    def load(self, w: torch.Tensor, bias: torch.Tensor) -> None:
        self.w = make_weight(w, self.quant_kind, bias.to(w.dtype).contiguous())

    def init_random(self, gen, std, dtype, device) -> None:
        self.load(randn_weight(gen, self.width, self.width, std, dtype, device), randn_weight(gen, 1, self.width, std, dtype, device)[0])

    def forward(self, act: Act) -> torch.Tensor:
        """The gate's argument ``[T, width]``."""
        return ops.linear(act, self.w)
