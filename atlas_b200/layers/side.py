"""A second token embedding that every layer takes its own share of.

``table [vocab, layers * dim]`` belongs to the model; layer ``i`` reads ``e = table[token, i * dim : (i + 1) * dim]`` and adds
``rms(proj(gelu_tanh(gate(x)) * e)) * norm`` to the stream ``x`` that its gate reads.  The norm is part of the residual kernel
(``ops.NormDelta``).  ``dim`` is zero-padded to whole operand rows of the products.
"""
from __future__ import annotations

from typing import Optional

import torch
import torch.nn.functional as F

from .. import ops
from ..ops import Act, LinearWeight
from .common import make_weight, randn_weight

SIDE_ALIGN = 8


class TokenSide:
    def __init__(self, width: int, dim: int, number: int, quant_kind: str):
        self.width, self.dim, self.number, self.quant_kind = width, dim, number, quant_kind
        self.table: Optional[torch.Tensor] = None             # the model's [vocab, layers * dim]
        self.gate: Optional[LinearWeight] = None
        self.proj: Optional[LinearWeight] = None
        self.norm: Optional[torch.Tensor] = None              # fp32 [width]

    def load(self, gate: torch.Tensor, proj: torch.Tensor, norm: torch.Tensor) -> None:
        pad = -self.dim % SIDE_ALIGN
        self.gate = make_weight(F.pad(gate, (0, 0, 0, pad)).contiguous(), self.quant_kind)
        self.proj = make_weight(F.pad(proj, (0, pad)).contiguous(), self.quant_kind)
        self.norm = norm

    def init_random(self, gen, std, dtype, device) -> None:
        self.load(randn_weight(gen, self.dim, self.width, std, dtype, device), randn_weight(gen, self.width, self.dim, std, dtype, device),
                  torch.ones(self.width, dtype=torch.float32, device=device))

    def forward(self, act: Act, token_ids: torch.Tensor) -> torch.Tensor:
        """What joins the stream after its norm ``[T, width]``."""
        return ops.linear(ops.gelu_embedding(ops.linear(act, self.gate), self.table, token_ids, self.number * self.dim, self.dim), self.proj)
