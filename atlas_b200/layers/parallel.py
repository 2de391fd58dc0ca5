"""Attention and a Mamba-2 mixer side by side on the same input.

Each output is RMS-normed over the model width with its own weight and the result is half their sum.  The two norms and the
sum happen where the result joins the residual streams (``ops.hyper_norm``), so the mixer hands both outputs over as they
leave their output projections.
"""
from __future__ import annotations

from typing import List, Optional, Tuple

import torch

from ..config import ModelConfig
from ..ops import Act
from .attention import Attention
from .common import ParallelCtx
from .mamba2 import Mamba2Mixer


class ParallelMixer:
    def __init__(self, cfg: ModelConfig, layer_idx: int, pctx: ParallelCtx, quant_kind: str):
        self.pctx = pctx
        self.left = Attention(cfg, layer_idx, pctx, quant_kind)
        self.right = Mamba2Mixer(cfg, layer_idx, pctx, quant_kind)
        self.hidden = cfg.hidden_size
        self.left_norm: Optional[torch.Tensor] = None         # [hidden] fp32
        self.right_norm: Optional[torch.Tensor] = None

    def init_random(self, gen, std, dtype, device) -> None:
        self.left.init_random(gen, std, dtype, device)
        self.right.init_random(gen, std, dtype, device)
        self.left_norm = torch.ones(self.hidden, dtype=torch.float32, device=device)
        self.right_norm = torch.ones(self.hidden, dtype=torch.float32, device=device)

    def alloc_state(self, num_slots: int, device, act_dtype) -> dict:
        return self.right.alloc_state(num_slots, device, act_dtype)

    def forward(self, act: Act, batch, kv, rope_cache: torch.Tensor, state: dict) -> Tuple[torch.Tensor, torch.Tensor]:
        return self.left.forward(act, batch, kv, rope_cache), self.right.forward(act, batch, state)

    def commit(self, num_accepted_rows: List[int], state: dict) -> None:
        self.right.commit(num_accepted_rows, state)
