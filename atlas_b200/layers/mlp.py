"""SwiGLU feed-forward: fused gate|up GEMM -> SiLU*mul (+FP8 quant) -> row-parallel down GEMM.

Under tensor parallelism gate/up are column-parallel and down is row-parallel with its reduction
fused into the GEMM epilogue.  (The reference replicates dense FFN weights across TP ranks,
``crates/spark-model/src/layers/dense_ffn*``; sharding them is this engine's choice.)
"""
from __future__ import annotations

from typing import Optional

import torch

from .. import ops
from ..config import ModelConfig
from ..ops import Act, LinearWeight
from ..lora import add_delta
from .common import ParallelCtx, make_weight, paired_rows, randn_weight, shard_cols, shard_rows


class DenseMLP:
    def __init__(self, cfg: ModelConfig, pctx: ParallelCtx, quant_kind: str, intermediate: Optional[int] = None,
                 shard: bool = True, activation: Optional[str] = None, glu_limit: Optional[float] = None, paired: bool = False):
        """``paired``: gate and up rows alternate, so that the product's epilogue applies the gated unit (silu or clamped)."""
        self.cfg, self.pctx, self.quant_kind = cfg, pctx, quant_kind
        self.paired = paired
        # "silu_glu": gate|up GEMM -> silu(gate) * up; "relu2": a single up GEMM -> relu(up)^2 (Nemotron-H), with biases where the
        # configuration has them
        self.activation = activation or getattr(cfg, "mlp_activation", "silu_glu")
        limit = cfg.glu_limit if glu_limit is None else glu_limit
        self.unit = (limit, cfg.glu_alpha, 1.0) if self.activation == "clamped_glu" else ops.SILU_UNIT
        assert not paired or self.activation in ("clamped_glu", "silu_glu")
        self.inter = intermediate or cfg.intermediate_size
        self.shard = shard and pctx.tp_size > 1 and self.inter % (pctx.tp_size * 128) == 0
        self.gate_up: Optional[LinearWeight] = None
        self.down: Optional[LinearWeight] = None
        self.down_bias: Optional[torch.Tensor] = None       # of a sharded down projection: joins the group's sum
        self.lora = None                    # lora.LoraSet shared by the model's layers
        self.lora_prefix = ""               # e.g. "layers.3.mlp."

    def load(self, gate: Optional[torch.Tensor], up: torch.Tensor, down: torch.Tensor, up_bias: Optional[torch.Tensor] = None,
             down_bias: Optional[torch.Tensor] = None) -> None:
        tp, r = (self.pctx.tp_size, self.pctx.tp_rank) if self.shard else (1, 0)
        if up_bias is not None:
            assert self.activation == "relu2", "gated units have no biases"
            up_bias = shard_rows(up_bias.to(up.dtype).reshape(-1, 1), r, tp)[:, 0].contiguous()
            down_bias = down_bias.to(down.dtype).contiguous()
        if self.activation == "relu2":
            gu = shard_rows(up, r, tp)
        elif self.paired:
            gu = paired_rows(shard_rows(gate, r, tp), shard_rows(up, r, tp)).contiguous()
        else:
            gu = torch.cat([shard_rows(gate, r, tp), shard_rows(up, r, tp)], 0)
        self.gate_up = make_weight(gu, self.quant_kind, up_bias)
        self.down_bias = down_bias if self.shard else None
        self.down = make_weight(shard_cols(down, r, tp).contiguous(), self.quant_kind, None if self.shard else down_bias)

    def init_random(self, gen, std, dtype, device) -> None:
        h = self.cfg.hidden_size
        gate, up = (randn_weight(gen, self.inter, h, std, dtype, device) for _ in range(2))
        down = randn_weight(gen, h, self.inter, std, dtype, device)
        biases = [randn_weight(gen, 1, n, std, dtype, device)[0] for n in (self.inter, h)] if self.cfg.mlp_bias else []
        self.load(gate, up, down, *biases)

    def hidden_act(self, act: Act) -> Act:
        """gate|up GEMM + SiLU * mul: the input of the down projection (no adapters)."""
        if self.paired:
            return ops.linear_gated_unit(act, self.gate_up, self.unit)
        if self.activation in ("gelu_tanh_glu", "clamped_glu"):
            return self._glu(ops.linear(act, self.gate_up), self.down.kind == "fp8_block")
        if self.down.kind == "fp8_block" and ops.swiglu_fusable(act, self.gate_up):
            return ops.linear_swiglu(act, self.gate_up)
        return ops.silu_mul_act(ops.linear(act, self.gate_up), want_fp8=self.down.kind == "fp8_block")

    def _glu(self, gate_up: torch.Tensor, want_fp8: bool) -> Act:
        if self.paired or self.activation == "clamped_glu":
            return ops.gated_unit_act(gate_up, self.unit, self.paired)
        return ops.glu_act(gate_up, want_fp8, "gelu_tanh")

    def _relu2(self, act: Act, reduce: bool) -> torch.Tensor:
        return self.down_product(ops.linear_relu2(act, self.gate_up), reduce)

    def down_product(self, a: torch.Tensor, reduce: bool = True) -> torch.Tensor:
        """Down projection of the hidden activations, summed over the group that shards it."""
        y = self.pctx.row_parallel_linear(a, self.down) if (self.shard and reduce) else ops.linear(a, self.down)
        return y if self.down_bias is None else y + self.down_bias

    def forward(self, act: Act, reduce: bool = True, batch=None) -> torch.Tensor:
        if self.activation == "relu2":
            return self._relu2(act, reduce)
        use_lora = self.lora is not None and batch is not None and batch.adapter_rows is not None and self.lora_prefix
        if (self.paired or self.activation in ("gelu_tanh_glu", "clamped_glu")) and not use_lora:
            a = self.hidden_act(act)
            return self.pctx.row_parallel_linear(a, self.down) if (self.shard and reduce) else ops.linear(a, self.down)
        if not use_lora and self.down.kind == "fp8_block" and ops.swiglu_fusable(act, self.gate_up):
            a = ops.linear_swiglu(act, self.gate_up)
            return self.pctx.row_parallel_linear(a, self.down) if (self.shard and reduce) else ops.linear(a, self.down)
        gu = ops.linear(act, self.gate_up)
        if use_lora:
            xin, half = act.plain(), gu.shape[1] // 2
            if self.paired:
                parts = torch.stack([gu[:, 0::2], gu[:, 1::2]]).contiguous()
                add_delta(parts[0], self.lora, self.lora_prefix + "gate_proj", xin, batch, 0, half)
                add_delta(parts[1], self.lora, self.lora_prefix + "up_proj", xin, batch, 0, half)
                gu = torch.stack([parts[0], parts[1]], -1).flatten(1)
            else:
                add_delta(gu, self.lora, self.lora_prefix + "gate_proj", xin, batch, 0, half)
                add_delta(gu, self.lora, self.lora_prefix + "up_proj", xin, batch, half, half)
        if self.paired or self.activation in ("gelu_tanh_glu", "clamped_glu"):
            a = self._glu(gu, False)
        else:
            a = ops.silu_mul_act(gu, want_fp8=self.down.kind == "fp8_block" and not use_lora)
        if use_lora:
            # with a sharded FFN this rank's columns of A give a partial delta: add it before the group reduction
            y = ops.linear(a, self.down)
            add_delta(y, self.lora, self.lora_prefix + "down_proj", a.plain(), batch)
            return self.pctx.all_reduce(y) if (self.shard and reduce) else y
        if self.shard and reduce:
            return self.pctx.row_parallel_linear(a, self.down)
        return ops.linear(a, self.down)
