"""Generic decoder-only LM assembled from the layer blocks.

One class covers the dense (Llama/Mistral/Qwen2/Qwen3), MoE (Qwen3-MoE) and hybrid
(Qwen3-Next: Gated DeltaNet + gated attention + MoE + MTP head; models given by a list of layers) families;
``ModelConfig`` decides the mixer and FFN kind of every layer and the form of the residual.

Reference parity: ``crates/spark-model/src/model/`` (``TransformerModel``), the decode program in
``model/trait_impl/decode_a2.rs`` and the chunked prefill program in ``model/trait_impl/prefill_b.rs``.
"""
from __future__ import annotations

import copy
import os
from dataclasses import dataclass, field
from typing import Dict, List, Optional, Tuple

import torch

from .. import ops
from ..config import ModelConfig
from ..layers import (MIXERS, Attention, DenseMLP, GatedDeltaNet, HyperConnection, InputConvolution, Mamba2Mixer, MLAttention, MoE,
                      ParallelCtx, SublayerGate, TokenSide)
from ..layers.common import make_weight, randn_weight, shard_rows
from ..ops import Act, DepthSum, LinearWeight, NormDelta, StreamDelta, reference as ref
from .batch import ForwardBatch

# tensor-parallel steps with at least this many rows run sequence-parallel (reduce-scatter / all-gather fused into the
# GEMMs); smaller steps keep the replicated residual stream and the fused GEMM + all-reduce
SEQ_PARALLEL_MIN_TOKENS = int(os.environ.get("ATLAS_SP_MIN_TOKENS", "1024"))
# smallest tensor-parallel group whose pure decode steps take the sequence-parallel path (0 = never)
SEQ_PARALLEL_DECODE_MIN_WORLD = int(os.environ.get("ATLAS_SP_DECODE_MIN_WORLD", "0"))

_DTYPES = {"float32": torch.float32, "bfloat16": torch.bfloat16, "float16": torch.float16,
           "torch.float32": torch.float32, "torch.bfloat16": torch.bfloat16, "torch.float16": torch.float16}


def kv_dtype_is_fp8(dtype) -> bool:
    return dtype == torch.float8_e4m3fn


KV_NVFP4 = torch.uint8          # cache dtype marker of the NVFP4 KV cache (packed e2m1 + e4m3 scales, GPU only)


def kv_dtype_is_quantised(dtype) -> bool:
    return dtype == torch.float8_e4m3fn or dtype == KV_NVFP4


def kv_element_bytes(dtype) -> float:
    """Bytes per cached element (NVFP4: half a byte of data plus one scale byte per 16 elements)."""
    return 9.0 / 16.0 if dtype == KV_NVFP4 else float(dtype.itemsize)


def alloc_kv(num_blocks: int, block_size: int, hkv: int, d: int, dtype, device):
    """Paged K and V pools as logical ``[num_blocks, block_size, Hkv, D]`` tensors (the GPU pools are views
    of the kernels' physical layout)."""
    if torch.device(device).type == "cuda" and (kv_dtype_is_quantised(dtype) or dtype in (torch.bfloat16, torch.float32)):
        return ops.cuda_ops().alloc_kv_cache(num_blocks, block_size, hkv, d, dtype, device)
    if dtype == KV_NVFP4:
        raise ValueError("the NVFP4 KV cache exists on the GPU kernels only")
    shape = (num_blocks, block_size, hkv, d)
    return torch.zeros(shape, dtype=dtype, device=device), torch.zeros(shape, dtype=dtype, device=device)


def torch_dtype(name: str) -> torch.dtype:
    return _DTYPES.get(str(name), torch.bfloat16)


def quant_kinds(cfg: ModelConfig) -> Tuple[str, str]:
    """(kind for dense projections, kind for MoE expert stacks)."""
    m = cfg.quant.method
    if m == "fp8_block":
        return "fp8_block", "fp8_block"
    if m == "nvfp4":
        return ("dense" if cfg.quant.experts_only else "nvfp4"), "nvfp4"
    return "dense", "dense"


@dataclass
class CacheStore:
    """Device memory the model reads/writes across steps: paged KV per attention layer and the
    recurrent-state slot pool per GDN layer."""
    kv: Dict[int, Tuple[torch.Tensor, torch.Tensor]] = field(default_factory=dict)
    kv_scales: Dict[int, Tuple[float, float]] = field(default_factory=dict)
    states: Dict[int, dict] = field(default_factory=dict)
    block_size: int = 16
    num_blocks: int = 0

    def layer_kv(self, i: int):
        k, v = self.kv[i]
        ks, vs = self.kv_scales.get(i, (1.0, 1.0))
        return k, v, ks, vs


class DecoderLayer:
    def __init__(self, cfg: ModelConfig, idx: int, pctx: ParallelCtx, ep_mode: str = "auto",
                 force_attention: bool = False):
        self.cfg, self.idx = cfg, idx
        dense_kind, expert_kind = quant_kinds(cfg)
        self.kind = "attention" if force_attention else cfg.layer_kind(idx)
        attn_cls = MLAttention if cfg.kv_lora_rank > 0 else Attention
        self.mixer = attn_cls(cfg, idx, pctx, dense_kind) if self.kind == "attention" else GatedDeltaNet(cfg, idx, pctx, dense_kind)
        self.is_moe = (cfg.num_experts > 0) if force_attention else cfg.is_moe_layer(idx)
        self.ffn = MoE(cfg, pctx, expert_kind, dense_kind, ep_mode) if self.is_moe else DenseMLP(cfg, pctx, dense_kind)
        self.input_norm: Optional[torch.Tensor] = None
        self.post_norm: Optional[torch.Tensor] = None
        # sandwich norms (Gemma): post_norm normalises the mixer's OUTPUT, pre_ffn_norm the FFN's input, post_ffn_norm
        # the FFN's output; without them post_norm is the FFN's input norm
        self.pre_ffn_norm: Optional[torch.Tensor] = None
        self.post_ffn_norm: Optional[torch.Tensor] = None
        self.rope_override: Optional[torch.Tensor] = None     # rotary table of sliding-window layers with their own base

    def init_random(self, gen, std, dtype, device):
        base = 0.0 if self.cfg.norm_plus_one else 1.0
        self.input_norm = torch.full((self.cfg.hidden_size,), base, dtype=dtype, device=device)
        self.post_norm = torch.full((self.cfg.hidden_size,), base, dtype=dtype, device=device)
        if self.cfg.sandwich_norms:
            self.pre_ffn_norm = torch.full((self.cfg.hidden_size,), base, dtype=dtype, device=device)
            self.post_ffn_norm = torch.full((self.cfg.hidden_size,), base, dtype=dtype, device=device)
        self.mixer.init_random(gen, std, dtype, device)
        self.ffn.init_random(gen, std, dtype, device)

    def _mixer_fp8(self) -> bool:
        w = self.mixer.qkv if self.kind == "attention" else self.mixer.in_proj
        return w.kind == "fp8_block"

    def _ffn_fp8(self) -> bool:
        return (not self.is_moe) and self.ffn.gate_up.kind == "fp8_block"

    def accepts_prenormed(self) -> bool:
        """This layer's input norm may be applied by the previous layer's down projection (deferred 1/rms factor): its
        only consumer of the normalised input is an FP8 linear layer."""
        return (self.kind == "attention" and isinstance(self.mixer, Attention) and self.mixer.qkv.kind == "fp8_block"
                and self.mixer.lora is None and not self.cfg.sandwich_norms)

    def forward(self, x, residual: Optional[torch.Tensor], batch: ForwardBatch, cache: CacheStore,
                rope_cache: torch.Tensor, next_norm: Optional[torch.Tensor] = None):
        """``x`` is the previous layer's output (to be added to ``residual`` and normalised here) or, when that layer
        already did both in its down projection's epilogue, the normalised activations as an ``Act``.  With
        ``next_norm`` (the next layer's input norm weight) this layer may do the same for its successor and return an
        ``Act`` in place of the plain output."""
        cfg = self.cfg
        eps, p1 = cfg.rms_norm_eps, cfg.norm_plus_one
        if self.rope_override is not None:
            rope_cache = self.rope_override
        if isinstance(x, Act):
            act = x
        elif residual is None:
            act, _ = ops.rmsnorm_act(x, self.input_norm, eps, None, p1, self._mixer_fp8())
            residual = x
        else:
            act, residual = ops.rmsnorm_act(x, self.input_norm, eps, residual, p1, self._mixer_fp8())
        if cfg.sandwich_norms:
            h = self.mixer.forward(act, batch, cache.layer_kv(self.idx), rope_cache)
            h, _ = ops.rmsnorm(h, self.post_norm, eps, None, p1)
            act, residual = ops.rmsnorm_act(h, self.pre_ffn_norm, eps, residual, p1, self._ffn_fp8())
            h = self.ffn.forward(act, batch=batch)
            h, _ = ops.rmsnorm(h, self.post_ffn_norm, eps, None, p1)
            return h, residual
        single = self.mixer.pctx.tp_size == 1
        no_lora = batch.adapter_rows is None
        dense_fp8_ffn = self._ffn_fp8() and self.ffn.down.kind == "fp8_block"
        if (self.kind == "attention" and single and no_lora and dense_fp8_ffn
                and ops.residual_norm_fusable(residual, self.mixer.o)):
            # o_proj + residual add + post-attention norm + FP8 quantisation in the projection's epilogue
            out = self.mixer.mix(act, batch, cache.layer_kv(self.idx), rope_cache)
            act, residual = ops.linear_residual_norm(out, self.mixer.o, residual, self.post_norm, eps, p1)
        else:
            fused = None
            tp_fusable = (not single and no_lora and dense_fp8_ffn and isinstance(self.mixer, Attention)
                          and getattr(self.ffn, "shard", False))
            if self.kind == "attention" and tp_fusable:
                # tensor parallel: o_proj + all-reduce + residual add + norm + FP8 quantisation in one kernel (decode-size
                # outputs; larger ones return None before anything is launched)
                out = self.mixer.mix(act, batch, cache.layer_kv(self.idx), rope_cache)
                fused = self.mixer.pctx.row_parallel_residual_norm(out, self.mixer.o, residual, self.post_norm, eps, p1)
                if fused is None:
                    h = self.mixer.pctx.row_parallel_linear(out, self.mixer.o)
            elif self.kind == "attention":
                h = self.mixer.forward(act, batch, cache.layer_kv(self.idx), rope_cache)
            else:
                h = self.mixer.forward(act, batch, cache.states[self.idx])
            if fused is not None:
                act, residual = fused
            else:
                act, residual = ops.rmsnorm_act(h, self.post_norm, eps, residual, p1, self._ffn_fp8())
        if (next_norm is not None and single and no_lora and dense_fp8_ffn
                and ops.residual_norm_fusable(residual, self.ffn.down)):
            # down_proj + residual add + the NEXT layer's input norm + FP8 quantisation in one epilogue
            return ops.linear_residual_norm(self.ffn.hidden_act(act), self.ffn.down, residual, next_norm, eps, p1)
        if (next_norm is not None and not single and no_lora and dense_fp8_ffn and getattr(self.ffn, "shard", False)
                and self.ffn.activation != "relu2" and ops.residual_norm_fusable(residual, self.ffn.down)):
            a = self.ffn.hidden_act(act)
            fused = self.ffn.pctx.row_parallel_residual_norm(a, self.ffn.down, residual, next_norm, eps, p1)
            if fused is not None:
                return fused
            return self.ffn.pctx.row_parallel_linear(a, self.ffn.down), residual
        if self.is_moe:
            hashed = self.ffn.hash_table is not None and batch.input_ids is not None
            h = self.ffn.forward(act, batch.input_ids.to(torch.int32) if hashed else None, batch=batch)
        else:
            h = self.ffn.forward(act, batch=batch)
        return h, residual


class SingleBlock:
    """A pre-norm residual block around ONE module (Nemotron-H): a Mamba-2 mixer, a position-free attention layer or a
    two-projection relu^2 MLP.  Same ``forward`` protocol as :class:`DecoderLayer`: the block's output is added to the
    residual stream by the next block's norm kernel."""

    def __init__(self, cfg: ModelConfig, idx: int, pctx: ParallelCtx):
        self.cfg, self.idx = cfg, idx
        dense_kind, _ = quant_kinds(cfg)
        self.block = cfg.block_types[idx]
        self.kind = cfg.layer_kind(idx)
        self.is_moe = False
        self.mixer = self.ffn = None
        if self.kind == "mamba2":
            self.mixer = Mamba2Mixer(cfg, idx, pctx, dense_kind)
        elif self.kind == "attention":
            self.mixer = Attention(cfg, idx, pctx, dense_kind)
        elif self.block == "mlp":
            self.ffn = DenseMLP(cfg, pctx, dense_kind, activation="relu2")
        else:
            raise ValueError(f"unsupported block type '{self.block}'")
        self.input_norm: Optional[torch.Tensor] = None
        self.post_norm = None

    def init_random(self, gen, std, dtype, device):
        self.input_norm = torch.ones(self.cfg.hidden_size, dtype=dtype, device=device)
        (self.mixer or self.ffn).init_random(gen, std, dtype, device)

    def accepts_prenormed(self) -> bool:
        return False

    def _fp8_in(self) -> bool:
        w = self.mixer.in_proj if self.kind == "mamba2" else (self.mixer.qkv if self.kind == "attention" else self.ffn.gate_up)
        return w.kind == "fp8_block"

    def forward(self, x, residual, batch: ForwardBatch, cache: CacheStore, rope_cache, next_norm=None):
        cfg = self.cfg
        if residual is None:
            act, _ = ops.rmsnorm_act(x, self.input_norm, cfg.rms_norm_eps, None, cfg.norm_plus_one, self._fp8_in())
            residual = x
        else:
            act, residual = ops.rmsnorm_act(x, self.input_norm, cfg.rms_norm_eps, residual, cfg.norm_plus_one, self._fp8_in())
        if self.kind == "mamba2":
            h = self.mixer.forward(act, batch, cache.states[self.idx])
        elif self.kind == "attention":
            h = self.mixer.forward(act, batch, cache.layer_kv(self.idx), rope_cache)
        else:
            h = self.ffn.forward(act, batch=batch)
        return h, residual


class StreamLayer:
    """A layer on hyper-connected residual streams (``layers/hyper.py``): a mixer of any kind and, where the model's layer
    list says so, a feed-forward sublayer.  Same ``forward`` protocol as :class:`DecoderLayer`, with the pending
    :class:`StreamDelta` in place of the previous layer's output and the streams in place of the residual."""

    def __init__(self, cfg: ModelConfig, idx: int, pctx: ParallelCtx):
        spec = cfg.layer_specs[idx]
        self.cfg, self.idx = cfg.for_layer(idx), idx
        dense_kind, _ = quant_kinds(cfg)
        self.kind, self.is_moe = spec.kind, False
        self.mixer = MIXERS[spec.kind](self.cfg, idx, pctx, dense_kind)
        self.ffn = DenseMLP(self.cfg, pctx, dense_kind) if spec.has_mlp else None
        self.conn1 = HyperConnection(cfg.residual_streams)
        self.conn2 = HyperConnection(cfg.residual_streams) if spec.has_mlp else None
        self.input_norm: Optional[torch.Tensor] = None         # fp32
        self.post_norm: Optional[torch.Tensor] = None
        self.rope_override: Optional[torch.Tensor] = None      # this layer's own rotary table

    def init_random(self, gen, std, dtype, device):
        ones = lambda: torch.ones(self.cfg.hidden_size, dtype=torch.float32, device=device)
        self.mixer.init_random(gen, std, dtype, device)
        self.conn1.init_random(gen, device)
        self.input_norm = ones()
        if self.ffn is not None:
            self.ffn.init_random(gen, std, dtype, device)
            self.conn2.init_random(gen, device)
            self.post_norm = ones()

    def accepts_prenormed(self) -> bool:
        return False

    def forward(self, x: StreamDelta, streams: Optional[torch.Tensor], batch: ForwardBatch, cache: CacheStore, rope_cache,
                next_norm=None):
        eps = self.cfg.rms_norm_eps
        rope_cache = rope_cache if self.rope_override is None else self.rope_override
        h, streams = ops.hyper_norm(streams, x, self.conn1.read, self.input_norm, eps)
        act = Act(x=h)
        if self.kind == "parallel":
            a, b = self.mixer.forward(act, batch, cache.layer_kv(self.idx), rope_cache, cache.states[self.idx])
            x = StreamDelta(a, self.conn1, y2=b, w1=self.mixer.left_norm, w2=self.mixer.right_norm)
        elif self.kind == "attention":
            x = StreamDelta(self.mixer.forward(act, batch, cache.layer_kv(self.idx), rope_cache), self.conn1)
        else:
            x = StreamDelta(self.mixer.forward(act, batch, cache.states[self.idx]), self.conn1)
        if self.ffn is not None:
            h, streams = ops.hyper_norm(streams, x, self.conn2.read, self.post_norm, eps)
            x = StreamDelta(self.ffn.forward(Act(x=h), batch=batch), self.conn2)
        return x, streams


class OutputNormLayer:
    """A layer whose norms sit on the sublayers' outputs: ``x += norm(mixer(x))``, then ``x += norm(ffn(x))`` where the layer has a
    feed-forward, on an fp32 residual stream that the sublayers read itself.  Same ``forward`` protocol as
    :class:`DecoderLayer`, with the pending :class:`NormDelta` in place of the previous layer's output.

    Where the configuration has them: layer norms in place of RMS norms, gates on the sublayers' results (from the stream as the
    sublayer gets it), a convolution on the mixer's input, a token input behind the feed-forward, and a weighted sum over all
    layers' results as what goes on."""

    def __init__(self, cfg: ModelConfig, idx: int, pctx: ParallelCtx, ep_mode: str = "auto"):
        spec = cfg.layer_specs[idx]
        self.cfg, self.idx = cfg.for_layer(idx), idx
        dense_kind, expert_kind = quant_kinds(cfg)
        self.kind, self.is_moe = spec.kind, cfg.is_moe_layer(idx)
        self.mixer = MIXERS[spec.kind](self.cfg, idx, pctx, dense_kind)
        self.ffn = None
        if spec.has_mlp:
            self.ffn = MoE(self.cfg, pctx, expert_kind, dense_kind, ep_mode) if self.is_moe else DenseMLP(self.cfg, pctx, dense_kind)
        self.input_norm: Optional[torch.Tensor] = None         # fp32, on the mixer's output
        self.post_norm: Optional[torch.Tensor] = None          # fp32, on the feed-forward's output
        self.input_bias: Optional[torch.Tensor] = None         # fp32: layer norms
        self.post_bias: Optional[torch.Tensor] = None
        self.conv = InputConvolution(cfg.hidden_size, cfg.input_conv_taps) if cfg.input_conv_taps else None
        if self.conv is not None and recurrent_of(self) is not self.conv:
            raise ValueError("a convolution on the input of a recurrent mixer needs a second state slot")
        self.gate1 = SublayerGate(cfg.hidden_size, dense_kind) if cfg.sublayer_gates else None
        self.gate2 = SublayerGate(cfg.hidden_size, dense_kind) if cfg.sublayer_gates and spec.has_mlp else None
        self.ffn_in: Optional[LinearWeight] = None             # the feed-forward's first product and its gate's in one
        self.side = TokenSide(cfg.hidden_size, cfg.token_side_dim, idx, dense_kind) if cfg.token_side_dim else None
        self.depth_factors: Optional[torch.Tensor] = None      # fp32 [idx + 2]: this layer's share of every result so far
        self.rope_override: Optional[torch.Tensor] = None      # this layer's own rotary table

    def init_random(self, gen, std, dtype, device):
        cfg = self.cfg
        fresh = lambda: torch.full((cfg.hidden_size,), 0.0 if cfg.norm_plus_one else 1.0, dtype=torch.float32, device=device)
        bias = lambda: torch.zeros(cfg.hidden_size, dtype=torch.float32, device=device) if cfg.layer_norms else None
        self.mixer.init_random(gen, std, dtype, device)
        self.input_norm, self.input_bias = fresh(), bias()
        if self.ffn is not None:
            self.ffn.init_random(gen, std, dtype, device)
            self.post_norm, self.post_bias = fresh(), bias()
        if self.conv is not None:
            self.conv.init_random(gen, dtype, device)
        for part in (self.gate1, self.gate2, self.side):
            if part is not None:
                part.init_random(gen, std, dtype, device)
        if cfg.depth_average:
            share = torch.rand(self.idx + 2, generator=gen, device=gen.device) * 0.1
            share[-1] = 1.0
            self.depth_factors = share.to(device)

    def fuse_inputs(self) -> None:
        """One product for the feed-forward's first projection, or its router, and for its gate, where the kernels take both (bf16, rows
        in whole 16-byte pieces, unquantised); the weights become its parts."""
        if self.gate2 is None or self.ffn_in is not None:
            return
        own = self.ffn.router if self.is_moe else self.ffn.gate_up
        g = self.gate2.w
        if (any(w.kind != "dense" or w.weight.dtype != torch.bfloat16 or w.bias is None or not ops.on_gpu(w.weight) for w in (own, g))
                or g.weight.shape[1] % 8 or not (self.is_moe or self.ffn.activation == "relu2")):
            return
        first, second = (g, own) if self.is_moe else (own, g)
        self.ffn_in = LinearWeight("dense", torch.cat([first.weight, second.weight], 0).contiguous(),
                                   bias=torch.cat([first.bias.float(), second.bias.float()]).contiguous())
        n = first.weight.shape[0]
        first.weight, second.weight = self.ffn_in.weight[:n], self.ffn_in.weight[n:]

    def accepts_prenormed(self) -> bool:
        return False

    def _feed_forward(self, act: Act, batch: ForwardBatch):
        """The feed-forward's output and the argument of its gate (None without one)."""
        ffn = self.ffn
        if self.ffn_in is not None and batch.adapter_rows is None and ops.on_gpu(act.x):
            if self.is_moe:
                z, logits = ops.linear_tail(act, self.ffn_in, self.cfg.hidden_size)
                return ffn.forward(act, batch=batch, rows_ok=True, logits=logits), z
            n = ffn.gate_up.weight.shape[0]
            both = ops.linear_relu2(act, self.ffn_in, n)
            return ffn.down_product(both[:, :n]), both[:, n:]
        y = ffn.forward(act, batch=batch, rows_ok=True) if self.is_moe else ffn.forward(act, batch=batch)
        return y, self.gate2.forward(act) if self.gate2 is not None else None

    def forward(self, x: NormDelta, stream: Optional[torch.Tensor], batch: ForwardBatch, cache: CacheStore, rope_cache, next_norm=None):
        eps, p1 = self.cfg.rms_norm_eps, self.cfg.norm_plus_one
        rope_cache = rope_cache if self.rope_override is None else self.rope_override
        history = x.depth.history if x.depth is not None else None
        h, stream = ops.add_normed(stream, x, eps, p1)
        u = h if self.conv is None else self.conv.forward(h, batch, cache.states[self.idx])
        if attention_of(self) is not None:
            y = self.mixer.forward(Act(x=u), batch, cache.layer_kv(self.idx), rope_cache)
        else:
            y = self.mixer.forward(Act(x=u), batch, cache.states[self.idx])
        x = NormDelta(y, self.input_norm, bias=self.input_bias, gate=self.gate1.forward(Act(x=h)) if self.gate1 is not None else None)
        if self.ffn is not None:
            h, stream = ops.add_normed(stream, x, eps, p1)
            y, z = self._feed_forward(Act(x=h), batch)
            x = NormDelta(y, self.post_norm, bias=self.post_bias, gate=z)
        if self.side is not None:
            h, stream = ops.add_normed(stream, x, eps, p1)
            x = NormDelta(self.side.forward(Act(x=h), batch.input_ids), self.side.norm)
        if history is not None:
            x.depth = DepthSum(history, self.idx + 1, self.depth_factors)
        return x, stream


class InputNormLayer:
    """A pre-norm layer of a model given by a list of layers: ``x += mixer(norm(x))``, then ``x += ffn(norm(x))`` where the layer has
    a feed-forward, on an fp32 residual stream.  One object per run of the layer: later passes of a looped layer share the
    weights of the first one and own a cache or state.  Same ``forward`` protocol as :class:`DecoderLayer`, with the pending
    :class:`NormDelta` in place of the previous layer's output."""

    def __init__(self, cfg: ModelConfig, idx: int, number: int, pctx: ParallelCtx, ep_mode: str = "auto"):
        """``idx``: place in the order of execution (cache and state); ``number``: place in the checkpoint."""
        spec = cfg.layer_specs[idx]
        self.cfg, self.idx, self.number = cfg.for_layer(idx), idx, number
        dense_kind, expert_kind = quant_kinds(cfg)
        self.kind, self.is_moe, self.shared = spec.kind, cfg.is_moe_layer(idx), spec.weights_of >= 0
        self.step_row = spec.step
        self.step: Optional[torch.Tensor] = None               # fp32: added to the residual ahead of this run
        self.mixer = MIXERS[spec.kind](self.cfg, number, pctx, dense_kind)
        self.ffn = None
        if spec.has_mlp:
            self.ffn = MoE(self.cfg, pctx, expert_kind, dense_kind, ep_mode) if self.is_moe else DenseMLP(self.cfg, pctx, dense_kind, paired=dense_kind == "dense")
        self.input_norm: Optional[torch.Tensor] = None         # fp32
        self.post_norm: Optional[torch.Tensor] = None
        self.rope_override: Optional[torch.Tensor] = None      # this layer's own rotary table

    def init_random(self, gen, std, dtype, device):
        fresh = lambda: torch.full((self.cfg.hidden_size,), 0.0 if self.cfg.norm_plus_one else 1.0, dtype=torch.float32, device=device)
        self.mixer.init_random(gen, std, dtype, device)
        self.input_norm = fresh()
        if self.ffn is not None:
            self.ffn.init_random(gen, std, dtype, device)
            self.post_norm = fresh()

    def share(self, first: "InputNormLayer") -> None:
        """Take the weights of the layer's first run.  The mixer is an object of its own: it keeps rows between speculative
        verification and commit."""
        self.mixer, self.ffn = copy.copy(first.mixer), first.ffn
        self.input_norm, self.post_norm = first.input_norm, first.post_norm

    def accepts_prenormed(self) -> bool:
        return False

    def forward(self, x: NormDelta, stream: Optional[torch.Tensor], batch: ForwardBatch, cache: CacheStore, rope_cache, next_norm=None):
        eps, p1 = self.cfg.rms_norm_eps, self.cfg.norm_plus_one
        rope_cache = rope_cache if self.rope_override is None else self.rope_override
        h, stream = ops.add_normed(stream, x, eps, p1, self.input_norm, step=self.step)
        if attention_of(self) is not None:
            x = NormDelta(self.mixer.forward(Act(x=h), batch, cache.layer_kv(self.idx), rope_cache))
        else:
            x = NormDelta(self.mixer.forward(Act(x=h), batch, cache.states[self.idx]))
        if self.ffn is not None:
            h, stream = ops.add_normed(stream, x, eps, p1, self.post_norm)
            x = NormDelta(self.ffn.forward(Act(x=h), batch=batch, rows_ok=True) if self.is_moe else self.ffn.forward(Act(x=h), batch=batch))
        return x, stream


def attention_of(layer):
    """The attention block of a layer (None without one): the owner of the layer's KV cache."""
    if layer.kind == "parallel":
        return layer.mixer.left
    return layer.mixer if layer.kind in ("attention", "latent_attention", "differential") else None


def recurrent_of(layer):
    """The block of a layer that owns a recurrent state slot: its mixer or the convolution on its input (None without one)."""
    if layer.kind in ("gdn", "mamba2", "wkv", "parallel", "mlstm", "rglru"):
        return layer.mixer
    return getattr(layer, "conv", None)


def kv_elements_of(attn) -> int:
    """Cached numbers per token of an attention block: a key and a value per head unless the block says otherwise."""
    n = getattr(attn, "kv_elements", None)
    return 2 * attn.hkv * attn.d if n is None else n


class DecoderLM:
    def __init__(self, cfg: ModelConfig, pctx: Optional[ParallelCtx] = None, device="cpu", ep_mode: str = "auto",
                 with_mtp: Optional[bool] = None):
        self.cfg = cfg
        self.pctx = pctx or ParallelCtx()
        self.device = torch.device(device)
        self.dtype = torch_dtype(cfg.dtype)
        if cfg.layer_specs:
            if bool(cfg.residual_streams) + cfg.output_norms + cfg.input_norms != 1:
                raise ValueError("a model given by a list of layers runs on hyper-connected residual streams, on normed outputs or on "
                                 "normed inputs")
            if cfg.input_norms:
                owners = [i for i, s in enumerate(cfg.layer_specs) if s.weights_of < 0]
                number = lambda i, s: owners.index(i if s.weights_of < 0 else s.weights_of)
                self.layers = [InputNormLayer(cfg, i, number(i, s), self.pctx, ep_mode) for i, s in enumerate(cfg.layer_specs)]
            elif any(s.weights_of >= 0 or s.step >= 0 for s in cfg.layer_specs):
                raise ValueError("layers run several times on normed inputs only")
            else:
                self.layers = [OutputNormLayer(cfg, i, self.pctx, ep_mode) if cfg.output_norms else StreamLayer(cfg, i, self.pctx)
                               for i in range(cfg.num_hidden_layers)]
        elif cfg.block_types:
            self.layers = [SingleBlock(cfg, i, self.pctx) for i in range(cfg.num_hidden_layers)]
        else:
            self.layers = [DecoderLayer(cfg, i, self.pctx, ep_mode) for i in range(cfg.num_hidden_layers)]
        self.embed: Optional[torch.Tensor] = None
        self.side_embed: Optional[torch.Tensor] = None       # [vocab, layers * token_side_dim]
        self.final_norm: Optional[torch.Tensor] = None
        self.final_bias: Optional[torch.Tensor] = None       # fp32: the final norm is a layer norm
        self.lm_head: Optional[LinearWeight] = None          # vocab-parallel slice under TP
        self.rope_cache: Optional[torch.Tensor] = None
        self.loop_step: Optional[torch.Tensor] = None        # fp32 [passes, hidden]: step vectors of looped layers
        self.mtp = None
        if (with_mtp if with_mtp is not None else cfg.mtp_num_layers > 0):
            from .mtp import MTPHead
            self.mtp = MTPHead(cfg, self.pctx, ep_mode)
        tp = self.pctx.tp_size
        self.vocab_parallel = tp > 1 and cfg.vocab_size % tp == 0
        self.sp_capacity_hint = 0            # the engine sets this to its largest step so the area is allocated once
        # layers whose output (the residual stream after the layer) is kept per step for a conditioned draft model
        self.capture_layers: Tuple[int, ...] = ()
        self.aux_hidden: List[torch.Tensor] = []
        self.dflash = None                   # models.dflash.BlockDiffusionDrafter
        self.vision = None                   # models.vision.VisionTower (multimodal checkpoints)
        if self.dtype == torch.float32 and self.device.type == "cuda":
            torch.backends.cuda.matmul.allow_tf32 = False      # a 32-bit model multiplies in full 32-bit

    # ------------------------------------------------------------------ weights
    def init_random(self, seed: int = 0, std: float = 0.02, max_pos: Optional[int] = None) -> "DecoderLM":
        cfg, dev, dt = self.cfg, self.device, self.dtype
        gen_dev = "cuda" if dev.type == "cuda" else "cpu"
        gen = torch.Generator(device=gen_dev)
        gen.manual_seed(seed)
        self.embed = randn_weight(gen, cfg.vocab_size, cfg.hidden_size, std, dt, dev)
        for layer in self.weight_layers():
            layer.init_random(gen, std, dt, dev)
        if cfg.loop_steps:
            self.loop_step = randn_weight(gen, cfg.loop_steps, cfg.hidden_size, std, torch.float32, dev)
        base = 0.0 if cfg.norm_plus_one else 1.0
        self.final_norm = torch.full((cfg.hidden_size,), base, dtype=torch.float32 if cfg.layer_specs else dt, device=dev)
        if cfg.layer_norms:
            self.final_bias = torch.zeros(cfg.hidden_size, dtype=torch.float32, device=dev)
        if cfg.token_side_dim:
            self.side_embed = randn_weight(gen, cfg.vocab_size, len(self.layers) * cfg.token_side_dim, 1.0, dt, dev)
        head = self.embed if cfg.tie_word_embeddings else randn_weight(gen, cfg.vocab_size, cfg.hidden_size, std, dt, dev)
        self.set_lm_head(head)
        if self.mtp is not None:
            self.mtp.init_random(gen, std, dt, dev)
        self.finalize(max_pos)
        return self

    def weight_layers(self) -> list:
        """The layers that own weights, in the checkpoint's order (one entry per layer, however often it runs)."""
        return [l for l in self.layers if not getattr(l, "shared", False)]

    def enable_lora(self, max_slots: int = 7):
        """Attach one adapter set to the attention, dense-FFN and mixture-of-experts blocks of every layer."""
        from ..lora import LoraSet
        if getattr(self, "lora", None) is None:
            self.lora = LoraSet(max_slots)
            for l in self.layers:
                if attention_of(l) is not None and getattr(attention_of(l), "takes_adapters", True):
                    attention_of(l).lora = self.lora
                if l.ffn is None:
                    continue
                prefix = f"layers.{getattr(l, 'number', l.idx)}.mlp."
                l.ffn.lora, l.ffn.lora_prefix = self.lora, prefix
                shared = getattr(l.ffn, "shared", None)
                if shared is not None:
                    shared.lora, shared.lora_prefix = self.lora, prefix + "shared_expert."
        return self.lora

    def set_kv_rotation(self, on: bool = True) -> bool:
        """"turbo8" cache: every plain attention layer (the draft head's included) rotates its q / k / v heads with the
        orthonormal Walsh-Hadamard transform before the FP8 cache write and rotates the attention output back.  Dot
        products are unchanged (the transform is orthogonal), rotated coordinates are near-Gaussian, so the FP8 range
        is not spent on a few outlier channels.  Returns False (nothing changed) when the model has layers the rotation
        does not cover: latent attention, or a head size other than 128 with full rotary width on the GPU.
        Reference: ``kernels/gb10/common/reshape_and_cache_turbo.cu`` (turbo8 = WHT + e4m3)."""
        from ..layers.attention import Attention
        cfg = self.cfg
        d = cfg.head_dim
        if cfg.kv_lora_rank > 0 or cfg.layer_specs or d & (d - 1):
            return False
        if self.device.type == "cuda" and not (d == 128 and cfg.rotary_dim == 128):
            return False
        layers = list(self.layers) + ([self.mtp.layer] if self.mtp is not None else [])
        for l in layers:
            if isinstance(getattr(l, "mixer", None), Attention):
                l.mixer.kv_rotate = bool(on)
        return True

    def register_adapter(self, adapter) -> int:
        """Make ``adapter`` (whole, as loaded) resident on this rank, cut like the base weights; returns its slot."""
        from ..lora import localize
        return self.enable_lora().register(localize(adapter, self))

    def set_lm_head(self, head: torch.Tensor) -> None:
        if self.vocab_parallel:
            head = shard_rows(head, self.pctx.tp_rank, self.pctx.tp_size).contiguous()
        self.lm_head = LinearWeight("dense", head)

    def finalize(self, max_pos: Optional[int] = None) -> None:
        cfg = self.cfg
        mp = max_pos or cfg.max_position_embeddings
        for l, spec in zip(self.layers, cfg.layer_specs if cfg.input_norms else ()):
            if spec.weights_of >= 0:
                l.share(self.layers[spec.weights_of])
            l.step = self.loop_step[spec.step] if spec.step >= 0 else None
        self.rope_cache = ref.build_rope_cache(cfg.rotary_dim, mp, cfg.rope_theta, cfg.rope_scaling, self.device)
        if cfg.rope_local_theta:
            local = ref.build_rope_cache(cfg.rotary_dim, mp, cfg.rope_local_theta, None, self.device)
            for l in self.layers:
                if l.kind == "attention" and getattr(l.mixer, "local", False):
                    l.rope_override = local
        for l in self.layers:
            if l.is_moe:
                l.ffn.fuse_inputs()
            if isinstance(l, OutputNormLayer):
                l.fuse_inputs()
                if l.side is not None:
                    l.side.table = self.side_embed
        tables: Dict[str, torch.Tensor] = {}
        for l in self.layers if cfg.layer_specs else ():
            if attention_of(l) is not None:
                key = (l.cfg.rotary_dim, l.cfg.rope_theta, l.cfg.rope_scaling)
                if str(key) not in tables:
                    tables[str(key)] = ref.build_rope_cache(key[0], mp, key[1], key[2], self.device)
                l.rope_override = tables[str(key)]

    # ------------------------------------------------------------------ cache allocation
    def attention_layers(self) -> List[int]:
        return [l.idx for l in self.layers if attention_of(l) is not None]

    def gdn_layers(self) -> List[int]:
        """Layers with a recurrent state slot (Gated DeltaNet, Mamba-2, WKV, attention beside Mamba-2)."""
        return [l.idx for l in self.layers if recurrent_of(l) is not None]

    def _cache_dtype(self, layer, kv_dtype, high_precision) -> torch.dtype:
        """Cache dtype of one layer: the engine's, 16 bits for layers that ask for high precision, the model's own for
        attention variants (chunks, sinks) whose kernels read nothing else."""
        a = attention_of(layer)
        if not getattr(a, "plain", True):
            return self.dtype
        if layer.idx in high_precision and kv_dtype_is_quantised(kv_dtype):
            return torch.bfloat16 if self.dtype == torch.bfloat16 else self.dtype
        return kv_dtype

    def kv_bytes_per_block(self, block_size: int, kv_dtype: torch.dtype, high_precision_layers=()) -> int:
        if self.cfg.layer_specs:
            owners = [(l, attention_of(l)) for l in self.layers if attention_of(l) is not None]
            return int(sum(block_size * kv_elements_of(a) * kv_element_bytes(self._cache_dtype(l, kv_dtype, set(high_precision_layers)))
                           for l, a in owners))
        n_attn = len(self.attention_layers()) + (1 if self.mtp is not None else 0)
        hkv = self.layers[self.attention_layers()[0]].mixer.hkv if n_attn else 0
        n_hi = len([i for i in self.attention_layers() if i in set(high_precision_layers)])
        per = 2 * block_size * hkv * self.cfg.head_dim
        return int(per * ((n_attn - n_hi) * kv_element_bytes(kv_dtype) + n_hi * max(2.0, kv_element_bytes(kv_dtype))))

    def alloc_cache(self, num_blocks: int, block_size: int, kv_dtype: torch.dtype, state_slots: int = 0,
                    high_precision_layers=()) -> CacheStore:
        """``high_precision_layers``: attention layers whose cache stays in 16 bits when ``kv_dtype`` is FP8 or NVFP4 (the
        layers most sensitive to KV quantisation, typically the first and last ones)."""
        store = CacheStore(block_size=block_size, num_blocks=num_blocks)
        hi = set(high_precision_layers)
        for l in self.layers:
            a = attention_of(l)
            if a is not None:
                dt = self._cache_dtype(l, kv_dtype, hi)
                own = getattr(a, "alloc_kv", None)
                store.kv[l.idx] = (own(num_blocks, block_size, dt, self.device) if own is not None
                                   else alloc_kv(num_blocks, block_size, a.hkv, a.d, dt, self.device))
                store.kv_scales[l.idx] = (1.0, 1.0)
            if recurrent_of(l) is not None:
                store.states[l.idx] = recurrent_of(l).alloc_state(max(1, state_slots), self.device, self.dtype)
        if self.mtp is not None:
            self.mtp.alloc_cache(store, num_blocks, block_size, kv_dtype, self.device)
        return store

    # ------------------------------------------------------------------ forward
    def embed_tokens(self, ids: torch.Tensor) -> torch.Tensor:
        from ..ops import checked
        if checked.ENABLED:
            checked.index_range("input_ids", ids, 0, self.cfg.vocab_size)
        e = self.embed[ids.long()]
        if self.cfg.embed_scale != 1.0 and not (self.cfg.residual_streams or self.cfg.input_norms):
            e = e * torch.tensor(self.cfg.embed_scale, dtype=e.dtype)      # the factor is rounded to the weight dtype first
        return e

    # ------------------------------------------------------------------ sequence-parallel prefill (tensor parallel)
    def _seq_parallel_area(self, batch: ForwardBatch, T: int):
        """The peer-memory area for a sequence-parallel step, or None when this step takes the replicated path.
        Decided from the model, the configuration and the step's row count only, so every rank decides alike."""
        p = self.pctx
        if p.tp_size <= 1 or p.comm is None or not hasattr(p.comm, "seq_parallel"):
            return None
        # prefill-size steps are owned in 128-row blocks; pure decode steps of at most 128 rows are owned row by row
        # (every rank reduces and normalises T / world rows), which pays off once the all-reduce latency of a wide
        # group dominates the step
        decode_sp = (SEQ_PARALLEL_DECODE_MIN_WORLD > 0 and p.tp_size >= SEQ_PARALLEL_DECODE_MIN_WORLD and T <= 128
                     and batch.num_decodes == batch.num_seqs and batch.max_query_len == 1)
        if T < SEQ_PARALLEL_MIN_TOKENS and not decode_sp:
            return None
        if batch.adapter_rows is not None or self.device.type != "cuda" or ops.FORCE_REFERENCE:
            return None
        if torch.cuda.is_current_stream_capturing():
            # a captured step may use an area that already exists (the eager passes before the capture create it); it
            # must never allocate or rendezvous
            areas = getattr(p.comm, "_sp_areas", None)
            area = areas.get(self.cfg.hidden_size) if (decode_sp and areas) else None
            if area is None or area.t_pad < T or not getattr(self, "_sp_model_ok", False):
                return None
            return area
        ok = getattr(self, "_sp_model_ok", None)
        if ok is None:
            ok = self.dtype == torch.bfloat16 and self.cfg.hidden_size % 256 == 0 and not self.cfg.sandwich_norms and all(
                l.kind == "attention" and not l.is_moe and l.ffn.shard and l.mixer.qkv.kind == "fp8_block"
                and l.mixer.o.kind == "fp8_block" and l.ffn.gate_up.kind == "fp8_block" and l.ffn.down.kind == "fp8_block"
                and l.mixer.o.bias is None and l.ffn.down.bias is None for l in self.layers)
            self._sp_model_ok = ok
        if not ok:
            return None
        return p.comm.seq_parallel(max(T, self.sp_capacity_hint), self.cfg.hidden_size)

    def _forward_seq_parallel(self, x: torch.Tensor, batch: ForwardBatch, cache: CacheStore, sp) -> torch.Tensor:
        """Dense tensor-parallel layers with a row-sharded residual stream: every row-parallel GEMM scatters its
        partial tiles to the row owners, the owner reduces, normalises and quantises its rows once and gathers them to
        all ranks, and the next column-parallel GEMM consumes the rows as they arrive."""
        cfg = self.cfg
        eps, p1 = cfg.rms_norm_eps, cfg.norm_plus_one
        res = sp.residual_shard(x)
        act, _ = ops.rmsnorm_act(x, self.layers[0].input_norm, eps, None, p1, True)
        n = len(self.layers)
        hidden = None
        for i, layer in enumerate(self.layers):
            out = layer.mixer.mix(act, batch, cache.layer_kv(layer.idx), self.rope_cache)
            sp.gemm_rs(out if isinstance(out, Act) else Act(x=out), layer.mixer.o)
            act = sp.reduce_norm(res, layer.post_norm, eps, p1)
            sp.gemm_rs(layer.ffn.hidden_act(act), layer.ffn.down)
            if i + 1 < n:
                act = sp.reduce_norm(res, self.layers[i + 1].input_norm, eps, p1)
            else:
                hidden = sp.reduce_hidden(res)
        self.last_prenorm = (hidden, None)
        y, _ = ops.rmsnorm(hidden, self.final_norm, eps, None, p1)
        return y

    @torch.inference_mode()
    def forward(self, batch: ForwardBatch, cache: CacheStore, layer_ids: Optional[List[int]] = None) -> torch.Tensor:
        """Returns the final-normed hidden states ``[T,H]`` of every row.  ``layer_ids`` runs only those layers, in
        order (the layer-skipping draft pass of self-speculative decoding: the kept layers read and write their own KV
        entries, the skipped ones are not touched)."""
        x = batch.inputs_embeds if batch.inputs_embeds is not None else self.embed_tokens(batch.input_ids)
        sp = self._seq_parallel_area(batch, x.shape[0]) if (not self.capture_layers and layer_ids is None) else None
        if sp is not None:
            return self._forward_seq_parallel(x, batch, cache, sp)
        residual = None
        if self.cfg.residual_streams:
            x = StreamDelta(x, scale=self.cfg.embed_scale)      # fp32 streams start from the scaled embedding
        elif self.cfg.output_norms or self.cfg.input_norms:
            x = NormDelta(x, scale=self.cfg.embed_scale if self.cfg.input_norms else 1.0)      # so does a plain fp32 stream
            if self.cfg.depth_average:
                entries = torch.empty((len(self.layers) + 1,) + tuple(x.y.shape), dtype=torch.float32, device=x.y.device)
                x.depth = DepthSum(entries, 0)
        elif batch.inputs_embeds is not None:
            x = x.clone()                     # fused epilogues update the residual stream in place
        if layer_ids is not None:
            layers = [self.layers[i] for i in layer_ids]
            for k, layer in enumerate(layers):
                nxt = layers[k + 1] if k + 1 < len(layers) else None
                next_norm = nxt.input_norm if (nxt is not None and nxt.accepts_prenormed()) else None
                x, residual = layer.forward(x, residual, batch, cache, self.rope_cache, next_norm=next_norm)
            return self._final_norm(x, residual)
        n = len(self.layers)
        self.aux_hidden = []
        for i, layer in enumerate(self.layers):
            nxt = self.layers[i + 1] if i + 1 < n else None
            next_norm = nxt.input_norm if (nxt is not None and nxt.accepts_prenormed()) else None
            x, residual = layer.forward(x, residual, batch, cache, self.rope_cache, next_norm=next_norm)
            if i in self.capture_layers and isinstance(x, (StreamDelta, NormDelta)):
                self.aux_hidden.append(self._stream_sum(x, residual))
            elif i in self.capture_layers:
                # the stream after layer i: already summed when the layer's epilogue handed over normalised activations
                self.aux_hidden.append(residual.clone() if isinstance(x, Act) else (x + residual if residual is not None else x.clone()))
        self.last_prenorm = (x, residual)
        return self._final_norm(x, residual)

    def _final_norm(self, x, residual) -> torch.Tensor:
        if isinstance(x, StreamDelta):
            y, _ = ops.hyper_norm(residual, x, self._stream_ones, self.final_norm, self.cfg.rms_norm_eps, write=False)
            return y
        if isinstance(x, NormDelta):
            return ops.add_normed(residual, x, self.cfg.rms_norm_eps, self.cfg.norm_plus_one, self.final_norm, write=False, out_bias=self.final_bias)[0]
        y, _ = ops.rmsnorm(x, self.final_norm, self.cfg.rms_norm_eps, residual, self.cfg.norm_plus_one)
        return y

    @property
    def _stream_ones(self) -> torch.Tensor:
        t = getattr(self, "_ones", None)
        if t is None:
            t = self._ones = torch.ones(self.cfg.residual_streams, dtype=torch.float32, device=self.device)
        return t

    def _stream_sum(self, x, streams: torch.Tensor) -> torch.Tensor:
        """Sum of the residual streams with a pending update applied (fp32)."""
        if isinstance(x, NormDelta):
            return ops.add_normed(streams.clone(), x, self.cfg.rms_norm_eps, self.cfg.norm_plus_one)[1]
        _, after = ops.hyper_norm(streams.clone(), x, self._stream_ones, self.final_norm, self.cfg.rms_norm_eps)
        return after.sum(1)

    @torch.inference_mode()
    def compute_logits(self, hidden: torch.Tensor, indices: Optional[torch.Tensor] = None) -> torch.Tensor:
        h = hidden if indices is None else hidden[indices]
        logits = ops.linear(h, self.lm_head)
        if self.vocab_parallel and self.pctx.comm is not None:
            logits = self.pctx.comm.all_gather(logits, dim=-1)
        cap = self.cfg.final_logit_softcapping
        if cap:
            logits = torch.tanh(logits.float() / cap).mul_(cap).to(logits.dtype)
        return logits

    def build_draft_head(self, row_ids: List[int], kind: str = "fp8_block") -> None:
        """A draft-only language-model head over the token ids ``row_ids`` (ascending), quantised to ``kind``: draft
        steps score these rows instead of the whole vocabulary (``draft_top1``).  On a vocabulary-parallel rank the head
        holds the chosen rows of this rank's shard.  Reference: ``crates/spark-model/src/layers/mtp_head/ranked_head.rs``
        (draft-only quantised head built from ranked rows of the full head)."""
        ids = torch.tensor(sorted(int(t) for t in row_ids), dtype=torch.long)
        lo = 0
        if self.vocab_parallel:
            shard = self.cfg.vocab_size // self.pctx.tp_size
            lo = self.pctx.tp_rank * shard
            ids = ids[(ids >= lo) & (ids < lo + shard)]
        if ids.numel() == 0:
            ids = torch.tensor([lo], dtype=torch.long)          # a rank never holds an empty head
        n = int(ids.numel())
        if self.device.type == "cuda" and n % 128:
            # the GEMM tiles want a multiple of 128 rows: repeat the last row (same logit, same token id, so the
            # argmax is unchanged) rather than add zero rows that could win against negative logits
            ids = torch.cat([ids, ids[-1:].expand(128 - n % 128)])
        w = self.lm_head.dequantized()[(ids - lo).to(self.lm_head.weight.device)]
        if kind == "fp8_block" and (w.shape[1] % 128 or not w.is_floating_point()):
            kind = "dense"
        self.draft_head = LinearWeight.from_dense(w.contiguous(), kind)
        self.draft_row_ids = ids.to(self.device)
        self.draft_rows = n

    @torch.inference_mode()
    def draft_top1(self, hidden: torch.Tensor, want_logprob: bool = False):
        """``(token ids [B], ln p(top-1) [B] or None)`` of a draft step: over the draft head's rows when one was built,
        over the whole vocabulary otherwise.  The probability is taken over the rows that were scored."""
        if getattr(self, "draft_head", None) is None:
            lg = self.compute_logits(hidden)
            tok = ops.argmax(lg)
            lp = lg.float().log_softmax(-1).gather(-1, tok.view(-1, 1).long())[:, 0] if want_logprob else None
            return tok, lp
        lg = ops.linear(hidden, self.draft_head)
        cap = self.cfg.final_logit_softcapping
        if cap:
            lg = torch.tanh(lg.float() / cap).mul_(cap).to(lg.dtype)
        idx, val = ops.argmax(lg, with_value=True)
        tok = self.draft_row_ids[idx.long()]
        lse = torch.logsumexp(lg[:, :self.draft_rows].float(), -1) if want_logprob else None      # not the repeated rows
        if self.vocab_parallel and self.pctx.comm is not None:
            cols = [val.double(), tok.double()] + ([lse.double()] if want_logprob else [])
            allp = self.pctx.comm.all_gather(torch.stack(cols, 1), dim=1).view(val.shape[0], self.pctx.tp_size, len(cols))
            best = ref.argmax_first(allp[..., 0])
            tok = allp[..., 1].gather(1, best[:, None])[:, 0].to(torch.int64)
            val = allp[..., 0].gather(1, best[:, None])[:, 0]
            if want_logprob:
                lse = torch.logsumexp(allp[..., 2], -1)
        lp = (val.float() - lse.float()) if want_logprob else None
        return tok, lp

    @torch.inference_mode()
    def greedy_tokens(self, hidden: torch.Tensor, indices: Optional[torch.Tensor] = None) -> torch.Tensor:
        """Argmax token per row without materialising the full-vocabulary logits on any rank: each rank takes the
        argmax of its vocabulary shard, the ranks exchange one (max, index) pair per row and the best shard wins
        (ties go to the lowest global index).  Replaces the all-gather of ``[rows, vocab]`` logits of
        :meth:`compute_logits` when every row of the step is plain greedy."""
        h = hidden if indices is None else hidden[indices]
        logits = ops.linear(h, self.lm_head)
        idx, val = ops.argmax(logits, with_value=True)
        if not (self.vocab_parallel and self.pctx.comm is not None):
            return idx
        shard = self.cfg.vocab_size // self.pctx.tp_size
        pair = torch.stack([val.double(), (idx + self.pctx.tp_rank * shard).double()], dim=1)       # [B, 2], exact
        allp = self.pctx.comm.all_gather(pair, dim=1).view(pair.shape[0], self.pctx.tp_size, 2)
        vals, ids = allp[..., 0], allp[..., 1]
        best = ref.argmax_first(vals)
        return ids.gather(1, best[:, None])[:, 0].to(torch.int64)

    def commit_spec(self, accepted_rows: List[int], cache: CacheStore) -> None:
        """After speculative verification: fold the accepted rows into every GDN layer's state."""
        for l in self.layers:
            if recurrent_of(l) is not None:
                recurrent_of(l).commit(accepted_rows, cache.states[l.idx])

    # ------------------------------------------------------------------ oracle
    @torch.inference_mode()
    def forward_dense_reference(self, token_ids: List[int]) -> torch.Tensor:
        """Plain eager forward of ONE sequence without any paging (logits of every position).

        Used by tests as the "plain eager forward" that the paged/batched engine must match.
        """
        n = len(token_ids)
        bs = 16
        nblk = (n + bs - 1) // bs
        kv_dtype = self.dtype
        tmp = self.alloc_cache(nblk, bs, kv_dtype, state_slots=1)
        fb = ForwardBatch.build([list(token_ids)], [0], [list(range(nblk))], bs, device=self.device,
                                state_slots=[0], has_state=[False], all_logits=True)
        h = self.forward(fb, tmp)
        return self.compute_logits(h)
