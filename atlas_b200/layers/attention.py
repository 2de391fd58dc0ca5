"""GQA attention block over the paged KV cache (optionally with q/k head norms and an output gate).

Data flow per step: fused QKV GEMM -> fused (q/k RMSNorm) + RoPE + FP8 quant + paged-cache write ->
paged attention (split-K decode kernel for single-row sequences, tiled prefill kernel for chunks) ->
(sigmoid gate) -> row-parallel output GEMM whose tensor-parallel reduction is fused into its epilogue.

Reference parity: ``crates/spark-model/src/layers/qwen3_attention/`` (decode:
``trait_impl/decode_inner.rs``, prefill: ``trait_impl/prefill_inner.rs``).
"""
from __future__ import annotations

import math
from typing import Dict, Optional, Tuple

import torch

from .. import ops
from ..config import ModelConfig
from ..ops import Act, LinearWeight
from ..lora import GATE_SUFFIX, add_delta
from .common import ParallelCtx, TailLinear, make_weight, randn_weight, shard_cols, shard_rows
from .mla import deinterleave_rows


def distance_bucket(n: int, rows: int, reach: int) -> int:
    """Row of a distance table for a key ``n`` tokens back: the first half of the rows are single distances, the others widen
    logarithmically up to ``reach``, and everything beyond shares the last one."""
    half = rows // 2
    if n < half:
        return n
    if n >= reach:
        return rows - 1
    far = rows - half
    b = int(math.log(n / half) / math.log(reach / half) * far)
    # the bucket is the largest b with (reach / half)^b <= (n / half)^far, which integers decide where logarithms round
    holds = lambda c: reach ** c * half ** far <= n ** far * half ** c
    while not holds(b):
        b -= 1
    while holds(b + 1):
        b += 1
    return min(rows - 1, half + b)


def distance_table(rel: torch.Tensor, reach: int) -> torch.Tensor:
    """``rel [rows, heads]`` per bucket -> fp32 ``[heads, n]`` per distance; keys from ``n - 1`` tokens on share the last column."""
    rows = rel.shape[0]
    if rows < 2 or reach < 1:
        raise ValueError(f"a distance table of {rows} rows does not reach {reach} tokens")
    idx = torch.tensor([distance_bucket(n, rows, reach) for n in range(max(reach, rows // 2) + 1)], device=rel.device)
    return rel.float()[idx].t().contiguous()


class Attention:
    def __init__(self, cfg: ModelConfig, layer_idx: int, pctx: ParallelCtx, quant_kind: str):
        self.cfg, self.layer_idx, self.pctx = cfg, layer_idx, pctx
        tp = pctx.tp_size
        assert cfg.num_attention_heads % tp == 0, "query heads must divide by tp"
        self.hq = cfg.num_attention_heads // tp
        self.hkv = max(1, cfg.num_key_value_heads // tp)
        self.kv_rep = max(1, tp // cfg.num_key_value_heads)     # ranks sharing one kv head
        # ``d`` is the width of a head in the cache and the kernels; query / key and value heads of other sizes are
        # zero-padded to it by their projections, which leaves scores and outputs unchanged
        self.dqk, self.dv = cfg.head_dim, cfg.v_head_dim or cfg.head_dim
        self.d = cfg.attn_cache_width or cfg.head_dim
        self.gated = cfg.attn_output_gate
        self.scale = cfg.attn_scale or self.dqk ** -0.5
        self.chunk = cfg.attn_chunk         # > 0: a token sees keys of its own ``chunk``-token block of the sequence only
        self.sinks: Optional[torch.Tensor] = None       # [hq] fp32: extra term exp(sink) of the softmax denominator
        self.softcap = cfg.attn_softcap     # > 0: scores are bounded before the softmax
        self.norm_plus_one = cfg.norm_plus_one if cfg.qk_norm_plus_one is None else cfg.qk_norm_plus_one
        self.distance: Optional[torch.Tensor] = None    # [hq, n] fp32: bias of a score by the distance of its key
        self.gated_qkv: Optional[TailLinear] = None     # head gates: q | k | v with one gate number per head as an fp32 tail
        # models with per-layer attention kinds (Gemma): only "sliding_attention" layers use the window
        kinds = cfg.layer_types if (cfg.family != "hybrid" and cfg.layer_types) else None
        self.local = bool(kinds) and kinds[layer_idx] == "sliding_attention"
        self.window = cfg.sliding_window if (kinds is None or self.local) else None
        self.quant_kind = quant_kind
        self.qkv: Optional[LinearWeight] = None
        self.o: Optional[LinearWeight] = None
        self.q_norm: Optional[torch.Tensor] = None
        self.k_norm: Optional[torch.Tensor] = None
        self.lora = None                    # lora.LoraSet shared by the model's layers
        self.selector = None                # kv.sparse_select.BlockSelector: block-selected decode attention (long contexts)
        self.kv_rotate = False              # "turbo8" cache: q / k / v heads Hadamard-rotated before the FP8 cache write

    # ------------------------------------------------------------------ weights
    def _kv_slice(self, w: torch.Tensor) -> torch.Tensor:
        tp, r = self.pctx.tp_size, self.pctx.tp_rank
        if tp == 1:
            return w
        head = (r // self.kv_rep) * self.hkv
        return w[head * self.d:(head + self.hkv) * self.d]

    def load(self, q: torch.Tensor, k: torch.Tensor, v: torch.Tensor, o: torch.Tensor,
             q_norm=None, k_norm=None, qkv_bias: Optional[Tuple] = None, sinks: Optional[torch.Tensor] = None,
             head_gate: Optional[torch.Tensor] = None, rel: Optional[torch.Tensor] = None, rope_interleaved: bool = False) -> None:
        """Takes full (unsharded) HF-layout tensors; slices for this rank, fuses, quantizes.  ``qkv_bias``: the three
        projections' biases; ``rel [rows, heads]``: the distance table; ``rope_interleaved``: rotated dimensions are paired
        (2i, 2i + 1) and move to the half-split order on both sides of the score.  Norm weights are one head's, or with
        ``qk_norm_rows`` those of all heads."""
        cfg, tp, r = self.cfg, self.pctx.tp_size, self.pctx.tp_rank
        cols = lambda b: None if b is None else b.reshape(-1, 1)
        bias = [cols(b) for b in qkv_bias] if qkv_bias is not None else None
        row_norm = cfg.qk_norm_rows
        if rope_interleaved and cfg.rotary_dim:
            turn = lambda w: None if w is None else self._half_split(w)
            q, k = turn(q), turn(k)
            bias = bias and [turn(bias[0]), turn(bias[1]), bias[2]]
            q_norm, k_norm = ((turn(cols(n))[:, 0] if n is not None else None) for n in (q_norm, k_norm))
        if self.d != self.dqk or self.d != self.dv:
            assert not self.gated, "padded heads: plain q / k / v projections only"
            pad = lambda n: None if n is None else self._pad_rows(cols(n), self.dqk)[:, 0]
            q_norm, k_norm = pad(q_norm), pad(k_norm)
            q, k, v = self._pad_rows(q, self.dqk), self._pad_rows(k, self.dqk), self._pad_rows(v, self.dv)
            bias = bias and [self._pad_rows(b, n) for b, n in zip(bias, (self.dqk, self.dqk, self.dv))]
            o = self._pad_rows(o.t(), self.dv).t()
        if row_norm and q_norm is not None:
            q_norm = shard_rows(cols(q_norm), r, tp)[:, 0].float().contiguous()
            k_norm = self._kv_slice(cols(k_norm))[:, 0].float().contiguous()
        if bias is not None:
            assert not self.gated and head_gate is None, "biased projections have no gates"
            bias = torch.cat([shard_rows(bias[0], r, tp), self._kv_slice(bias[1]), self._kv_slice(bias[2])], 0)[:, 0].to(q.dtype).contiguous()
        if rel is not None:
            self.distance = distance_table(shard_rows(rel.t(), r, tp).t(), cfg.attn_distance_reach).to(o.device)
        if sinks is None and cfg.attn_sink_score is not None:
            sinks = torch.full((cfg.num_attention_heads,), float(cfg.attn_sink_score), dtype=torch.float32, device=o.device)
        if sinks is not None:
            self.sinks = shard_rows(sinks.reshape(-1, 1), r, tp).reshape(-1).float().to(o.device).contiguous()
        if self.gated:   # HF q_proj rows are per head [q(D) | gate(D)]
            qg = q.view(cfg.num_attention_heads, 2, self.d, -1)
            q, gate = qg[:, 0].reshape(-1, q.shape[-1]), qg[:, 1].reshape(-1, q.shape[-1])
        parts = [shard_rows(q, r, tp), self._kv_slice(k), self._kv_slice(v)]
        if self.gated:
            parts.append(shard_rows(gate, r, tp))
        fused = torch.cat(parts, 0)
        if head_gate is not None:
            self.gated_qkv = TailLinear(fused, shard_rows(head_gate, r, tp), self.quant_kind)
            self.qkv = self.gated_qkv.w
        else:
            self.qkv = make_weight(fused, self.quant_kind, bias)
        self.o = make_weight(shard_cols(o, r, tp).contiguous(), self.quant_kind)
        self.q_norm, self.k_norm = q_norm, k_norm

    def _half_split(self, w: torch.Tensor) -> torch.Tensor:
        """Rows of every ``dqk``-row head with the rotated ones in half-split order."""
        heads = w.reshape(-1, self.dqk, w.shape[-1])
        n = self.cfg.rotary_dim
        order = deinterleave_rows(torch.arange(n).view(n, 1), n)[:, 0].to(w.device)
        return torch.cat([heads[:, order], heads[:, n:]], 1).reshape(w.shape)

    def _pad_rows(self, w: torch.Tensor, d: int) -> torch.Tensor:
        """``[heads * d, K]`` with every head's rows zero-padded to the cache width."""
        if d == self.d:
            return w
        heads = w.reshape(-1, d, w.shape[-1])
        return torch.nn.functional.pad(heads, (0, 0, 0, self.d - d)).reshape(-1, w.shape[-1])

    def init_random(self, gen, std, dtype, device) -> None:
        cfg = self.cfg
        h = cfg.hidden_size
        qmul = 2 if self.gated else 1
        q = randn_weight(gen, cfg.num_attention_heads * self.dqk * qmul, h, std, dtype, device)
        k = randn_weight(gen, cfg.num_key_value_heads * self.dqk, h, std, dtype, device)
        v = randn_weight(gen, cfg.num_key_value_heads * self.dv, h, std, dtype, device)
        o = randn_weight(gen, h, cfg.num_attention_heads * self.dv, std, dtype, device)
        qn = kn = None
        if cfg.qk_norm:
            base = float(not self.norm_plus_one)
            nq, nk = (cfg.num_attention_heads, cfg.num_key_value_heads) if cfg.qk_norm_rows else (1, 1)
            qn = torch.full((nq * self.dqk,), base, dtype=dtype, device=device)
            kn = torch.full((nk * self.dqk,), base, dtype=dtype, device=device)
        learned = cfg.attn_sinks and cfg.attn_sink_score is None
        sinks = torch.zeros(cfg.num_attention_heads, dtype=torch.float32, device=device) if learned else None
        gate = randn_weight(gen, cfg.num_attention_heads, h, std, dtype, device) if cfg.attn_head_gate else None
        bias = tuple(randn_weight(gen, w.shape[0], 1, std, dtype, device)[:, 0] for w in (q, k, v)) if cfg.attention_bias else None
        rel = randn_weight(gen, cfg.attn_distance_rows, cfg.num_attention_heads, 0.5, torch.float32, device) if cfg.attn_distance_rows else None
        self.load(q, k, v, o, qn, kn, qkv_bias=bias, sinks=sinks, head_gate=gate, rel=rel)

    @property
    def plain(self) -> bool:
        """No chunked visibility, sink, bounded scores, distance bias or norm over all heads: every cache dtype and attention
        kernel applies.  Otherwise the layer keeps a cache in the model's own dtype."""
        return not (self.chunk or self.cfg.attn_sinks or self.softcap or self.cfg.attn_distance_rows or self.cfg.qk_norm_rows)

    # ------------------------------------------------------------------ forward
    def forward(self, act: Act, batch, kv: Tuple[torch.Tensor, torch.Tensor, float, float],
                rope_cache: torch.Tensor) -> torch.Tensor:
        out = self.mix(act, batch, kv, rope_cache)
        if self.lora is not None and batch.adapter_rows is not None:
            # this rank's columns of A give a partial delta: it joins the partial product before the group reduction
            y = ops.linear(out, self.o)
            add_delta(y, self.lora, f"layers.{self.layer_idx}.self_attn.o_proj", out, batch)
            return self.pctx.all_reduce(y)
        return self.pctx.row_parallel_linear(out, self.o)

    def mix(self, act: Act, batch, kv: Tuple[torch.Tensor, torch.Tensor, float, float],
            rope_cache: torch.Tensor):
        """Everything before the output projection: this rank's heads' attention output ``[T, hq * d]`` (a tensor, or an
        ``Act`` holding its FP8 form when the attention kernel quantised it)."""
        cfg = self.cfg
        k_cache, v_cache, k_scale, v_scale = kv
        qkv, head_gate = self.gated_qkv(act) if self.gated_qkv is not None else (ops.linear(act, self.qkv), None)
        T = qkv.shape[0]
        nq, nkv = self.hq * self.d, self.hkv * self.d
        if self.lora is not None and batch.adapter_rows is not None:
            xin, pre = act.plain(), f"layers.{self.layer_idx}.self_attn."
            add_delta(qkv, self.lora, pre + "q_proj", xin, batch, 0, nq)
            add_delta(qkv, self.lora, pre + "k_proj", xin, batch, nq, nkv)
            add_delta(qkv, self.lora, pre + "v_proj", xin, batch, nq + nkv, nkv)
            if self.gated:
                add_delta(qkv, self.lora, pre + "q_proj" + GATE_SUFFIX, xin, batch, nq + 2 * nkv, nq)
        q = qkv[:, :nq].view(T, self.hq, self.d)
        k = qkv[:, nq:nq + nkv].view(T, self.hkv, self.d)
        v = qkv[:, nq + nkv:nq + 2 * nkv].view(T, self.hkv, self.d)
        rope_pos, rope_cache = batch.rope_inputs(rope_cache, cfg.mrope_section)
        if cfg.qk_norm_rows:
            q = ops.qk_row_norm_kv_write(q, k, v, rope_pos, rope_cache, cfg.rotary_dim, k_cache, v_cache, batch.slot_mapping, batch.positions,
                                         self.q_norm, self.k_norm, cfg.rms_norm_eps, cfg.num_attention_heads * self.dqk,
                                         cfg.num_key_value_heads * self.dqk, cfg.attn_query_temp, cfg.attn_query_temp_every,
                                         self._group_sums(q, k))
        else:
            q = ops.qk_norm_rope_kv_write(q, k, v, rope_pos, rope_cache, cfg.rotary_dim, k_cache, v_cache,
                                          batch.slot_mapping, k_scale, v_scale, self.q_norm, self.k_norm,
                                          cfg.rms_norm_eps, self.norm_plus_one, rotate=self.kv_rotate, norm_dim=self.dqk)
        if self.selector is not None:
            from ..kv.sparse_select import attend_selected
            self.selector.on_write(self.layer_idx, k_cache, batch, k_scale)
            out = attend_selected(ops.paged_attention, self.selector, self.layer_idx, q, k_cache, v_cache, batch, self.scale,
                                  k_scale, v_scale, self.window)
        else:
            if (self.o.kind == "fp8_block" and not self.gated and head_gate is None and self.o.bias is None and not self.kv_rotate
                    and (self.lora is None or batch.adapter_rows is None) and self.plain):
                a = ops.paged_attention_fp8_out(q, k_cache, v_cache, batch, self.scale, k_scale, v_scale, self.window)
                if a is not None:
                    return a                  # decode step: rows already quantised for the output projection
            out = ops.paged_attention(q, k_cache, v_cache, batch, self.scale, k_scale, v_scale, self.window, self.chunk, self.sinks,
                                      self.softcap, self.distance)
        if self.kv_rotate:
            out = ops.head_rotate(out)        # sum_j p_j (H v_j) = H o, and H is its own inverse
        if head_gate is not None:
            out = ops.head_gate(out, head_gate)
        out = out.reshape(T, nq)
        if self.gated:
            gate = qkv[:, nq + 2 * nkv:]
            if ops.on_gpu(out) and out.dtype == torch.bfloat16 and nq % 8 == 0 and gate.stride(0) % 8 == 0 and gate.data_ptr() % 16 == 0:
                out = ops.cuda_ops().sigmoid_gate_mul(out, gate)          # one kernel, in place
            else:
                out = (out.float() * torch.sigmoid(gate.float())).to(out.dtype)
        return out

    def _group_sums(self, q: torch.Tensor, k: torch.Tensor) -> Optional[torch.Tensor]:
        """Sums of squares ``[T, 2]`` of all ranks' queries and keys (norms over whole projections whose heads are sharded)."""
        if self.pctx.tp_size == 1:
            return None
        sums = torch.stack([q.float().square().sum((1, 2)), k.float().square().sum((1, 2)) / self.kv_rep], 1)
        return self.pctx.all_reduce(sums.contiguous())
