"""Differential attention over the paged KV cache.

Every head holds two maps: attentions of their own, with their own queries and keys, over the same values.  Per token, ``H`` heads on
``G`` key / value heads::

    [q | k | v | g] = in_proj(h)               q [H, 2, dim], k [G, 2, dim], v [G, vdim], g [H, vdim]
    q, k = rotate(rmsnorm(.) * weight)         per head and map, one weight for all of them
    a_m = softmax(q_m . k_m * scale) v         m = 1, 2
    o = (1 - c) * rms(a_1 - lam * a_2)         over the head's vdim numbers;  lam = exp(lq1 . lk1) - exp(lq2 . lk2) + c
    out = W_o( o * sigmoid(g) )

A cached key holds both maps' keys side by side, ``[k_1 | k_2]``, and a value exists once.  The two maps of a head are two query rows,
``[q_1 | 0]`` and ``[0 | q_2]``, of the same key / value head, so that every attention kernel of the package (paged decode, tensor-core
prefill, fp32; windows, sinks and the others) runs them as ``2 H`` query heads on ``G`` key / value heads.  Keys and values are
zero-padded to the cache width.

The checkpoint's rotary columns come in pairs ``(2i, 2i + 1)``; the loader reorders those rows to the half-split convention of the
rotary tables on the query and the key side alike, which leaves the scores unchanged.  Tensor parallelism is head-parallel.
"""
from __future__ import annotations

import math
from typing import Optional, Tuple

import torch

from .. import ops
from ..config import ModelConfig
from ..ops import Act, LinearWeight
from .common import ParallelCtx, make_weight, randn_weight, shard_cols, shard_rows
from .mla import deinterleave_rows


class DifferentialAttention:
    lora = None
    takes_adapters = False
    plain = False                # the cache keeps the model's own dtype

    def __init__(self, cfg: ModelConfig, layer_idx: int, pctx: ParallelCtx, quant_kind: str):
        self.cfg, self.layer_idx, self.pctx, self.quant_kind = cfg, layer_idx, pctx, quant_kind
        tp = pctx.tp_size
        assert cfg.num_attention_heads % tp == 0, "query heads must divide by tp"
        self.heads = cfg.num_attention_heads // tp
        self.hq = 2 * self.heads                              # query rows per token, as the attention kernels count them
        self.hkv = max(1, cfg.num_key_value_heads // tp)
        self.kv_rep = max(1, tp // cfg.num_key_value_heads)   # ranks sharing one kv head
        self.dqk, self.dv = cfg.head_dim, cfg.v_head_dim or cfg.head_dim
        self.d = cfg.attn_cache_width
        assert 2 * self.dqk <= self.d and self.dv <= self.d
        self.scale = cfg.attn_scale or self.dqk ** -0.5
        self.window = cfg.sliding_window
        self.gated = cfg.attn_output_gate
        self.rest = 1.0 - cfg.attn_diff
        self.lam = 0.0
        self.in_proj: Optional[LinearWeight] = None           # rows [q | k | v | g]
        self.q_norm: Optional[torch.Tensor] = None            # fp32 [dim]
        self.k_norm: Optional[torch.Tensor] = None
        self.o: Optional[LinearWeight] = None

    # ------------------------------------------------------------------ weights
    def load(self, q, k, v, o, gate, q_norm, k_norm, lams, rope_interleaved: bool = True) -> None:
        """Full tensors: ``q`` / ``k`` rows per head ``[map 1 | map 2]``, norm weights of one map, ``lams`` = the four vectors lq1, lk1,
        lq2, lk2 (each ``[dim]``)."""
        tp, r = self.pctx.tp_size, self.pctx.tp_rank
        n = self.cfg.rotary_dim
        if rope_interleaved and n:
            order = torch.cat([deinterleave_rows(torch.arange(n).view(n, 1), n)[:, 0], torch.arange(n, self.dqk)]).to(q.device)
            turn = lambda w: w.reshape(-1, self.dqk, w.shape[-1])[:, order].reshape(w.shape)
            q, k, q_norm, k_norm = turn(q), turn(k), q_norm[order.to(q_norm.device)], k_norm[order.to(k_norm.device)]
        head = (r // self.kv_rep) * self.hkv
        kv = lambda w, per: w[head * per:(head + self.hkv) * per] if tp > 1 else w
        parts = [shard_rows(q, r, tp), kv(k, 2 * self.dqk), kv(v, self.dv)] + ([shard_rows(gate, r, tp)] if self.gated else [])
        self.in_proj = make_weight(torch.cat(parts, 0).contiguous(), self.quant_kind)
        self.o = make_weight(shard_cols(o, r, tp).contiguous(), self.quant_kind)
        self.q_norm, self.k_norm = (w.to(device=q.device, dtype=torch.float32).contiguous() for w in (q_norm, k_norm))
        lq1, lk1, lq2, lk2 = (t.double().cpu() for t in lams)
        self.lam = math.exp((lq1 * lk1).sum().item()) - math.exp((lq2 * lk2).sum().item()) + self.cfg.attn_diff

    def init_random(self, gen, std, dtype, device) -> None:
        cfg = self.cfg
        h, H, G = cfg.hidden_size, cfg.num_attention_heads, cfg.num_key_value_heads
        rnd = lambda n, k: randn_weight(gen, n, k, std, dtype, device)
        ones = torch.ones(self.dqk, device=device)
        self.load(rnd(2 * H * self.dqk, h), rnd(2 * G * self.dqk, h), rnd(G * self.dv, h), rnd(h, H * self.dv),
                  rnd(H * self.dv, h) if self.gated else None, ones, ones, [randn_weight(gen, 1, self.dqk, 0.1, torch.float32, device)[0] for _ in range(4)])

    # ------------------------------------------------------------------ forward
    def forward(self, act: Act, batch, kv, rope_cache: torch.Tensor) -> torch.Tensor:
        return self.pctx.row_parallel_linear(self.mix(act, batch, kv, rope_cache), self.o)

    def mix(self, act: Act, batch, kv: Tuple[torch.Tensor, torch.Tensor, float, float], rope_cache: torch.Tensor) -> torch.Tensor:
        """Everything before the output projection: this rank's heads ``[T, heads * vdim]``."""
        k_cache, v_cache = kv[0], kv[1]
        x = ops.linear(act, self.in_proj)
        T, nq, nk, nv = x.shape[0], self.hq * self.dqk, 2 * self.hkv * self.dqk, self.hkv * self.dv
        q, k, v = x[:, :nq], x[:, nq:nq + nk], x[:, nq + nk:nq + nk + nv]
        rope_pos, rope_cache = batch.rope_inputs(rope_cache, self.cfg.mrope_section)
        q = ops.map_norm_kv_write(q.view(T, self.heads, 2, self.dqk), k.view(T, self.hkv, 2, self.dqk), v.view(T, self.hkv, self.dv), rope_pos,
                                  rope_cache, self.cfg.rotary_dim, k_cache, v_cache, batch.slot_mapping, self.q_norm, self.k_norm,
                                  self.cfg.rms_norm_eps)
        a = ops.paged_attention(q, k_cache, v_cache, batch, self.scale, sliding_window=self.window)
        return ops.map_difference(a, self.dv, self.lam, self.rest, self.cfg.rms_norm_eps, x[:, nq + nk + nv:] if self.gated else None)
