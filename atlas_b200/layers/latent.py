"""Latent attention over a paged cache of latents.

Projections per token, ``H`` heads, latent rank ``R``, head sizes ``nope`` / ``rope`` / ``v``::

    [q | ckv] = in_proj(h)                                  q [H, nope + rope], ckv [R + rope]
    c = rmsnorm(ckv[:R]),  r = rotate(ckv[R:])              the cache row of the token: [c | r], shared by all heads
    score = (q_nope . W_uk c' + rotate(q_rope) . r') * scale
    out = W_o( softmax(score) W_uv c' )

Where :mod:`layers.mla` caches every head's expanded key and value, this block caches the ``R + rope`` numbers that the design
needs.  Attention takes one of two forms, chosen per sequence of a step by the number of its rows:

* absorbed (decode and short portions): ``W_uk`` is folded into the query, ``W_uv`` into the output; all heads then read the same
  cache row, keys ``R + rope`` wide and values the row's first ``R`` numbers.
* expanded (long portions): the visible rows of the cache go through ``[W_uk; W_uv]`` once, in one matrix product, into
  per-head keys and values on scratch pages, and the attention kernels of the GQA blocks read those.

The checkpoint's rotary columns come in pairs ``(2i, 2i + 1)``; the loader reorders those rows to the half-split convention of
the rotary tables on the query and the key side alike, which leaves the scores unchanged.  ``R`` and ``rope`` are zero-padded to
multiples of :data:`LATENT_ALIGN`.  Tensor parallelism is head-parallel (every rank holds the whole latent).
"""
from __future__ import annotations

from typing import Optional, Tuple

import torch
import torch.nn.functional as F

from .. import ops
from ..config import ModelConfig
from ..ops import Act, LinearWeight, reference as ref
from .common import ParallelCtx, TailLinear, make_weight, randn_weight, shard_cols, shard_rows
from .mla import deinterleave_rows

LATENT_ALIGN = 16                # widths of the two parts of a cache row are multiples of this


def _pad_to(n: int, m: int) -> int:
    return (n + m - 1) // m * m


class LatentAttention:
    lora = None
    takes_adapters = False
    gated = False
    plain = False                # the cache keeps the model's own dtype

    def __init__(self, cfg: ModelConfig, layer_idx: int, pctx: ParallelCtx, quant_kind: str):
        self.cfg, self.layer_idx, self.pctx, self.quant_kind = cfg, layer_idx, pctx, quant_kind
        assert cfg.num_attention_heads % pctx.tp_size == 0, "heads must divide by tp"
        self.hq, self.hkv = cfg.num_attention_heads // pctx.tp_size, 1
        self.nope, self.rope, self.vd, self.rank = cfg.qk_nope_head_dim, cfg.qk_rope_head_dim, cfg.v_head_dim, cfg.kv_lora_rank
        self.rotary = cfg.rotary_dim
        assert self.rotary <= self.rope
        self.rp, self.ep = _pad_to(self.rank, LATENT_ALIGN), _pad_to(self.rope, LATENT_ALIGN)
        self.width = self.rp + self.ep                        # numbers of a cache row
        self.d = self.width
        self.dx = cfg.attn_cache_width                        # padded head width of the expanded form
        self.scale = cfg.attn_scale or (self.nope + self.rope) ** -0.5
        self.window = cfg.sliding_window
        self.in_proj: Optional[TailLinear] = None             # q rows per head [rope | nope]; tail [R | rope] in fp32
        self.c_norm: Optional[torch.Tensor] = None            # fp32 [R]
        self.uk: Optional[torch.Tensor] = None                # [H, rp, nope]: latent component of a head's unrotated query
        self.uv: Optional[torch.Tensor] = None                # [H, v, rp]
        self.expand: Optional[torch.Tensor] = None            # [H * (nope + v), rp]: unrotated keys and values of every head
        self.o: Optional[LinearWeight] = None

    # ------------------------------------------------------------------ weights
    def load(self, q, dkv, c_norm, uk, uv, o, rope_interleaved: bool = True) -> None:
        """Full tensors: ``q`` rows per head ``[nope | rope]``, ``dkv`` rows ``[R | rope]``, ``uk`` / ``uv`` rows per head."""
        tp, r = self.pctx.tp_size, self.pctx.tp_rank
        H = self.cfg.num_attention_heads
        mine = slice(r * self.hq, (r + 1) * self.hq)
        # only the first ``rotary`` of a head's rope rows turn
        turn = (lambda w: torch.cat([deinterleave_rows(w[:self.rotary], self.rotary), w[self.rotary:]])) if rope_interleaved else (lambda w: w)
        qh = q.view(H, self.nope + self.rope, -1)[mine]
        qh = torch.cat([torch.stack([turn(h) for h in qh[:, self.nope:]]), qh[:, :self.nope]], 1)
        down = torch.cat([dkv[:self.rank], turn(dkv[self.rank:])], 0)
        self.in_proj = TailLinear(qh.reshape(-1, q.shape[-1]).contiguous(), down.contiguous(), self.quant_kind)
        self.c_norm = c_norm.float().to(q.device).contiguous()
        ukh = F.pad(uk.view(H, self.nope, self.rank)[mine], (0, self.rp - self.rank))
        uvh = F.pad(uv.view(H, self.vd, self.rank)[mine], (0, self.rp - self.rank))
        self.uk, self.uv = ukh.transpose(1, 2).contiguous(), uvh.contiguous()
        self.expand = torch.cat([ukh, uvh], 1).reshape(-1, self.rp).contiguous()
        self.o = make_weight(shard_cols(o, r, tp).contiguous(), self.quant_kind)

    def init_random(self, gen, std, dtype, device) -> None:
        h, H = self.cfg.hidden_size, self.cfg.num_attention_heads
        rnd = lambda n, k: randn_weight(gen, n, k, std, dtype, device)
        self.load(rnd(H * (self.nope + self.rope), h), rnd(self.rank + self.rope, h), torch.ones(self.rank), rnd(H * self.nope, self.rank),
                  rnd(H * self.vd, self.rank), rnd(h, H * self.vd))

    # ------------------------------------------------------------------ cache
    @property
    def kv_elements(self) -> int:
        """Cached numbers per token."""
        return self.width

    def alloc_kv(self, num_blocks: int, block_size: int, dtype, device) -> Tuple[torch.Tensor, torch.Tensor]:
        """Latent pages ``[num_blocks, block_size, 1, width]`` and an empty second pool (values are a part of the keys)."""
        from ..utils import guards
        shape = (num_blocks, block_size, 1, self.width)
        if torch.device(device).type == "cuda":
            k = guards.zeros("kv.latent", shape, dtype, device)
        else:
            k = torch.zeros(shape, dtype=dtype, device=device)
        return k, torch.empty(num_blocks, block_size, 1, 0, dtype=dtype, device=device)

    # ------------------------------------------------------------------ forward
    def forward(self, act: Act, batch, kv, rope_cache: torch.Tensor) -> torch.Tensor:
        return self.pctx.row_parallel_linear(self.mix(act, batch, kv, rope_cache), self.o)

    def mix(self, act: Act, batch, kv, rope_cache: torch.Tensor) -> torch.Tensor:
        """This rank's heads' attention output ``[T, hq * v]``."""
        q, ckv = self.in_proj(act)
        if ops.on_gpu(q):
            return ops.cuda_ops().latent_attention(self, q, ckv, batch, kv[0], rope_cache)
        return self._mix_ref(q, ckv, batch, kv[0], rope_cache)

    def _mix_ref(self, q, ckv, batch, cache, rope_cache) -> torch.Tensor:
        T, H, eps = q.shape[0], self.hq, self.cfg.rms_norm_eps
        row, q_rope = ref.latent_rows(ckv, q.view(T, H, -1)[:, :, :self.rope], self.c_norm, self.rank, self.rp, self.ep, batch.positions,
                                      rope_cache, self.rotary, eps)
        ok = batch.slot_mapping >= 0
        slots, bs = batch.slot_mapping[ok].long(), cache.shape[1]
        cache[slots // bs, slots % bs, 0] = row[ok].to(cache.dtype)
        qa = torch.einsum("thd,hrd->thr", q.view(T, H, -1)[:, :, self.rope:].float(), self.uk.float())
        o = ref.latent_attention(torch.cat([qa, q_rope], -1), cache, self.rp, batch.block_tables, batch.seq_lens, batch.query_start_loc,
                                 self.scale, self.window)
        return torch.einsum("thr,hvr->thv", o, self.uv.float()).reshape(T, H * self.vd).to(q.dtype)
