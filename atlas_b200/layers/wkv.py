"""WKV time mixing (RWKV-style linear attention with data-dependent decay) on a per-sequence recurrent state slot.

Per token, with ``h'`` the previous token's input (zeros before the first), ``H`` heads of ``D`` channels::

    m_s    = h + (h' - h) * mu_s                           s in r, k, v, g, w
    r, k, v = W_r m_r, W_k m_k, W_v m_v                     [H, D] each
    w      = exp(-exp(W_w2 tanh(W_w1 m_w) + w0))            decay per head and key channel
    o      = (S + diag(u) k v^T)^T r                        the current token enters with the bonus u
    S      = diag(w) S + k v^T                              fp32 state [D key, D value]
    out    = W_o( o / rms(o per head) * norm * silu(W_g m_g) )

State of a sequence: ``shift [hidden]`` (the previous token's input) and ``h [H, D value, D key]``.  Slots, snapshots and the
write-on-accept protocol are those of the other recurrent mixers.  Tensor parallelism is head-parallel.
"""
from __future__ import annotations

from typing import List, Optional

import torch

from .. import ops
from ..config import ModelConfig
from ..ops import Act, LinearWeight, reference as ref
from .common import ParallelCtx, make_weight, randn_weight, shard_cols, shard_rows

MIXES = ("r", "k", "v", "g", "w")          # order of the token-shift mixes


class WKVMixer:
    def __init__(self, cfg: ModelConfig, layer_idx: int, pctx: ParallelCtx, quant_kind: str):
        self.cfg, self.layer_idx, self.pctx, self.quant_kind = cfg, layer_idx, pctx, quant_kind
        assert cfg.wkv_num_heads % pctx.tp_size == 0, "WKV heads must divide by tp"
        self.h, self.d = cfg.wkv_num_heads // pctx.tp_size, cfg.wkv_head_dim
        self.inner = self.h * self.d
        self.mu: Optional[torch.Tensor] = None                # [5, hidden] fp32, order MIXES
        self.r: Optional[LinearWeight] = None
        self.k: Optional[LinearWeight] = None
        self.v: Optional[LinearWeight] = None
        self.g: Optional[LinearWeight] = None
        self.w1: Optional[LinearWeight] = None                # [rank, hidden]
        self.w2: Optional[LinearWeight] = None                # [H * D, rank]
        self.o: Optional[LinearWeight] = None
        self.w0 = self.u = self.norm_w = None                 # fp32 [H * D], [H, D], [H * D]
        self._pending = None

    # ------------------------------------------------------------------ weights
    def load(self, mu: List[torch.Tensor], r, k, v, g, w1, w2, w0, u, norm_w, o, device) -> None:
        """Full (unsharded) tensors; ``mu`` in the order of ``MIXES``."""
        tp, rk = self.pctx.tp_size, self.pctx.tp_rank
        f32 = lambda t: t.to(device=device, dtype=torch.float32).contiguous()
        self.mu = f32(torch.stack([m.reshape(-1).float() for m in mu]))
        mk = lambda w: make_weight(shard_rows(w, rk, tp).contiguous(), self.quant_kind)
        self.r, self.k, self.v, self.g = mk(r), mk(k), mk(v), mk(g)
        # the decay's low-rank pair is small and its output is exponentiated twice: it stays in the model dtype
        self.w1, self.w2 = make_weight(w1.contiguous(), "dense"), make_weight(shard_rows(w2, rk, tp).contiguous(), "dense")
        self.w0 = f32(shard_rows(w0.reshape(-1, 1), rk, tp).reshape(-1))
        self.u = f32(shard_rows(u.reshape(self.h * tp, self.d), rk, tp))
        self.norm_w = f32(shard_rows(norm_w.reshape(-1, 1), rk, tp).reshape(-1))
        self.o = make_weight(shard_cols(o, rk, tp).contiguous(), self.quant_kind)

    def init_random(self, gen, std, dtype, device) -> None:
        H, D, W = self.cfg.wkv_num_heads, self.d, self.cfg.hidden_size
        n, rank = H * D, max(16, W // 64)
        rnd = lambda a, b: randn_weight(gen, a, b, std, dtype, device)
        mu = [torch.rand(W, generator=gen, device=gen.device) for _ in MIXES]
        self.load(mu, rnd(n, W), rnd(n, W), rnd(n, W), rnd(n, W), rnd(rank, W), rnd(n, rank),
                  torch.linspace(-6.0, -1.0, n), torch.rand(n, generator=gen, device=gen.device), torch.ones(n), rnd(W, n), device)

    # ------------------------------------------------------------------ state
    def alloc_state(self, num_slots: int, device, act_dtype) -> dict:
        return {"shift": torch.zeros(num_slots, self.cfg.hidden_size, dtype=act_dtype, device=device),
                "h": torch.zeros(num_slots, self.h, self.d, self.d, dtype=torch.float32, device=device)}

    # ------------------------------------------------------------------ forward
    def forward(self, act: Act, batch, state: dict) -> torch.Tensor:
        x = act.plain()
        if ops.on_gpu(x):
            m = ops.cuda_ops().token_shift_mix(x, self.mu, batch, state["shift"])
        else:
            m = self._mix_ref(x, batch.query_lens_host, batch.state_slots_host, batch.has_state_host, state)
        r, k, v, g = (ops.linear(m[i], w) for i, w in enumerate((self.r, self.k, self.v, self.g)))
        raw = ops.linear(ops.tanh_(ops.linear(m[4], self.w1)), self.w2)
        if batch.spec_verify:
            self._pending = (x.clone(), k, v, raw, list(batch.query_lens_host), list(batch.state_slots_host),
                             list(batch.has_state_host))
        if ops.on_gpu(x):
            o = ops.cuda_ops().wkv_forward(self, x, r, k, v, raw, batch, state, commit=not batch.spec_verify)
        else:
            o = self._scan_ref(x, r, k, v, raw, batch.query_lens_host, batch.state_slots_host, batch.has_state_host, state,
                               commit=not batch.spec_verify, snapshot_plan=batch.snapshot_plan)
        y = ops.group_norm_gate(o, g, self.norm_w, self.d, self.cfg.rms_norm_eps, gate_first=False)
        return self.pctx.row_parallel_linear(y, self.o)

    def _mix_ref(self, x, qlens, slots, has_state, state) -> torch.Tensor:
        prev = torch.zeros_like(x)
        t0 = 0
        for n, slot, live in zip(qlens, slots, has_state):
            prev[t0 + 1:t0 + n] = x[t0:t0 + n - 1]
            if live:
                prev[t0] = state["shift"][slot]
            t0 += n
        return ref.token_shift_mix(x, prev, self.mu)

    def _scan_ref(self, x, r, k, v, raw, qlens: List[int], slots: List[int], has_state: List[bool], state: dict, commit: bool,
                  limit: Optional[List[int]] = None, snapshot_plan: Optional[dict] = None) -> torch.Tensor:
        out = torch.zeros(x.shape[0], self.inner, dtype=x.dtype, device=x.device)
        heads = lambda t: t.float().view(-1, self.h, self.d)
        decay = heads(torch.exp(-torch.exp(raw.float() + self.w0)))
        r = torch.zeros_like(k) if r is None else r
        t0 = 0
        for i, (n, slot) in enumerate(zip(qlens, slots)):
            use = n if limit is None else limit[i]
            base, t0 = t0, t0 + n
            if use == 0:
                continue
            h = state["h"][slot].clone() if has_state[i] else torch.zeros_like(state["h"][slot])
            snap_at = {a: d for a, d in (snapshot_plan or {}).get(i, []) if 0 < a <= use}
            a = 0
            for b in sorted(set(snap_at) | {use}):
                rows = slice(base + a, base + b)
                o, h = ref.wkv_scan(heads(r[rows]), heads(k[rows]), heads(v[rows]), decay[rows], self.u, h)
                out[rows] = o.reshape(b - a, self.inner).to(x.dtype)
                if b in snap_at:
                    state["h"][snap_at[b]] = h
                    state["shift"][snap_at[b]] = x[base + b - 1]
                a = b
            if commit:
                state["h"][slot] = h
                state["shift"][slot] = x[base + use - 1]
        return out

    def commit(self, num_accepted_rows: List[int], state: dict) -> None:
        """Fold the first ``num_accepted_rows[i]`` stashed rows of each sequence into its state (write-on-accept)."""
        if self._pending is None:
            return
        x, k, v, raw, qlens, slots, has_state = self._pending
        self._pending = None
        if ops.on_gpu(x):
            ops.cuda_ops().wkv_commit(self, x, k, v, raw, qlens, slots, has_state, state, num_accepted_rows)
        else:
            self._scan_ref(x, None, k, v, raw, qlens, slots, has_state, state, commit=True, limit=num_accepted_rows)
