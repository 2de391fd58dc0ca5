"""mLSTM mixer (the matrix memory of xLSTM) on a per-sequence recurrent state slot.

Per token, with ``H`` heads of ``D`` key and ``V`` value channels, all gate arithmetic in fp32::

    [q | k | v | g | i | f] = in_proj(h)                    q, k [H, D], v, g [H, V], raw gates i, f [H]
    i = cap * tanh((i + b_i) / cap)                         log input gate
    f = logsigmoid(cap * tanh((f + b_f) / cap))             log forget gate
    m' = max(f + m, i)                                      running maximum, 0 before the first token
    S = exp(f + m - m') S + exp(i - m') v k^T               [V, D];  n likewise with k alone;  m = m'
    o = S q / (max(|n . q|, exp(-m)) + 1e-6)                q scaled by D^-1/2
    out = W_o( o / rms(o per head) * norm * sigmoid(g) )

State of a sequence: ``h [H, V + 1, D]`` fp32, whose last row is ``n`` (the memory of a value channel that is always one), and
``m [H]`` fp32.  Slots, snapshots and the write-on-accept protocol are those of the other recurrent mixers.  Tensor parallelism
is head-parallel.
"""
from __future__ import annotations

from typing import List, Optional

import torch

from .. import ops
from ..config import ModelConfig
from ..ops import Act, LinearWeight, reference as ref
from .common import ParallelCtx, TailLinear, make_weight, randn_weight, shard_cols, shard_rows


class MLSTMMixer:
    def __init__(self, cfg: ModelConfig, layer_idx: int, pctx: ParallelCtx, quant_kind: str):
        self.cfg, self.layer_idx, self.pctx, self.quant_kind = cfg, layer_idx, pctx, quant_kind
        assert cfg.mlstm_num_heads % pctx.tp_size == 0, "mLSTM heads must divide by tp"
        self.h, self.d, self.v = cfg.mlstm_num_heads // pctx.tp_size, cfg.mlstm_head_dim, cfg.mlstm_value_dim
        self.nk, self.nv = self.h * self.d, self.h * self.v
        self.cap, self.scale = cfg.mlstm_gate_cap, self.d ** -0.5
        self.in_proj: Optional[TailLinear] = None             # [q | k | v | g] in the activations' dtype, [i | f] in fp32
        self.gate_bias: Optional[torch.Tensor] = None         # fp32 [2 H]: input gates, forget gates
        self.norm_w: Optional[torch.Tensor] = None            # fp32 [H * V]
        self.o: Optional[LinearWeight] = None
        self._pending = None

    # ------------------------------------------------------------------ weights
    def load(self, q, k, v, g, i, i_bias, f, f_bias, norm_w, o, device) -> None:
        """Full (unsharded) tensors."""
        tp, r = self.pctx.tp_size, self.pctx.tp_rank
        cut = lambda w: shard_rows(w, r, tp)
        flat = lambda t: shard_rows(t.reshape(-1, 1), r, tp).reshape(-1).to(device=device, dtype=torch.float32)
        self.in_proj = TailLinear(torch.cat([cut(w) for w in (q, k, v, g)], 0), torch.cat([cut(i), cut(f)], 0), self.quant_kind)
        self.gate_bias = torch.cat([flat(i_bias), flat(f_bias)]).contiguous()
        self.norm_w = flat(norm_w).contiguous()
        self.o = make_weight(shard_cols(o, r, tp).contiguous(), self.quant_kind)

    def init_random(self, gen, std, dtype, device) -> None:
        H, W = self.cfg.mlstm_num_heads, self.cfg.hidden_size
        rnd = lambda n: randn_weight(gen, n, W, std, dtype, device)
        nk, nv = H * self.d, H * self.v
        # forget gates open over a range of spans, input gates around one
        self.load(rnd(nk), rnd(nk), rnd(nv), rnd(nv), rnd(H), torch.zeros(H), rnd(H), torch.linspace(3.0, 6.0, H), torch.ones(nv),
                  randn_weight(gen, W, nv, std, dtype, device), device)

    # ------------------------------------------------------------------ state
    def alloc_state(self, num_slots: int, device, act_dtype) -> dict:
        return {"h": torch.zeros(num_slots, self.h, self.v + 1, self.d, dtype=torch.float32, device=device),
                "m": torch.zeros(num_slots, self.h, dtype=torch.float32, device=device)}

    # ------------------------------------------------------------------ forward
    def forward(self, act: Act, batch, state: dict) -> torch.Tensor:
        main, raw = self.in_proj(act)
        q, k, v, g = main.split([self.nk, self.nk, self.nv, self.nv], -1)
        if batch.spec_verify:
            self._pending = (k, v, raw, list(batch.query_lens_host), list(batch.state_slots_host), list(batch.has_state_host))
        if ops.on_gpu(main):
            num, den = ops.cuda_ops().mlstm_forward(self, q, k, v, raw, batch, state, commit=not batch.spec_verify)
        else:
            num, den = self._scan_ref(q, k, v, raw, batch.query_lens_host, batch.state_slots_host, batch.has_state_host, state,
                                      commit=not batch.spec_verify, snapshot_plan=batch.snapshot_plan)
        y = ops.group_norm_gate(num, g, self.norm_w, self.v, self.cfg.rms_norm_eps, gate_first=False, gate="sigmoid", den=den)
        return self.pctx.row_parallel_linear(y, self.o)

    def _scan_ref(self, q, k, v, raw, qlens: List[int], slots: List[int], has_state: List[bool], state: dict, commit: bool,
                  limit: Optional[List[int]] = None, snapshot_plan: Optional[dict] = None):
        T = k.shape[0]
        num = torch.zeros(T, self.nv, dtype=k.dtype, device=k.device)
        den = torch.ones(T, self.h, dtype=torch.float32, device=k.device)
        heads = lambda t, d: t.float().reshape(-1, self.h, d)
        q = torch.zeros_like(k) if q is None else q
        t0 = 0
        for i, (n, slot) in enumerate(zip(qlens, slots)):
            use = n if limit is None else limit[i]
            base, t0 = t0, t0 + n
            if use == 0:
                continue
            h, m = ((state[s][slot].clone() if has_state[i] else torch.zeros_like(state[s][slot])) for s in ("h", "m"))
            snap_at = {a: d for a, d in (snapshot_plan or {}).get(i, []) if 0 < a <= use}
            a = 0
            for b in sorted(set(snap_at) | {use}):
                rows = slice(base + a, base + b)
                la, lb, ms = ref.mlstm_gates(raw[rows], self.gate_bias, self.cap, m)
                o, dots, h = ref.mlstm_scan(heads(q[rows], self.d) * self.scale, heads(k[rows], self.d), heads(v[rows], self.v), la, lb, h)
                m = ms[-1]
                num[rows] = o.reshape(b - a, self.nv).to(k.dtype)
                den[rows] = torch.maximum(dots.abs(), torch.exp(-ms)) + ref.MLSTM_EPS
                for name, t in (("h", h), ("m", m)) if b in snap_at else ():
                    state[name][snap_at[b]] = t
                a = b
            if commit:
                state["h"][slot], state["m"][slot] = h, m
        return num, den

    def commit(self, num_accepted_rows: List[int], state: dict) -> None:
        """Fold the first ``num_accepted_rows[i]`` stashed rows of each sequence into its state (write-on-accept)."""
        if self._pending is None:
            return
        k, v, raw, qlens, slots, has_state = self._pending
        self._pending = None
        if ops.on_gpu(k):
            ops.cuda_ops().mlstm_commit(self, k, v, raw, qlens, slots, has_state, state, num_accepted_rows)
        else:
            self._scan_ref(None, k, v, raw, qlens, slots, has_state, state, commit=True, limit=num_accepted_rows)
