"""RG-LRU mixer (the recurrent block of Griffin) on a per-sequence recurrent state slot.

Per token, ``W`` channels in ``blocks`` equal parts, everything behind the convolution in fp32::

    [y | x] = in_proj(h) + bias
    u   = causal_conv1d(x) + bias                            depth-wise, state = the last taps - 1 inputs
    r   = sigmoid(ra[b] u_b + ra_bias[b])                    one square matrix per block
    i   = sigmoid(ri[b] u_b + ri_bias[b])
    a   = exp(-8 r softplus(lam))
    S   = a S + sqrt(1 - a^2) i u                            [W] fp32, zero before the first token
    out = W_o( S * gelu_tanh(y) )

State of a sequence: ``conv [W, taps - 1]`` in the activations' dtype and ``h [W]`` fp32.  Slots, snapshots and the
write-on-accept protocol are those of the other recurrent mixers.  Tensor parallelism cuts between blocks.
"""
from __future__ import annotations

from typing import List, Optional

import torch
import torch.nn.functional as F

from .. import ops
from ..config import ModelConfig
from ..ops import Act, LinearWeight, reference as ref
from .common import ParallelCtx, make_weight, randn_weight, shard_cols, shard_rows

GATE_TILE_M, GATE_TILE_K = 128, 64            # a block's gate matrices are zero-padded to whole tiles


def gate_tiles(gates: torch.Tensor) -> torch.Tensor:
    """``[2, blocks, n, n]`` -> ``[blocks, Mt, Kt, 2, 128, 64]``: 128 x 64 tiles of both gates as the tensor cores read them from
    shared memory (the 16-byte pieces of row ``r`` permuted by ``r % 8``), so that a plain copy brings them in."""
    _, nb, n, _ = gates.shape
    p = F.pad(gates, (0, -n % GATE_TILE_K, 0, -n % GATE_TILE_M))
    p = p.view(2, nb, p.shape[2] // GATE_TILE_M, GATE_TILE_M, p.shape[3] // GATE_TILE_K, 8, 8).permute(1, 2, 4, 0, 3, 5, 6)
    rows, pieces = torch.arange(GATE_TILE_M, device=gates.device), torch.arange(8, device=gates.device)
    return p[..., rows[:, None], pieces[None, :] ^ (rows[:, None] & 7), :].flatten(-2).contiguous()


class RGLRUMixer:
    def __init__(self, cfg: ModelConfig, layer_idx: int, pctx: ParallelCtx, quant_kind: str):
        self.cfg, self.layer_idx, self.pctx, self.quant_kind = cfg, layer_idx, pctx, quant_kind
        assert cfg.rglru_blocks % pctx.tp_size == 0, "RG-LRU blocks must divide by tp"
        self.blocks = cfg.rglru_blocks // pctx.tp_size
        self.n = cfg.rglru_width // cfg.rglru_blocks          # channels of a block
        self.c = self.blocks * self.n                         # channels of this rank
        self.W = cfg.rglru_conv_kernel
        self.in_proj: Optional[LinearWeight] = None           # rows [y | x]
        self.o: Optional[LinearWeight] = None
        self.conv_w = self.conv_b = None                      # [c, taps], [c]
        self.gates: Optional[torch.Tensor] = None             # [2, blocks, n, n]: r, i
        self.gate_tiles: Optional[torch.Tensor] = None        # the same as operand tiles (bf16, GPU)
        self.gate_bias: Optional[torch.Tensor] = None         # fp32 [2, c]
        self.lam: Optional[torch.Tensor] = None               # fp32 [c]
        self._pending = None

    # ------------------------------------------------------------------ weights
    def load(self, y, y_bias, x, x_bias, conv_w, conv_b, ra, ra_bias, ri, ri_bias, lam, o) -> None:
        """Full (unsharded) tensors: ``ra`` / ``ri`` ``[blocks, n, n]`` as (out, in)."""
        tp, r = self.pctx.tp_size, self.pctx.tp_rank
        dev = y.device
        cut = lambda w: shard_rows(w, r, tp)
        f32 = lambda t: cut(t.reshape(self.cfg.rglru_width, 1))[:, 0].to(device=dev, dtype=torch.float32).contiguous()
        vec = lambda t: cut(t.reshape(-1, 1))[:, 0].to(device=dev, dtype=y.dtype)
        self.in_proj = make_weight(torch.cat([cut(y), cut(x)], 0).contiguous(), self.quant_kind, torch.cat([vec(y_bias), vec(x_bias)]).contiguous())
        self.conv_w, self.conv_b = cut(conv_w).to(device=dev, dtype=y.dtype).contiguous(), vec(conv_b).contiguous()
        self.gates = torch.stack([cut(ra), cut(ri)]).to(device=dev, dtype=y.dtype).contiguous()
        if y.is_cuda and y.dtype == torch.bfloat16:
            self.gate_tiles = gate_tiles(self.gates)
        self.gate_bias = torch.stack([f32(ra_bias), f32(ri_bias)]).contiguous()
        self.lam = f32(lam)
        self.o = make_weight(shard_cols(o, r, tp).contiguous(), self.quant_kind)

    def init_random(self, gen, std, dtype, device) -> None:
        C, nb, n, h = self.cfg.rglru_width, self.cfg.rglru_blocks, self.n, self.cfg.hidden_size
        rnd = lambda a, b: randn_weight(gen, a, b, std, dtype, device)
        square = lambda: randn_weight(gen, nb * n, n, n ** -0.5, dtype, device).view(nb, n, n)
        # decays between 0.9 and 0.999 for an open gate
        lam = torch.log(torch.expm1(-torch.log(torch.linspace(0.9, 0.999, C)) / 8.0))
        zero = torch.zeros(C, device=device)
        self.load(rnd(C, h), zero, rnd(C, h), zero, randn_weight(gen, C, self.W, 0.3, dtype, device), zero, square(), zero, square(), zero,
                  lam, rnd(h, C))

    # ------------------------------------------------------------------ state
    def alloc_state(self, num_slots: int, device, act_dtype) -> dict:
        return {"conv": torch.zeros(num_slots, self.c, self.W - 1, dtype=act_dtype, device=device),
                "h": torch.zeros(num_slots, self.c, dtype=torch.float32, device=device)}

    # ------------------------------------------------------------------ forward
    def forward(self, act: Act, batch, state: dict) -> torch.Tensor:
        yx = ops.linear(act, self.in_proj)
        y, x = yx[:, :self.c], yx[:, self.c:]
        if batch.spec_verify:
            self._pending = (x, list(batch.query_lens_host), list(batch.state_slots_host), list(batch.has_state_host))
        if ops.on_gpu(yx):
            out = ops.cuda_ops().rglru_forward(self, y, x, batch, state, commit=not batch.spec_verify)
        else:
            out = self._scan_ref(y, x, batch.query_lens_host, batch.state_slots_host, batch.has_state_host, state,
                                 commit=not batch.spec_verify, snapshot_plan=batch.snapshot_plan)
        return self.pctx.row_parallel_linear(out, self.o)

    def _scan_ref(self, y, x, qlens: List[int], slots: List[int], has_state: List[bool], state: dict, commit: bool,
                  limit: Optional[List[int]] = None, snapshot_plan: Optional[dict] = None) -> torch.Tensor:
        out = torch.zeros(x.shape[0], self.c, dtype=x.dtype, device=x.device)
        t0 = 0
        for i, (n, slot) in enumerate(zip(qlens, slots)):
            use = n if limit is None else limit[i]
            base, t0 = t0, t0 + n
            if use == 0:
                continue
            conv, h = ((state[s][slot].clone() if has_state[i] else torch.zeros_like(state[s][slot])) for s in ("conv", "h"))
            snap_at = {a: d for a, d in (snapshot_plan or {}).get(i, []) if 0 < a <= use}
            a = 0
            for b in sorted(set(snap_at) | {use}):
                rows = slice(base + a, base + b)
                u, conv = ref.causal_conv1d(x[rows], conv, self.conv_w, self.conv_b, activation=False)
                z = torch.einsum("tbk,gbnk->gtbn", u.float().view(b - a, self.blocks, self.n), self.gates.float()).flatten(2) + self.gate_bias[:, None]
                s = ref.linear_recurrence(*ref.rglru_gates(u, z[0], z[1], self.lam), h)
                h = s[-1]
                if y is not None:
                    out[rows] = (s * F.gelu(y[rows].float(), approximate="tanh")).to(x.dtype)
                for name, t in (("conv", conv), ("h", h)) if b in snap_at else ():
                    state[name][snap_at[b]] = t
                a = b
            if commit:
                state["conv"][slot], state["h"][slot] = conv, h
        return out

    def commit(self, num_accepted_rows: List[int], state: dict) -> None:
        """Fold the first ``num_accepted_rows[i]`` stashed rows of each sequence into its state (write-on-accept)."""
        if self._pending is None:
            return
        x, qlens, slots, has_state = self._pending
        self._pending = None
        if ops.on_gpu(x):
            ops.cuda_ops().rglru_commit(self, x, qlens, slots, has_state, state, num_accepted_rows)
        else:
            self._scan_ref(None, x, qlens, slots, has_state, state, commit=True, limit=num_accepted_rows)
