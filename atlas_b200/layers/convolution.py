"""Short causal convolution added to a sublayer's input, on a per-sequence state slot.

Per channel: ``u_t = h_t + sum_j w[:, j] h_(t - taps + 1 + j)``, zeros ahead of the sequence.  State of a sequence: its last ``taps - 1``
inputs, ``[width, taps - 1]`` in the activations' dtype.  Slots, snapshots and the write-on-accept protocol are those of the recurrent
mixers; any layer can own one, whatever its mixer (see ``models/decoder.py::recurrent_of``).
"""
from __future__ import annotations

from typing import List, Optional

import torch

from .. import ops
from ..ops import reference as ref
from .common import randn_weight


class InputConvolution:
    def __init__(self, width: int, taps: int):
        if taps < 1:
            raise ValueError("a convolution has at least one tap")
        self.width, self.W = width, taps
        self.w: Optional[torch.Tensor] = None                 # [width, taps]
        self._pending = None

    # ------------------------------------------------------------------ weights
    def load(self, w: torch.Tensor) -> None:
        assert w.shape == (self.width, self.W)
        self.w = w.contiguous()

    def init_random(self, gen, dtype, device) -> None:
        self.load(randn_weight(gen, self.width, self.W, 0.3, dtype, device))

    # ------------------------------------------------------------------ state
    def alloc_state(self, num_slots: int, device, act_dtype) -> dict:
        return {"inputs": torch.zeros(num_slots, self.width, self.W - 1, dtype=act_dtype, device=device)}

    # ------------------------------------------------------------------ forward
    def forward(self, h: torch.Tensor, batch, state: dict) -> torch.Tensor:
        if batch.spec_verify:
            self._pending = (h, list(batch.query_lens_host), list(batch.state_slots_host), list(batch.has_state_host))
        if ops.on_gpu(h):
            return ops.cuda_ops().input_conv(self, h, batch, state, commit=not batch.spec_verify)
        return self._ref(h, batch.query_lens_host, batch.state_slots_host, batch.has_state_host, state, commit=not batch.spec_verify,
                         snapshot_plan=batch.snapshot_plan)

    def _ref(self, h, qlens: List[int], slots: List[int], has_state: List[bool], state: dict, commit: bool, limit: Optional[List[int]] = None,
             snapshot_plan: Optional[dict] = None) -> torch.Tensor:
        out = torch.zeros_like(h)
        t0 = 0
        for i, (n, slot) in enumerate(zip(qlens, slots)):
            use = n if limit is None else limit[i]
            base, t0 = t0, t0 + n
            if use == 0:
                continue
            win = state["inputs"][slot].clone() if has_state[i] else torch.zeros_like(state["inputs"][slot])
            snap_at = {a: d for a, d in (snapshot_plan or {}).get(i, []) if 0 < a <= use}
            a = 0
            for b in sorted(set(snap_at) | {use}):
                rows = h[base + a:base + b]
                y, win = ref.causal_conv1d(rows.float(), win, self.w, None, activation=False)
                out[base + a:base + b] = (rows.float() + y).to(h.dtype)
                if b in snap_at:
                    state["inputs"][snap_at[b]] = win
                a = b
            if commit:
                state["inputs"][slot] = win
        return out

    def commit(self, num_accepted_rows: List[int], state: dict) -> None:
        """Fold the first ``num_accepted_rows[i]`` stashed rows of each sequence into its state (write-on-accept)."""
        if self._pending is None:
            return
        h, qlens, slots, has_state = self._pending
        self._pending = None
        if ops.on_gpu(h):
            ops.cuda_ops().input_conv_commit(self, h, qlens, slots, has_state, state, num_accepted_rows)
        else:
            self._ref(h, qlens, slots, has_state, state, commit=True, limit=num_accepted_rows)
