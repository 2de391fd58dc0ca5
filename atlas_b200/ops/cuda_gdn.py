"""Binding of the Gated-DeltaNet kernels (``csrc/gdn.cu``)."""
from __future__ import annotations

import ctypes as C
from typing import List, Optional

import torch

from . import cuda as K

_vp, _ll, _i = C.c_void_p, C.c_longlong, C.c_int
_bound = False
USE_CHUNKED = True          # tests switch this off to compare the two kernels
CHUNK_MIN_ROWS = 32


def _lib():
    global _bound
    lib = K.lib()
    if not _bound:
        lib.atlas_gdn_conv.argtypes = [_vp, _ll, _vp, _i, _i, _vp, _vp, _vp, _vp, _vp, _vp, _ll, _i, _vp]
        lib.atlas_gdn_conv_state.argtypes = [_vp, _ll, _i, _i, _vp, _vp, _vp, _vp, _vp, _vp, _vp, _i, _i, _vp]
        lib.atlas_gdn_recurrent.argtypes = [_vp, _ll, _vp, _ll, _vp, _ll, _vp, _vp, _vp, _vp, _ll, _vp, _vp, _vp, _vp, _vp,
                                            _vp, _i, _i, _i, _i, _i, _i, _i, _vp]
        lib.atlas_gdn_chunked.argtypes = [_vp, _ll, _vp, _ll, _vp, _ll, _vp, _vp, _vp, _vp, _ll, _vp, _vp, _vp, _vp, _vp, _i,
                                          _i, _i, _i, _i, _i, _i, _vp]
        _bound = True
    return lib


class _Meta:
    """Device-side per-step sequence metadata shared by all GDN layers of one forward pass."""

    def __init__(self, qlens: List[int], slots: List[int], has_state: List[bool], device, snapshot_plan=None,
                 limit: Optional[List[int]] = None):
        B = len(qlens)
        qsl = [0]
        seq_of = []
        for i, n in enumerate(qlens):
            qsl.append(qsl[-1] + n)
            seq_of.extend([i] * n)
        snaps = max((len(v) for v in (snapshot_plan or {}).values()), default=0)
        rows = [0] * (B * max(1, snaps))
        dsts = [0] * (B * max(1, snaps))
        for i, lst in (snapshot_plan or {}).items():
            for s, (r, d) in enumerate(lst):
                rows[i * snaps + s], dsts[i * snaps + s] = r, d
        ints = torch.tensor(qsl + seq_of + slots + rows + dsts + (limit or []), dtype=torch.int32).pin_memory()
        dev = ints.to(device, non_blocking=True)
        o = 0
        self.qsl = dev[o:o + B + 1]; o += B + 1
        self.seq_of = dev[o:o + len(seq_of)]; o += len(seq_of)
        self.slots = dev[o:o + B]; o += B
        self.snap_rows = dev[o:o + len(rows)]; o += len(rows)
        self.snap_slots = dev[o:o + len(dsts)]; o += len(dsts)
        self.limit = dev[o:o + B] if limit is not None else None
        self.has = torch.tensor([1 if h else 0 for h in has_state], dtype=torch.uint8).pin_memory().to(device, non_blocking=True)
        self.B, self.T, self.snaps = B, len(seq_of), snaps
        self.longest = max(qlens, default=0)
        # every sequence brings exactly one row and no row limit or snapshot applies (decode)
        self.one_row = int(limit is None and self.snaps == 0 and all(n == 1 for n in qlens))
        # the chunked (64-token, tensor-core) kernel takes prefill-sized steps (a snapshot row just ends a chunk early)
        self.chunk_ok = limit is None and max(qlens, default=0) >= CHUNK_MIN_ROWS


    @classmethod
    def decode(cls, qsl: torch.Tensor, slots: torch.Tensor, live: torch.Tensor) -> "_Meta":
        """Metadata of a decode step whose slots live in fixed device buffers (CUDA graphs): one row per sequence."""
        self = cls.__new__(cls)
        n = slots.shape[0]
        self.qsl, self.slots, self.has, self.limit = qsl, slots, live, None
        self.seq_of = torch.arange(n, dtype=torch.int32, device=slots.device)
        self.snap_rows = self.snap_slots = torch.zeros(1, dtype=torch.int32, device=slots.device)
        self.B, self.T, self.snaps, self.chunk_ok, self.one_row, self.longest = n, n, 0, False, 1, 1
        return self


def _run(layer, mixed, a, b, meta: _Meta, state, commit: bool):
    lib, st = _lib(), K._stream()
    K._dev(mixed)
    T, Cc = mixed.shape
    y = torch.empty(T, Cc, dtype=torch.bfloat16, device=mixed.device)
    out = torch.empty(T, layer.hv * layer.dv, dtype=torch.bfloat16, device=mixed.device)
    conv, h = state["conv"], state["h"]
    assert conv.dtype == torch.bfloat16 and h.dtype == torch.float32 and conv.is_contiguous() and h.is_contiguous()
    cw = layer.conv_w if layer.conv_w.dtype == torch.bfloat16 else layer.conv_w.bfloat16()
    K._check(lib.atlas_gdn_conv(mixed.data_ptr(), mixed.stride(0), cw.data_ptr(), Cc, layer.W, conv.data_ptr(),
                                meta.seq_of.data_ptr(), meta.qsl.data_ptr(), meta.slots.data_ptr(), meta.has.data_ptr(),
                                y.data_ptr(), Cc, T, st), "gdn_conv")
    rc = 1
    if USE_CHUNKED and meta.chunk_ok and commit and layer.dk == 128 and layer.dv == 128:
        rc = lib.atlas_gdn_chunked(y.data_ptr(), Cc, a.data_ptr(), a.stride(0), b.data_ptr(), b.stride(0),
                                   layer.A_log.data_ptr(), layer.dt_bias.data_ptr(), h.data_ptr(), out.data_ptr(),
                                   layer.hv * layer.dv, meta.qsl.data_ptr(), meta.slots.data_ptr(), meta.has.data_ptr(),
                                   meta.snap_rows.data_ptr(), meta.snap_slots.data_ptr(), meta.snaps, meta.B, layer.hk,
                                   layer.hv, layer.dk, layer.dv, 1, st)
        if rc != 1:
            K._check(rc, "gdn_chunked")
    if rc == 1:
      K._check(lib.atlas_gdn_recurrent(y.data_ptr(), Cc, a.data_ptr(), a.stride(0), b.data_ptr(), b.stride(0),
                                       layer.A_log.data_ptr(), layer.dt_bias.data_ptr(), h.data_ptr(), out.data_ptr(),
                                       layer.hv * layer.dv, meta.qsl.data_ptr(), meta.slots.data_ptr(), meta.has.data_ptr(),
                                       K._ptr(meta.limit), meta.snap_rows.data_ptr(), meta.snap_slots.data_ptr(), meta.snaps,
                                       meta.B, layer.hk, layer.hv, layer.dk, layer.dv, 1 if commit else 0, st), "gdn_recurrent")
    if commit:
        K._check(lib.atlas_gdn_conv_state(mixed.data_ptr(), mixed.stride(0), Cc, layer.W, conv.data_ptr(), meta.qsl.data_ptr(),
                                          meta.slots.data_ptr(), meta.has.data_ptr(), K._ptr(meta.limit),
                                          meta.snap_rows.data_ptr(), meta.snap_slots.data_ptr(), meta.snaps, meta.B, st),
                 "gdn_conv_state")
    return out


def gdn_forward(layer, mixed, a, b, batch, state, commit):
    meta = getattr(batch, "_gdn_meta", None)
    if meta is None:
        meta = _Meta(batch.query_lens_host, batch.state_slots_host, batch.has_state_host, mixed.device, batch.snapshot_plan)
        batch._gdn_meta = meta
    o = _run(layer, mixed, a, b, meta, state, commit)
    return o.view(mixed.shape[0], layer.hv, layer.dv)


def gdn_commit(layer, mixed, a, b, qlens, slots, has_state, state, num_accepted_rows):
    meta = _Meta(qlens, slots, has_state, mixed.device, None, limit=list(num_accepted_rows))
    _run(layer, mixed, a, b, meta, state, True)


# ----------------------------------------------------------------------------- relu^2 (csrc/elementwise.cu)
def _relu2_lib():
    lib = K.lib()
    lib.atlas_relu2.argtypes = [_vp, _ll, _vp, _ll, _i, _i, _vp]
    return lib


def relu_squared(x):
    x2 = x.reshape(-1, x.shape[-1])
    if x2.stride(1) != 1 or x2.stride(0) % 8 or x2.data_ptr() % 16:
        x2 = x2.contiguous()
    out = torch.empty(x2.shape, dtype=x.dtype, device=x.device)
    K._dev(x2)
    K._check(_relu2_lib().atlas_relu2(x2.data_ptr(), x2.stride(0), out.data_ptr(), out.stride(0), x2.shape[0], x2.shape[1],
                                  K._stream()), "relu2")
    return out.view(x.shape)
