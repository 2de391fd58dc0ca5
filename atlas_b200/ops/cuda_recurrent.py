"""Binding of the residual-stream, recurrence and 32-bit attention kernels (``csrc/streams.cu``, ``csrc/recurrent.cu``,
``csrc/conv1d.cu``, ``csrc/mlstm.cu``, ``csrc/rglru.cu``, ``csrc/row_norm_kv.cu``, ``csrc/attention_f32.cu``).  Activations are bf16 or fp32; every entry point takes the choice as its ``f32`` flag."""
from __future__ import annotations

import ctypes as C
from typing import List, Optional

import torch

from . import cuda as K
from .cuda_gdn import _Meta

_vp, _ll, _i, _f = C.c_void_p, C.c_longlong, C.c_int, C.c_float
_bound = False


class _Rglru(C.Structure):
    """Mirror of ``AtlasRglru`` (csrc/host_api.h)."""
    _fields_ = [("x", _vp), ("ldx", _ll), ("u", _vp), ("ldu", _ll), ("zr", _vp), ("zi", _vp), ("z_row", _ll), ("z_block", _ll), ("y", _vp),
                ("ldy", _ll), ("conv_w", _vp), ("conv_b", _vp), ("conv_state", _vp), ("tiles", _vp), ("gate_bias", _vp), ("lam", _vp), ("h", _vp),
                ("P", _vp), ("S", _vp), ("endP", _vp), ("endS", _vp), ("out", _vp), ("ldo", _ll), ("seq_of", _vp), ("qsl", _vp), ("slots", _vp),
                ("has", _vp), ("limit", _vp), ("snap_rows", _vp), ("snap_slots", _vp), ("status", _vp), ("snaps", _i), ("rows", _i), ("C", _i),
                ("n", _i), ("taps", _i), ("commit", _i), ("one_row", _i)]


class _NormedExtras(C.Structure):
    """Mirror of ``AtlasNormedExtras`` (csrc/host_api.h)."""
    _fields_ = [("gate", _vp), ("ldg", _ll), ("b", _vp), ("out_b", _vp), ("hist", _vp), ("hist_ld", _ll), ("factors", _vp), ("hist_index", _i)]


def _lib():
    global _bound
    lib = K.lib()
    if not _bound:
        lib.atlas_hyper_norm.argtypes = [_vp, _i, _i, _i, _vp, _ll, _vp, _ll, _vp, _vp, _vp, _vp, _vp, _vp, _vp, _ll, _i, _i, _f, _f, _i, _vp]
        lib.atlas_token_shift_mix.argtypes = [_vp, _ll, _vp, _vp, _vp, _vp, _vp, _vp, _vp, _i, _i, _i, _vp]
        lib.atlas_gated_unit.argtypes = [_vp, _ll, _i, _i, _vp, _ll, _f, _f, _f, _i, _i, _vp]
        lib.atlas_rglru_tc.argtypes = [C.POINTER(_Rglru), _vp]
        lib.atlas_rglru_scan.argtypes = [C.POINTER(_Rglru), _i, _vp]
        lib.atlas_row_norm_kv_write.argtypes = [_vp, _ll, _vp, _ll, _vp, _ll] + [_vp] * 9 + [_i] * 8 + [_f, _f, _i, _i, _vp]
        lib.atlas_tanh.argtypes = [_vp, _ll, _i, _vp]
        lib.atlas_mamba2_scan.argtypes = [_vp, _ll, _vp, _ll, _vp, _vp, _vp, _f, _vp, _vp, _ll, _vp, _vp, _vp, _vp, _vp, _vp] + [_i] * 9 + [_vp]
        lib.atlas_wkv_scan.argtypes = [_vp, _ll, _vp, _ll, _vp, _ll, _vp, _ll, _vp, _vp, _vp, _vp, _ll, _vp, _ll, _vp, _i, _vp, _vp, _vp,
                                       _vp, _vp, _vp] + [_i] * 7 + [_vp]
        lib.atlas_group_norm_gate.argtypes = [_vp, _ll, _vp, _ll, _vp, _vp, _ll, _i, _i, _i, _f, _i, _i, _vp, _i, _vp]
        lib.atlas_add_normed.argtypes = [_vp, _ll, _vp, _ll, _vp, _vp, _i, _vp, _ll, _vp, _vp, _vp, _vp, _ll] + [_i] * 5 + [_f, _f, _i, C.POINTER(_NormedExtras), _vp]
        lib.atlas_gelu_embedding.argtypes = [_vp, _ll, _vp, _ll, _vp, _i, _i, _i, _vp, _ll, _i, _i, _vp]
        lib.atlas_conv1d_add.argtypes = [_vp, _ll, _vp, _i, _i, _vp, _vp, _vp, _vp, _vp, _vp, _ll, _i, _i, _i, _vp]
        lib.atlas_head_gate.argtypes = [_vp, _ll, _vp, _ll, _i, _i, _i, _i, _vp]
        lib.atlas_mlstm_gates.argtypes = [_vp, _ll, _vp, _f] + [_vp] * 10 + [_i] * 4 + [_vp]
        lib.atlas_mlstm_scan.argtypes = [_vp, _ll, _vp, _ll, _vp, _ll, _vp, _vp, _vp, _f, _vp, _vp, _ll] + [_vp] * 7 + [_i] * 8 + [_vp]
        lib.atlas_mlstm_chunk.argtypes = [_vp, _ll, _vp, _ll, _vp, _ll, _vp, _vp, _vp, _f, _vp, _vp, _ll] + [_vp] * 6 + [_i] * 6 + [_vp]
        lib.atlas_conv1d_bias_silu.argtypes = [_vp, _ll, _vp, _vp, _i, _i, _vp, _vp, _vp, _vp, _vp, _vp, _ll, _i, _i, _i, _vp]
        lib.atlas_conv1d_state.argtypes = [_vp, _ll, _i, _i, _vp, _vp, _vp, _vp, _vp, _vp, _vp, _i, _i, _i, _vp]
        lib.atlas_rope_kv_write_f32.argtypes = [_vp, _ll, _vp, _ll, _vp, _ll, _vp, _vp, _vp, _vp, _vp, _i, _i, _i, _i, _i, _i, _vp, _vp, _i, _i, _f, _vp]
        lib.atlas_attn_f32.argtypes = [_vp, _ll, _vp, _ll, _vp, _vp, _vp, _i, _vp, _vp, _i, _i, _f, _i, _i, _i, _i, _i, _i, _vp, _f, _vp, _i, _vp]
        _bound = True
    return lib


def _f32(t: torch.Tensor) -> int:
    if t.dtype not in (torch.bfloat16, torch.float32):
        raise K.KernelError(f"activations must be bf16 or fp32, not {t.dtype}")
    assert t.stride(-1) == 1
    return 1 if t.dtype == torch.float32 else 0


def step_meta(batch, device) -> _Meta:
    """Device-side sequence metadata of the step, shared by all recurrent layers of one forward pass."""
    meta = getattr(batch, "_gdn_meta", None)
    if meta is None:
        meta = _Meta(batch.query_lens_host, batch.state_slots_host, batch.has_state_host, device, batch.snapshot_plan)
        batch._gdn_meta = meta
    return meta


# ----------------------------------------------------------------------------- residual streams
def hyper_norm(streams: Optional[torch.Tensor], delta, read, norm_w, eps: float, write: bool):
    y, y2, conn = delta.y, delta.y2, delta.conn
    T, W = y.shape
    S = read.shape[0]
    K._dev(y)
    f32 = _f32(y)
    if conn is None:
        streams = torch.empty(T, S, W, dtype=torch.float32, device=y.device)
    assert streams.dtype == torch.float32 and streams.shape == (T, S, W) and streams.is_contiguous()
    assert read.dtype == norm_w.dtype == torch.float32 and norm_w.numel() == W
    if y2 is not None:
        assert y2.dtype == y.dtype and y2.shape == y.shape and delta.w1.dtype == delta.w2.dtype == torch.float32
    out = torch.empty(T, W, dtype=y.dtype, device=y.device)
    K._check(_lib().atlas_hyper_norm(streams.data_ptr(), T, S, W, y.data_ptr(), y.stride(0), K._ptr(y2), y2.stride(0) if y2 is not None else 0,
                                     K._ptr(delta.w1), K._ptr(delta.w2), K._ptr(conn.mix if conn else None),
                                     K._ptr(conn.write if conn else None), read.data_ptr(), norm_w.data_ptr(), out.data_ptr(), W,
                                     0 if conn else 1, 1 if write else 0, float(delta.scale), float(eps), f32, K._stream()), "hyper_norm")
    return out, streams


def token_shift_mix(x, mu, batch, shift):
    T, W = x.shape
    K._dev(x)
    f32 = _f32(x)
    assert mu.shape == (5, W) and mu.dtype == torch.float32 and shift.dtype == x.dtype and shift.is_contiguous()
    meta = step_meta(batch, x.device)
    out = torch.empty(5, T, W, dtype=x.dtype, device=x.device)
    K._check(_lib().atlas_token_shift_mix(x.data_ptr(), x.stride(0), mu.data_ptr(), shift.data_ptr(), meta.seq_of.data_ptr(),
                                          meta.qsl.data_ptr(), meta.slots.data_ptr(), meta.has.data_ptr(), out.data_ptr(), T, W, f32,
                                          K._stream()), "token_shift_mix")
    return out


def gated_unit(gate_up, unit, paired: bool = False):
    T, I2 = gate_up.shape
    K._dev(gate_up)
    f32 = _f32(gate_up)
    y = torch.empty(T, I2 // 2, dtype=gate_up.dtype, device=gate_up.device)
    K._check(_lib().atlas_gated_unit(gate_up.data_ptr(), gate_up.stride(0), T, I2 // 2, y.data_ptr(), y.stride(0),
                                     *(float(v) for v in unit), 1 if paired else 0, f32, K._stream()), "gated_unit")
    return y


def tanh_(x):
    K._dev(x)
    assert x.is_contiguous()
    K._check(_lib().atlas_tanh(x.data_ptr(), x.numel(), _f32(x), K._stream()), "tanh")
    return x


# ----------------------------------------------------------------------------- recurrences
def group_norm_gate(y, z, w, group: int, eps: float, gate_first: bool, gate: str = "silu", den=None):
    T, n = y.shape
    K._dev(y)
    f32 = _f32(y)
    assert z.dtype == y.dtype and z.shape == y.shape and z.stride(1) == 1 and n % group == 0
    assert den is None or (den.dtype == torch.float32 and den.is_contiguous() and den.numel() == T * (n // group))
    wf = K._float_cached(w)
    out = torch.empty(T, n, dtype=y.dtype, device=y.device)
    K._check(_lib().atlas_group_norm_gate(y.data_ptr(), y.stride(0), z.data_ptr(), z.stride(0), wf.data_ptr(), out.data_ptr(), n, T,
                                          n // group, group, float(eps), 1 if gate_first else 0, 1 if gate == "sigmoid" else 0, K._ptr(den),
                                          f32, K._stream()), "group_norm_gate")
    return out


def _mamba2_run(layer, xbc, dt, meta: _Meta, state, commit: bool):
    lib, st = _lib(), K._stream()
    K._dev(xbc)
    f32 = _f32(xbc)
    T, Cc = xbc.shape
    conv, h = state["conv"], state["h"]
    assert conv.dtype == xbc.dtype and h.dtype == torch.float32 and conv.is_contiguous() and h.is_contiguous()
    assert dt.dtype == xbc.dtype and dt.stride(1) == 1 and layer.conv_w.dtype == xbc.dtype and layer.conv_w.is_contiguous()
    assert layer.conv_b is None or layer.conv_b.dtype == xbc.dtype
    y = torch.empty(T, Cc, dtype=xbc.dtype, device=xbc.device)
    out = torch.empty(T, layer.d_inner, dtype=xbc.dtype, device=xbc.device)
    K._check(lib.atlas_conv1d_bias_silu(xbc.data_ptr(), xbc.stride(0), layer.conv_w.data_ptr(), K._ptr(layer.conv_b), Cc, layer.W,
                                        conv.data_ptr(), meta.seq_of.data_ptr(), meta.qsl.data_ptr(), meta.slots.data_ptr(),
                                        meta.has.data_ptr(), y.data_ptr(), Cc, T, 1, f32, st), "conv1d")
    K._check(lib.atlas_mamba2_scan(y.data_ptr(), Cc, dt.data_ptr(), dt.stride(0), layer.A_log.data_ptr(), layer.D.data_ptr(),
                                   layer.dt_bias.data_ptr(), float(layer.cfg.mamba_dt_min), h.data_ptr(), out.data_ptr(),
                                   layer.d_inner, meta.qsl.data_ptr(), meta.slots.data_ptr(), meta.has.data_ptr(),
                                   K._ptr(meta.limit), meta.snap_rows.data_ptr(), meta.snap_slots.data_ptr(), meta.snaps, meta.B,
                                   layer.h, layer.p, layer.n, layer.g, 1 if commit else 0, meta.one_row, f32, st), "mamba2_scan")
    if commit:
        K._check(lib.atlas_conv1d_state(xbc.data_ptr(), xbc.stride(0), Cc, layer.W, conv.data_ptr(), meta.qsl.data_ptr(),
                                        meta.slots.data_ptr(), meta.has.data_ptr(), K._ptr(meta.limit),
                                        meta.snap_rows.data_ptr(), meta.snap_slots.data_ptr(), meta.snaps, meta.B, f32, st),
                 "conv1d_state")
    return out


def mamba2_forward(layer, xbc, dt, batch, state, commit):
    return _mamba2_run(layer, xbc, dt, step_meta(batch, xbc.device), state, commit)


def mamba2_commit(layer, xbc, dt, qlens, slots, has_state, state, num_accepted_rows):
    meta = _Meta(qlens, slots, has_state, xbc.device, None, limit=list(num_accepted_rows))
    _mamba2_run(layer, xbc, dt, meta, state, True)


def _wkv_run(layer, x, r, k, v, raw, meta: _Meta, state, commit: bool):
    K._dev(x)
    f32 = _f32(x)
    shift, h = state["shift"], state["h"]
    for t in (k, v, raw) + ((r,) if r is not None else ()):
        assert t.dtype == x.dtype and t.stride(1) == 1
    assert shift.dtype == x.dtype and h.dtype == torch.float32 and shift.is_contiguous() and h.is_contiguous()
    out = torch.empty(x.shape[0], layer.inner, dtype=x.dtype, device=x.device) if r is not None else None
    K._check(_lib().atlas_wkv_scan(K._ptr(r), r.stride(0) if r is not None else 0, k.data_ptr(), k.stride(0), v.data_ptr(), v.stride(0),
                                   raw.data_ptr(), raw.stride(0), layer.w0.data_ptr(), layer.u.data_ptr(), h.data_ptr(), K._ptr(out),
                                   layer.inner, x.data_ptr(), x.stride(0), shift.data_ptr(), x.shape[1], meta.qsl.data_ptr(),
                                   meta.slots.data_ptr(), meta.has.data_ptr(), K._ptr(meta.limit), meta.snap_rows.data_ptr(),
                                   meta.snap_slots.data_ptr(), meta.snaps, meta.B, layer.h, layer.d, 1 if commit else 0, meta.one_row,
                                   f32, K._stream()), "wkv_scan")
    return out


def wkv_forward(layer, x, r, k, v, raw, batch, state, commit):
    return _wkv_run(layer, x, r, k, v, raw, step_meta(batch, x.device), state, commit)


def wkv_commit(layer, x, k, v, raw, qlens, slots, has_state, state, num_accepted_rows):
    meta = _Meta(qlens, slots, has_state, x.device, None, limit=list(num_accepted_rows))
    _wkv_run(layer, x, None, k, v, raw, meta, state, True)


MLSTM_CHUNKED = True         # tests switch this off to compare the two forms
MLSTM_CHUNK_MIN_ROWS = 16    # longest portion of a step from which the chunked kernel takes the step


def _mlstm_run(layer, q, k, v, raw, meta: _Meta, state, commit: bool):
    lib, st = _lib(), K._stream()
    K._dev(k)
    f32 = _f32(k)
    h, m = state["h"], state["m"]
    T, H, dev = k.shape[0], layer.h, k.device
    for t in (k, v) + ((q,) if q is not None else ()):
        assert t.dtype == k.dtype and t.stride(1) == 1
    assert raw.dtype == layer.gate_bias.dtype == torch.float32 and raw.stride(1) == 1
    assert h.dtype == m.dtype == torch.float32 and h.is_contiguous() and m.is_contiguous()
    la, lb, top = torch.empty(3, T, H, dtype=torch.float32, device=dev)
    seq = (meta.qsl.data_ptr(), meta.slots.data_ptr(), meta.has.data_ptr())
    snaps = (meta.snap_rows.data_ptr(), meta.snap_slots.data_ptr(), meta.snaps, meta.B)
    K._check(lib.atlas_mlstm_gates(raw.data_ptr(), raw.stride(0), layer.gate_bias.data_ptr(), float(layer.cap), m.data_ptr(), la.data_ptr(),
                                   lb.data_ptr(), top.data_ptr(), *seq, K._ptr(meta.limit), *snaps, H, 1 if commit else 0, st), "mlstm_gates")
    num = den = None
    if q is not None:
        num = torch.empty(T, layer.nv, dtype=k.dtype, device=dev)
        den = torch.empty(T, H, dtype=torch.float32, device=dev)
    rows = (K._ptr(q), q.stride(0) if q is not None else 0, k.data_ptr(), k.stride(0), v.data_ptr(), v.stride(0), la.data_ptr(), lb.data_ptr(),
            top.data_ptr(), float(layer.scale), h.data_ptr(), K._ptr(num), layer.nv, K._ptr(den)) + seq
    rc = 1
    if MLSTM_CHUNKED and not f32 and q is not None and meta.limit is None and meta.T >= MLSTM_CHUNK_MIN_ROWS and meta.longest >= MLSTM_CHUNK_MIN_ROWS:
        rc = lib.atlas_mlstm_chunk(*rows, *snaps, H, layer.v, layer.d, 1 if commit else 0, st)
        if rc != 1:
            K._check(rc, "mlstm_chunk")
    if rc == 1:
        K._check(lib.atlas_mlstm_scan(*rows, K._ptr(meta.limit), *snaps, H, layer.v, layer.d, 1 if commit else 0, meta.one_row, f32, st),
                 "mlstm_scan")
    return num, den


def mlstm_forward(layer, q, k, v, raw, batch, state, commit):
    return _mlstm_run(layer, q, k, v, raw, step_meta(batch, k.device), state, commit)


def mlstm_commit(layer, k, v, raw, qlens, slots, has_state, state, num_accepted_rows):
    meta = _Meta(qlens, slots, has_state, k.device, None, limit=list(num_accepted_rows))
    _mlstm_run(layer, None, k, v, raw, meta, state, True)


RGLRU_CHUNK = 32              # rows per chunk of the recurrence (kRgChunk in csrc/rglru.cu)
RGLRU_TENSOR_CORES = True     # tests switch this off to compare the two forms


def _rglru_run(layer, y, x, meta: _Meta, state, commit: bool):
    lib, st = _lib(), K._stream()
    dev = K._dev(x)
    f32 = _f32(x)
    conv, h = state["conv"], state["h"]
    T, Cc = x.shape
    assert conv.dtype == x.dtype and h.dtype == torch.float32 and conv.is_contiguous() and h.is_contiguous() and Cc == layer.c
    assert layer.conv_w.dtype == layer.conv_b.dtype == x.dtype and layer.gate_bias.dtype == layer.lam.dtype == torch.float32
    out = torch.empty(T, Cc, dtype=x.dtype, device=x.device) if y is not None else None
    a = _Rglru(x=x.data_ptr(), ldx=x.stride(0), conv_w=layer.conv_w.data_ptr(), conv_b=layer.conv_b.data_ptr(), conv_state=conv.data_ptr(),
               gate_bias=layer.gate_bias.data_ptr(), lam=layer.lam.data_ptr(), h=h.data_ptr(), seq_of=meta.seq_of.data_ptr(),
               qsl=meta.qsl.data_ptr(), slots=meta.slots.data_ptr(), has=meta.has.data_ptr(), limit=K._ptr(meta.limit),
               snap_rows=meta.snap_rows.data_ptr(), snap_slots=meta.snap_slots.data_ptr(), status=K._status_ptr[dev], snaps=meta.snaps, rows=T,
               C=Cc, n=layer.n, taps=layer.W, commit=1 if commit else 0)
    if y is not None:
        assert y.dtype == x.dtype and y.stride(1) == 1
        a.y, a.ldy, a.out, a.ldo = y.data_ptr(), y.stride(0), out.data_ptr(), Cc
    tc = RGLRU_TENSOR_CORES and layer.gate_tiles is not None
    a.one_row = 1 if tc and meta.one_row and y is not None else 0
    rc = 1
    if a.one_row:
        a.tiles = layer.gate_tiles.data_ptr()
        rc = lib.atlas_rglru_tc(C.byref(a), st)
        a.one_row = 1 if rc != 1 else 0
        if rc != 1:
            K._check(rc, "rglru_step")
    if rc == 1:
        rows, ends = torch.empty(2, T, Cc, dtype=torch.float32, device=x.device), torch.empty(2, -(-T // RGLRU_CHUNK), Cc, dtype=torch.float32, device=x.device)
        a.P, a.S, a.endP, a.endS = rows[0].data_ptr(), rows[1].data_ptr(), ends[0].data_ptr(), ends[1].data_ptr()
        if tc:
            a.tiles = layer.gate_tiles.data_ptr()
            rc = lib.atlas_rglru_tc(C.byref(a), st)
            if rc != 1:
                K._check(rc, "rglru_tc")
    if rc == 1:
        u = torch.empty(T, Cc, dtype=x.dtype, device=x.device)
        K._check(lib.atlas_conv1d_bias_silu(x.data_ptr(), x.stride(0), layer.conv_w.data_ptr(), layer.conv_b.data_ptr(), Cc, layer.W, conv.data_ptr(),
                                            meta.seq_of.data_ptr(), meta.qsl.data_ptr(), meta.slots.data_ptr(), meta.has.data_ptr(), u.data_ptr(),
                                            Cc, T, 0, f32, st), "conv1d")
        # gate sums [2, blocks, T, n] in fp32
        z = torch.matmul(u.float().view(T, layer.blocks, layer.n).transpose(0, 1), layer.gates.float().transpose(2, 3))
        a.u, a.ldu, a.zr, a.zi, a.z_row, a.z_block = u.data_ptr(), Cc, z[0].data_ptr(), z[1].data_ptr(), layer.n, T * layer.n
        K._check(lib.atlas_rglru_scan(C.byref(a), f32, st), "rglru_scan")
    if commit:
        K._check(lib.atlas_conv1d_state(x.data_ptr(), x.stride(0), Cc, layer.W, conv.data_ptr(), meta.qsl.data_ptr(), meta.slots.data_ptr(),
                                        meta.has.data_ptr(), K._ptr(meta.limit), meta.snap_rows.data_ptr(), meta.snap_slots.data_ptr(), meta.snaps,
                                        meta.B, f32, st), "conv1d_state")
    return out


def rglru_forward(layer, y, x, batch, state, commit):
    return _rglru_run(layer, y, x, step_meta(batch, x.device), state, commit)


def rglru_commit(layer, x, qlens, slots, has_state, state, num_accepted_rows):
    meta = _Meta(qlens, slots, has_state, x.device, None, limit=list(num_accepted_rows))
    _rglru_run(layer, None, x, meta, state, True)


# ----------------------------------------------------------------------------- sublayer outputs on an fp32 residual
def add_normed(stream: Optional[torch.Tensor], delta, eps: float, plus_one: bool, out_norm, write: bool, step=None, out_bias=None):
    rows = delta.y if hasattr(delta.y, "slot_of") else None
    y = rows.y if rows is not None else delta.y
    W = y.shape[1]
    T = rows.w.shape[0] if rows is not None else y.shape[0]
    K._dev(y)
    f32 = _f32(y)
    first = stream is None
    if first:
        assert delta.norm is None
        stream, write = torch.empty(T, W, dtype=torch.float32, device=y.device), True
    assert stream.dtype == torch.float32 and stream.shape == (T, W) and stream.is_contiguous()
    gate, depth = delta.gate, delta.depth
    extras = None
    if gate is not None or delta.bias is not None or out_bias is not None or depth is not None:
        extras = _NormedExtras(b=K._ptr(delta.bias), out_b=K._ptr(out_bias))
        if gate is not None:
            assert gate.dtype == y.dtype and gate.shape == (T, W) and gate.stride(1) == 1
            extras.gate, extras.ldg = gate.data_ptr(), gate.stride(0)
        if depth is not None:
            hist, fac = depth.history, depth.factors
            assert hist.dtype == torch.float32 and hist.is_contiguous() and hist.shape[1:] == (T, W) and 0 <= depth.index < hist.shape[0]
            assert fac is None or (fac.dtype == torch.float32 and fac.is_contiguous() and fac.numel() == depth.index + 1)
            extras.hist, extras.hist_ld, extras.factors, extras.hist_index = hist.data_ptr(), T * W, K._ptr(fac), depth.index
    assert (delta.bias is None or delta.norm is not None) and (out_bias is None or out_norm is not None)
    for w in (delta.norm, out_norm, step, delta.bias, out_bias):
        assert w is None or (w.dtype == torch.float32 and w.numel() == W and w.is_contiguous())
    if rows is not None:
        assert rows.slot_of.dtype == torch.int32 and rows.w.dtype == torch.float32 and rows.w.is_contiguous()
    extra = rows.extra if rows is not None else None
    if extra is not None:
        assert extra.dtype == y.dtype and extra.shape == (T, W) and extra.stride(1) == 1
    out = torch.empty(T, W, dtype=y.dtype, device=y.device)
    K._check(_lib().atlas_add_normed(stream.data_ptr(), W, y.data_ptr(), y.stride(0), K._ptr(rows.slot_of) if rows is not None else None,
                                     K._ptr(rows.w) if rows is not None else None, rows.w.shape[1] if rows is not None else 0,
                                     K._ptr(extra), extra.stride(0) if extra is not None else 0, K._ptr(delta.norm), K._ptr(out_norm),
                                     K._ptr(step), out.data_ptr(), W, T, W, 1 if plus_one else 0, 1 if write else 0, 1 if first else 0, float(eps),
                                     float(delta.scale), f32, C.byref(extras) if extras is not None else None, K._stream()), "add_normed")
    return out, stream


def gelu_embedding(z, table, ids, first: int, n: int):
    T, N = z.shape
    K._dev(z)
    assert table.dtype == z.dtype and table.is_contiguous() and ids.dtype == torch.int64 and ids.is_contiguous() and ids.numel() == T
    out = torch.empty(T, N, dtype=z.dtype, device=z.device)
    K._check(_lib().atlas_gelu_embedding(z.data_ptr(), z.stride(0), table.data_ptr(), table.shape[1], ids.data_ptr(), int(first), int(n), N,
                                         out.data_ptr(), N, T, _f32(z), K._stream()), "gelu_embedding")
    return out


# ----------------------------------------------------------------------------- convolution on a sublayer's input
def _input_conv_state(layer, h, meta: _Meta, win) -> None:
    K._check(_lib().atlas_conv1d_state(h.data_ptr(), h.stride(0), layer.width, layer.W, win.data_ptr(), meta.qsl.data_ptr(), meta.slots.data_ptr(),
                                       meta.has.data_ptr(), K._ptr(meta.limit), meta.snap_rows.data_ptr(), meta.snap_slots.data_ptr(), meta.snaps,
                                       meta.B, _f32(h), K._stream()), "conv1d_state")


def input_conv(layer, h, batch, state, commit: bool):
    meta, win = step_meta(batch, h.device), state["inputs"]
    T, W = h.shape
    K._dev(h)
    f32 = _f32(h)
    assert W == layer.width and win.dtype == h.dtype == layer.w.dtype and win.is_contiguous() and layer.w.is_contiguous()
    out = torch.empty(T, W, dtype=h.dtype, device=h.device)
    advance = commit and meta.one_row
    K._check(_lib().atlas_conv1d_add(h.data_ptr(), h.stride(0), layer.w.data_ptr(), W, layer.W, win.data_ptr(), meta.seq_of.data_ptr(),
                                     meta.qsl.data_ptr(), meta.slots.data_ptr(), meta.has.data_ptr(), out.data_ptr(), W, T, 1 if advance else 0, f32,
                                     K._stream()), "conv1d_add")
    if commit and not advance:
        _input_conv_state(layer, h, meta, win)
    return out


def input_conv_commit(layer, h, qlens, slots, has_state, state, num_accepted_rows):
    K._dev(h)
    _input_conv_state(layer, h, _Meta(qlens, slots, has_state, h.device, None, limit=list(num_accepted_rows)), state["inputs"])


def head_gate(x, g):
    T, H, D = x.shape
    K._dev(x)
    assert x.stride(2) == 1 and x.stride(1) == D and g.dtype == torch.float32 and g.shape == (T, H) and g.stride(1) == 1
    K._check(_lib().atlas_head_gate(x.data_ptr(), x.stride(0), g.data_ptr(), g.stride(0), T, H, D, _f32(x), K._stream()), "head_gate")
    return x


# ----------------------------------------------------------------------------- norm over all heads
def qk_row_norm_kv_write(q, k, v, positions, rope_cache, rotary_dim, k_cache, v_cache, slot_mapping, seq_positions, q_w, k_w, eps, nq, nk, temp,
                         temp_every, sums):
    T, Hq, D = q.shape
    Hkv = k.shape[1]
    K._dev(q)
    K._kv_layout_ok(k_cache, v_cache)
    f32 = _f32(q)
    assert k_cache.dtype == v_cache.dtype == q.dtype == k.dtype == v.dtype, "this cache holds the activations' dtype"
    assert q.stride(1) == k.stride(1) == v.stride(1) == D and positions.dtype == seq_positions.dtype == slot_mapping.dtype == torch.int32
    assert q_w.dtype == k_w.dtype == torch.float32 and q_w.numel() == Hq * D and k_w.numel() == Hkv * D and q_w.is_contiguous() and k_w.is_contiguous()
    assert sums is None or (sums.dtype == torch.float32 and sums.shape == (T, 2) and sums.is_contiguous())
    if K.checked.ENABLED:
        K.checked.kv_write(slot_mapping, positions, k_cache.shape[0], k_cache.shape[1], rope_cache.shape[0] if rotary_dim else 0)
    K._check(_lib().atlas_row_norm_kv_write(q.data_ptr(), q.stride(0), k.data_ptr(), k.stride(0), v.data_ptr(), v.stride(0), positions.data_ptr(),
                                            rope_cache.data_ptr(), seq_positions.data_ptr(), q_w.data_ptr(), k_w.data_ptr(), K._ptr(sums),
                                            k_cache.data_ptr(), v_cache.data_ptr(), slot_mapping.data_ptr(), T, Hq, Hkv, D, rotary_dim,
                                            k_cache.shape[1], int(nq), int(nk), float(eps), float(temp), int(temp_every), f32, K._stream()),
             "row_norm_kv_write")
    return q


# ----------------------------------------------------------------------------- 32-bit attention
def rope_kv_write_f32(q, k, v, positions, rope_cache, rotary_dim, k_cache, v_cache, slot_mapping, q_norm, k_norm, norm_dim, plus_one, eps):
    T, Hq, D = q.shape
    Hkv = k.shape[1]
    K._dev(q)
    assert q.stride(2) == 1 and q.stride(1) == k.stride(1) == v.stride(1) == D and k_cache.dtype == torch.float32
    assert positions.dtype == slot_mapping.dtype == torch.int32 and rope_cache.dtype == torch.float32
    assert q_norm is None or (q_norm.dtype == k_norm.dtype == torch.float32 and q_norm.numel() == k_norm.numel() == D)
    K._check(_lib().atlas_rope_kv_write_f32(q.data_ptr(), q.stride(0), k.data_ptr(), k.stride(0), v.data_ptr(), v.stride(0),
                                            positions.data_ptr(), rope_cache.data_ptr(), k_cache.data_ptr(), v_cache.data_ptr(),
                                            slot_mapping.data_ptr(), T, Hq, Hkv, D, rotary_dim, k_cache.shape[1], K._ptr(q_norm),
                                            K._ptr(k_norm), int(norm_dim), 1 if plus_one else 0, float(eps), K._stream()), "rope_kv_write_f32")
    return q


def attention_f32(q, k_cache, v_cache, batch, scale, window: int, chunk: int, sinks, softcap: float = 0.0, distance=None):
    T, Hq, D = q.shape
    K._dev(q)
    assert k_cache.dtype == torch.float32 and q.stride(2) == 1 and q.stride(1) == D
    out = torch.empty(T, Hq, D, dtype=q.dtype, device=q.device)
    bt = batch.block_tables
    K._check(_lib().atlas_attn_f32(q.data_ptr(), q.stride(0), out.data_ptr(), Hq * D, k_cache.data_ptr(), v_cache.data_ptr(),
                                   bt.data_ptr(), bt.stride(0), batch.seq_lens.data_ptr(), batch.query_start_loc.data_ptr(),
                                   batch.num_seqs, T, float(scale), Hq, k_cache.shape[2], D, k_cache.shape[1], window, chunk,
                                   K._ptr(sinks), softcap, K._ptr(distance), distance.shape[1] - 1 if distance is not None else 0, K._stream()), "attn_f32")
    return out
