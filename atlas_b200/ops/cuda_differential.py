"""Binding of the differential attention kernels (``csrc/differential.cu``)."""
from __future__ import annotations

import ctypes as C

import torch

from . import cuda as K
from .cuda_recurrent import _f32

_vp, _ll, _i, _f = C.c_void_p, C.c_longlong, C.c_int, C.c_float
_bound = False


def _lib():
    global _bound
    lib = K.lib()
    if not _bound:
        lib.atlas_map_norm_kv_write.argtypes = [_vp, _ll, _vp, _ll, _vp, _ll] + [_vp] * 8 + [_i] * 8 + [_f, _i, _vp]
        lib.atlas_map_difference.argtypes = [_vp, _vp, _ll, _vp] + [_i] * 4 + [_f] * 3 + [_i, _vp]
        _bound = True
    return lib


def map_norm_kv_write(q, k, v, positions, rope_cache, rotary_dim, k_cache, v_cache, slot_mapping, q_norm_w, k_norm_w, eps):
    T, H, two, n = q.shape
    G, dv, D = k.shape[1], v.shape[2], k_cache.shape[3]
    K._dev(q)
    K._kv_layout_ok(k_cache, v_cache)
    f32 = _f32(q)
    assert two == k.shape[2] == 2 and k.shape[3] == n and k_cache.shape[2] == G
    assert k_cache.dtype == v_cache.dtype == q.dtype == k.dtype == v.dtype, "this cache holds the activations' dtype"
    for t, tail in ((q, (2 * n, n, 1)), (k, (2 * n, n, 1)), (v, (dv, 1))):
        assert t.stride()[1:] == tail or t.shape[1] == 1 and t.stride()[2:] == tail[1:]
    assert positions.dtype == slot_mapping.dtype == torch.int32 and rope_cache.dtype == torch.float32
    assert q_norm_w.dtype == k_norm_w.dtype == torch.float32 and q_norm_w.numel() == k_norm_w.numel() == n
    if K.checked.ENABLED:
        K.checked.kv_write(slot_mapping, positions, k_cache.shape[0], k_cache.shape[1], rope_cache.shape[0] if rotary_dim else 0)
    rows = torch.empty(T, 2 * H, D, dtype=q.dtype, device=q.device)
    K._check(_lib().atlas_map_norm_kv_write(q.data_ptr(), q.stride(0), k.data_ptr(), k.stride(0), v.data_ptr(), v.stride(0), rows.data_ptr(),
                                            positions.data_ptr(), rope_cache.data_ptr(), q_norm_w.data_ptr(), k_norm_w.data_ptr(), k_cache.data_ptr(),
                                            v_cache.data_ptr(), slot_mapping.data_ptr(), T, H, G, n, dv, D, int(rotary_dim), k_cache.shape[1],
                                            float(eps), f32, K._stream()), "map_norm_kv_write")
    return rows


def map_difference(a, dv, lam, rest, eps, gate):
    T, rows, D = a.shape
    H = rows // 2
    K._dev(a)
    assert a.is_contiguous()
    if gate is not None:
        assert gate.dtype == a.dtype and gate.shape == (T, H * dv) and gate.stride(1) == 1
    out = torch.empty(T, H * dv, dtype=a.dtype, device=a.device)
    K._check(_lib().atlas_map_difference(a.data_ptr(), K._ptr(gate), gate.stride(0) if gate is not None else 0, out.data_ptr(), T, H, D, int(dv),
                                         float(lam), float(rest), float(eps), _f32(a), K._stream()), "map_difference")
    return out
