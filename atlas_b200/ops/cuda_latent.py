"""Binding of the latent-attention kernels (``csrc/latent.cu``) and the choice of the form per sequence of a step."""
from __future__ import annotations

import ctypes as C
from types import SimpleNamespace
from typing import List, Optional

import torch

from . import checked, cuda as K

_vp, _ll, _i, _f = C.c_void_p, C.c_longlong, C.c_int, C.c_float
_bound = False
EXPAND_MIN_ROWS = 96          # portions of at least this many rows take the expanded form
_KEYS_PER_SPLIT = 64          # the least a split of the keys is given


def _lib():
    global _bound
    lib = K.lib()
    if not _bound:
        lib.atlas_latent_rows.argtypes = [_vp, _ll, _vp, _ll] + [_vp] * 8 + [_i] * 9 + [_f, _i, _vp]
        lib.atlas_head_gemm.argtypes = [_vp, _ll, _i, _vp, _vp, _ll, _i, _vp, _vp, _i, _i, _i, _i, _vp]
        lib.atlas_latent_attn.argtypes = [_vp] * 6 + [_i] + [_vp] * 5 + [_i] * 10 + [_f, _vp]
        lib.atlas_latent_attn_f32.argtypes = [_vp] * 4 + [_i] + [_vp] * 2 + [_i] * 7 + [_f, _vp]
        lib.atlas_latent_gather.argtypes = [_vp, _vp, _i, _vp, _vp, _vp, _i, _i, _i, _i, _vp, _vp]
        lib.atlas_latent_pages.argtypes = [_vp, _vp, _vp, _i, _vp, _vp, _vp] + [_i] * 9 + [_vp] * 3
        lib.atlas_latent_unpad.argtypes = [_vp, _vp, _i, _i, _i, _i, _vp, _vp]
        _bound = True
    return lib


def decode_splits(B: int, H: int, mt: int, visible: int, sms: int) -> int:
    """Key splits of the absorbed decode kernel: about one CTA per SM."""
    ctas = B * ((H + 16 * mt - 1) // (16 * mt))
    return max(1, min(sms // max(1, ctas), (visible + _KEYS_PER_SPLIT - 1) // _KEYS_PER_SPLIT, 32))


def row_tiles(layer) -> int:
    """16-row units per CTA: two where a token has more than sixteen heads (and the cache rows are not too wide)."""
    return 2 if layer.hq > 16 and layer.rp <= 512 and layer.width <= 576 else 1


def scratch_bytes(batch_sizes, layer, max_seq_len: int, sms: int):
    """Worst case of the split decode partials over the given batch sizes: (outputs, (max, sum) pairs) in bytes."""
    po = pml = 0
    visible = min(max_seq_len, layer.window or max_seq_len)
    for b in batch_sizes:
        s = decode_splits(b, layer.hq, row_tiles(layer), visible, sms)
        if s > 1:
            po, pml = max(po, b * layer.hq * s * layer.rp * 4), max(pml, b * layer.hq * s * 8)
    return po, pml


class _Plan:
    """Which sequences of a step take which form, shared by the step's latent layers of the same window and tiling."""

    def __init__(self, batch, window: int, H: int, mt: int, block_size: int, device):
        qlens, nd, B = batch.query_lens_host, batch.num_decodes, batch.num_seqs
        expand = [i for i in range(nd, B) if qlens[i] >= EXPAND_MIN_ROWS and block_size % 16 == 0]
        short = [i for i in range(nd, B) if qlens[i] < EXPAND_MIN_ROWS or block_size % 16]
        self.nd, self.n_short, self.n_expand = nd, len(short), len(expand)
        starts = [0]
        for n in qlens:
            starts.append(starts[-1] + n)
        T = starts[-1]
        self.rows_x = sum(qlens[i] for i in expand)
        self.rows_a = T - self.rows_x
        self.row_map = self.row_start = self.list_a = self.list_x = self.tiles = None
        parts: List[List[int]] = []
        if expand:
            row_map, row_start, list_a, list_x = [0] * T, [0] * B, [], []
            for i in range(B):
                rows = range(starts[i], starts[i + 1])
                dst = list_x if i in set(expand) else list_a
                row_start[i] = len(dst)
                for r in rows:
                    row_map[r] = -(len(dst) + 1) if dst is list_x else len(dst)
                    dst.append(r)
            parts += [row_map, row_start, list_a, list_x]
        if short:
            seqs, firsts = [], []
            for i in short:
                for r in range(0, qlens[i] * H, 16 * mt):
                    seqs.append(i)
                    firsts.append(r)
            self.n_tiles = len(seqs)
            parts += [seqs, firsts]
        if expand:
            # the visible tokens of every expanded sequence on scratch pages, counted from the first page a row can see
            page_seq, page_idx, tables, lens, qsl, self.x_lens, self.x_qlens = [], [], [], [], [0], [], []
            for i in expand:
                L, n = batch.seq_lens_host[i], qlens[i]
                lo = max(0, L - n - window + 1) // 16 if window else 0
                hi = (L + 15) // 16
                tables.append(list(range(len(page_seq), len(page_seq) + hi - lo)))
                page_seq += [i] * (hi - lo)
                page_idx += list(range(lo, hi))
                lens.append(L - 16 * lo)
                qsl.append(qsl[-1] + n)
                self.x_lens.append(L - 16 * lo)
                self.x_qlens.append(n)
            wide = max(len(t) for t in tables)
            flat = [x for t in tables for x in t + [0] * (wide - len(t))]
            self.pages, self.table_cols = len(page_seq), wide
            parts += [page_seq, page_idx, flat, lens, qsl]
        if not parts:
            return
        host = torch.tensor([x for p in parts for x in p], dtype=torch.int32).pin_memory()
        dev = host.to(device, non_blocking=True)
        self._keep = dev
        cut = list(dev.split([len(p) for p in parts]))
        if expand:
            self.row_map, self.row_start, self.list_a, self.list_x = cut[:4]
            cut = cut[4:]
        if short:
            self.tiles = (cut[0], cut[1])
            cut = cut[2:]
        if expand:
            self.page_seq, self.page_idx, table, lens, qsl = cut
            self.batch_x = SimpleNamespace(block_tables=table.view(len(expand), self.table_cols), seq_lens=lens, query_start_loc=qsl, num_decodes=0,
                                           num_seqs=len(expand), query_lens_host=self.x_qlens, seq_lens_host=self.x_lens,
                                           max_seq_len=max(self.x_lens))


def _plan(batch, window: int, H: int, mt: int, block_size: int, device) -> _Plan:
    plans = getattr(batch, "_latent_plans", None)
    if plans is None:
        plans = batch._latent_plans = {}
    key = (window, H, mt)
    if key not in plans:
        plans[key] = _Plan(batch, window, H, mt, block_size, device)
    return plans[key]


def _head_gemm(x, row: int, head: int, w, out, out_row: int, out_head: int, rows: int, in_rows=None, out_rows=None, offset: int = 0) -> None:
    H, N, Kd = w.shape
    K._check(_lib().atlas_head_gemm(x.data_ptr() + offset * x.element_size(), row, head, w.data_ptr(), out.data_ptr(), out_row, out_head,
                                    K._ptr(in_rows), K._ptr(out_rows), rows, H, N, Kd, K._stream()), "head_gemm")


def latent_attention(layer, q, ckv, batch, cache, rope_cache) -> torch.Tensor:
    """``q [T, H * (rope + nope)]``, ``ckv [T, rank + rope]`` fp32 -> ``[T, H * v]``; writes the step's cache rows."""
    T, H, W, rp = q.shape[0], layer.hq, layer.width, layer.rp
    bs, dev = cache.shape[1], q.device
    d = K._dev(q)
    lib, st = _lib(), K._stream()
    f32 = q.dtype == torch.float32
    assert q.stride(1) == 1 and ckv.dtype == torch.float32 and ckv.stride(1) == 1 and cache.dtype == q.dtype and cache.is_contiguous()
    assert batch.positions.dtype == batch.slot_mapping.dtype == torch.int32 and rope_cache.dtype == torch.float32
    if checked.ENABLED:
        checked.kv_write(batch.slot_mapping, batch.positions, cache.shape[0], bs, rope_cache.shape[0] if layer.rotary else 0)
        checked.paged_read(batch.block_tables, batch.seq_lens, cache.shape[0], bs)
    window, bt = int(layer.window or 0), batch.block_tables
    plan: Optional[_Plan] = None if f32 else _plan(batch, window, H, row_tiles(layer), bs, dev)
    rows_a, rows_x = (T, 0) if f32 else (plan.rows_a, plan.rows_x)
    qa = torch.empty(rows_a, H, W, dtype=q.dtype, device=dev) if rows_a else None
    qx = torch.empty(rows_x, H, layer.dx, dtype=q.dtype, device=dev) if rows_x else None
    K._check(lib.atlas_latent_rows(q.data_ptr(), q.stride(0), ckv.data_ptr(), ckv.stride(0), layer.c_norm.data_ptr(), batch.positions.data_ptr(),
                                   rope_cache.data_ptr(), batch.slot_mapping.data_ptr(), K._ptr(plan.row_map) if plan else None, cache.data_ptr(),
                                   K._ptr(qa), K._ptr(qx), T, H, layer.nope, layer.rope, layer.rotary, layer.rank, rp, layer.ep, layer.dx,
                                   float(layer.cfg.rms_norm_eps), 1 if f32 else 0, st), "latent_rows")
    qd = layer.rope + layer.nope
    if f32:
        # 32-bit products per head: a vendor product each way
        qa[:, :, :rp] = torch.einsum("thd,hrd->thr", q.view(T, H, qd)[:, :, layer.rope:], layer.uk)
        lat = torch.empty(T, H, rp, dtype=q.dtype, device=dev)
        K._check(lib.atlas_latent_attn_f32(qa.data_ptr(), cache.data_ptr(), lat.data_ptr(), bt.data_ptr(), bt.stride(0), batch.seq_lens.data_ptr(),
                                           batch.query_start_loc.data_ptr(), batch.num_seqs, T, H, rp, layer.ep, bs, window, float(layer.scale), st),
                 "latent_attn_f32")
        return torch.einsum("thr,hvr->thv", lat, layer.uv).reshape(T, H * layer.vd)
    out = torch.empty(T, H * layer.vd, dtype=q.dtype, device=dev)
    if rows_a:
        _head_gemm(q, q.stride(0), qd, layer.uk, qa, H * W, W, rows_a, in_rows=plan.list_a, offset=layer.rope)
        lat = torch.empty(rows_a, H, rp, dtype=q.dtype, device=dev)
        mt = row_tiles(layer)
        args = (bt.data_ptr(), bt.stride(0), batch.seq_lens.data_ptr(), batch.query_start_loc.data_ptr(), K._ptr(plan.row_start))
        if plan.nd:
            visible = min(batch.max_seq_len, window or batch.max_seq_len)
            splits = decode_splits(plan.nd, H, mt, visible, K._num_sms[d])
            po = pml = None
            if splits > 1:
                po = K.scratch("latent_part_o", plan.nd * H * splits * rp * 4, dev)
                pml = K.scratch("latent_part_ml", plan.nd * H * splits * 8, dev)
            K._check(lib.atlas_latent_attn(qa.data_ptr(), cache.data_ptr(), lat.data_ptr(), K._ptr(po), K._ptr(pml), *args, None, None, 0, plan.nd,
                                           plan.nd, H, rp, layer.ep, bs, window, splits, mt, float(layer.scale), st), "latent_attn_decode")
        if plan.n_short:
            K._check(lib.atlas_latent_attn(qa.data_ptr(), cache.data_ptr(), lat.data_ptr(), None, None, *args, plan.tiles[0].data_ptr(),
                                           plan.tiles[1].data_ptr(), plan.n_tiles, batch.num_seqs, rows_a, H, rp, layer.ep, bs, window, 1, mt,
                                           float(layer.scale), st), "latent_attn_rows")
        _head_gemm(lat, H * rp, rp, layer.uv, out, H * layer.vd, layer.vd, rows_a, out_rows=plan.list_a)
    if rows_x:
        c = torch.empty(plan.pages * 16, rp, dtype=q.dtype, device=dev)
        K._check(lib.atlas_latent_gather(cache.data_ptr(), bt.data_ptr(), bt.stride(0), batch.seq_lens.data_ptr(), plan.page_seq.data_ptr(),
                                         plan.page_idx.data_ptr(), plan.pages, bs, rp, W, c.data_ptr(), st), "latent_gather")
        kv = K.gemm_bf16(c, layer.expand)
        kp = torch.empty(plan.pages, H, 16, layer.dx, dtype=q.dtype, device=dev)
        vp = torch.empty(plan.pages, H, layer.dx, 16, dtype=q.dtype, device=dev)
        K._check(lib.atlas_latent_pages(kv.data_ptr(), cache.data_ptr(), bt.data_ptr(), bt.stride(0), batch.seq_lens.data_ptr(),
                                        plan.page_seq.data_ptr(), plan.page_idx.data_ptr(), plan.pages, bs, H, layer.nope, layer.rope, layer.vd, rp, W,
                                        layer.dx, kp.data_ptr(), vp.data_ptr(), st), "latent_pages")
        ox = K.paged_attention(qx, kp.permute(0, 2, 1, 3), vp.permute(0, 3, 1, 2), plan.batch_x, layer.scale, 1.0, 1.0, window)
        K._check(lib.atlas_latent_unpad(ox.data_ptr(), K._ptr(plan.list_x), rows_x, H, layer.vd, layer.dx, out.data_ptr(), st), "latent_unpad")
    return out
