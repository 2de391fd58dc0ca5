"""Plain-PyTorch restatement of every fused op the engine uses.

Each function here is (a) the CPU execution path and (b) the oracle that the
sm_100a kernels in ``atlas_b200/csrc`` are tested against.  They are written
for clarity, in fp32, with the same operation order the kernels use.

Layouts
-------
* activations are flattened over tokens: ``[T, ...]`` (continuous batching);
* paged KV cache: ``k_cache, v_cache [num_blocks, block_size, Hkv, D]`` (NHD),
  ``slot_mapping[t] = block * block_size + offset`` (-1 = padding row);
  reference layout: ``kernels/gb10/common/reshape_and_cache.cu:1-20``;
* GDN state per sequence slot: ``h [Hv, Dk, Dv]`` fp32 and a conv window
  ``[C, W-1]`` (reference: ``crates/spark-model/src/model/ssm_pool.rs``).
"""
from __future__ import annotations

import math
from typing import Optional, Tuple

import torch
import torch.nn.functional as F

from ..quant import FP8, FP8_MAX, per_token_group_quant_fp8


# ----------------------------------------------------------------------------- norms
def rmsnorm(x: torch.Tensor, w: torch.Tensor, eps: float, residual: Optional[torch.Tensor] = None,
            plus_one: bool = False) -> Tuple[torch.Tensor, Optional[torch.Tensor]]:
    """``r = x + residual``; ``y = r * rsqrt(mean(r^2)+eps) * (w | 1+w)``.  Returns ``(y, r)``."""
    dt = x.dtype
    xf = x.float()
    if residual is not None:
        xf = xf + residual.float()
        new_res = xf.to(dt)
        xf = new_res.float()          # the kernel normalises the rounded residual stream
    else:
        new_res = None
    var = xf.pow(2).mean(-1, keepdim=True)
    wf = w.float() + 1.0 if plus_one else w.float()
    y = (xf * torch.rsqrt(var + eps) * wf).to(dt)
    return y, new_res


def rmsnorm_quant_fp8(x, w, eps, residual=None, plus_one=False, group: int = 128):
    """Fused residual-add + RMSNorm + per-token-group FP8 quant. Returns ``(q, scale, r)``."""
    y, r = rmsnorm(x, w, eps, residual, plus_one)
    q, s = per_token_group_quant_fp8(y, group)
    return q, s, r


def gated_rmsnorm(x: torch.Tensor, z: torch.Tensor, w: torch.Tensor, eps: float) -> torch.Tensor:
    """``rmsnorm(x) * w * silu(z)`` over the last dim (GDN output norm)."""
    xf = x.float()
    var = xf.pow(2).mean(-1, keepdim=True)
    y = xf * torch.rsqrt(var + eps) * w.float()
    return (y * F.silu(z.float())).to(x.dtype)


def l2norm(x: torch.Tensor, eps: float = 1e-6) -> torch.Tensor:
    xf = x.float()
    return (xf * torch.rsqrt(xf.pow(2).sum(-1, keepdim=True) + eps)).to(x.dtype)


# ----------------------------------------------------------------------------- rope
def build_rope_cache(rotary_dim: int, max_pos: int, theta: float, scaling: Optional[dict] = None,
                     device="cpu") -> torch.Tensor:
    """``[max_pos, rotary_dim]`` fp32 table: first half cos, second half sin.

    Supports plain, linear, llama3 and YaRN scaling (reference: ``kernels/gb10/common/rope.cu``).
    """
    if rotary_dim <= 0:                  # position-free attention (no rotation)
        return torch.zeros(max_pos, 0, dtype=torch.float32, device=device)
    half = rotary_dim // 2
    inv_freq = 1.0 / (theta ** (torch.arange(0, half, dtype=torch.float64) * 2.0 / rotary_dim))
    mscale = 1.0
    if scaling:
        kind = scaling.get("rope_type", scaling.get("type", "default"))
        factor = float(scaling.get("factor", 1.0))
        if kind == "linear":
            inv_freq = inv_freq / factor
        elif kind == "llama3":
            lo, hi = float(scaling.get("low_freq_factor", 1.0)), float(scaling.get("high_freq_factor", 4.0))
            orig = float(scaling.get("original_max_position_embeddings", 8192))
            wavelen = 2 * math.pi / inv_freq
            smooth = ((orig / wavelen) - lo) / (hi - lo)
            scaled = torch.where(wavelen > orig / lo, inv_freq / factor,
                                 torch.where(wavelen < orig / hi, inv_freq,
                                             (1 - smooth) * inv_freq / factor + smooth * inv_freq))
            inv_freq = scaled
        elif kind == "yarn":
            orig = float(scaling.get("original_max_position_embeddings", 4096))
            beta_fast, beta_slow = float(scaling.get("beta_fast", 32)), float(scaling.get("beta_slow", 1))

            def corr(n_rot):
                return (rotary_dim * math.log(orig / (n_rot * 2 * math.pi))) / (2 * math.log(theta))
            low, high = max(math.floor(corr(beta_fast)), 0), min(math.ceil(corr(beta_slow)), rotary_dim - 1)
            ramp = ((torch.arange(half, dtype=torch.float64) - low) / max(high - low, 1e-3)).clamp(0, 1)
            mask = 1 - ramp
            inv_freq = inv_freq / factor * (1 - mask) + inv_freq * mask
            get = lambda m: 1.0 if factor <= 1 else 0.1 * m * math.log(factor) + 1.0
            if scaling.get("attention_factor"):
                mscale = float(scaling["attention_factor"])
            elif scaling.get("mscale") and scaling.get("mscale_all_dim"):     # DeepSeek convention: ratio of the two
                mscale = get(float(scaling["mscale"])) / get(float(scaling["mscale_all_dim"]))
            else:
                mscale = get(1.0)
    t = torch.arange(max_pos, dtype=torch.float64)
    freqs = torch.outer(t, inv_freq)
    cache = torch.cat([freqs.cos() * mscale, freqs.sin() * mscale], dim=-1).float()
    return cache.to(device)


def apply_rope(x: torch.Tensor, positions: torch.Tensor, cache: torch.Tensor, rotary_dim: int) -> torch.Tensor:
    """NeoX ("rotate half") rotary embedding on the first ``rotary_dim`` lanes of ``x [T,H,D]``."""
    half = rotary_dim // 2
    cs = cache[positions.long()]
    cos, sin = cs[:, None, :half], cs[:, None, half:]
    xf = x.float()
    x1, x2 = xf[..., :half], xf[..., half:rotary_dim]
    out = xf.clone()
    out[..., :half] = x1 * cos - x2 * sin
    out[..., half:rotary_dim] = x2 * cos + x1 * sin
    return out.to(x.dtype)


def head_rmsnorm(x: torch.Tensor, w: torch.Tensor, eps: float, plus_one: bool, dim: int = 0) -> torch.Tensor:
    """``dim``: channels the mean counts (0 = all)."""
    xf = x.float()
    var = xf.pow(2).sum(-1, keepdim=True) / (dim or x.shape[-1])
    wf = w.float() + 1.0 if plus_one else w.float()
    return (xf * torch.rsqrt(var + eps) * wf).to(x.dtype)


_HADAMARD: dict = {}


def hadamard(d: int, device="cpu") -> torch.Tensor:
    """Orthonormal Sylvester (natural-order) Hadamard matrix ``[d, d]``, ``H[i][j] = (-1)^popcount(i & j) / sqrt(d)``."""
    key = (d, str(device))
    if key not in _HADAMARD:
        assert d > 0 and d & (d - 1) == 0, "the Walsh-Hadamard rotation needs a power-of-two head_dim"
        h = torch.ones(1, 1)
        while h.shape[0] < d:
            h = torch.cat([torch.cat([h, h], 1), torch.cat([h, -h], 1)], 0)
        _HADAMARD[key] = (h / d ** 0.5).to(device)
    return _HADAMARD[key]


def head_rotate(x: torch.Tensor) -> torch.Tensor:
    return (x.float() @ hadamard(x.shape[-1], x.device)).to(x.dtype)


def qk_norm_rope_kv_write(q: torch.Tensor, k: torch.Tensor, v: torch.Tensor, positions: torch.Tensor,
                          rope_cache: torch.Tensor, rotary_dim: int,
                          k_cache: torch.Tensor, v_cache: torch.Tensor, slot_mapping: torch.Tensor,
                          k_scale: float = 1.0, v_scale: float = 1.0,
                          q_norm_w: Optional[torch.Tensor] = None, k_norm_w: Optional[torch.Tensor] = None,
                          eps: float = 1e-6, norm_plus_one: bool = False, rotate: bool = False, norm_dim: int = 0) -> torch.Tensor:
    """Fused (q/k head RMSNorm) + RoPE + (head rotation) + (FP8 quant) + paged cache write.

    ``q [T,Hq,D]``, ``k,v [T,Hkv,D]``.  Returns the roped ``q``; k/v go to the cache at
    ``slot_mapping`` (rows with slot < 0 are skipped).
    """
    if q_norm_w is not None:
        q = head_rmsnorm(q, q_norm_w, eps, norm_plus_one, norm_dim)
        k = head_rmsnorm(k, k_norm_w, eps, norm_plus_one, norm_dim)
    q = apply_rope(q, positions, rope_cache, rotary_dim)
    k = apply_rope(k, positions, rope_cache, rotary_dim)
    if rotate:
        q, k, v = head_rotate(q), head_rotate(k), head_rotate(v)
    nb, bs, hkv, d = k_cache.shape
    valid = slot_mapping >= 0
    slots = slot_mapping[valid].long()
    blk, off = slots // bs, slots % bs          # index the logical dims: the cache may be a permuted view
    if k_cache.dtype == FP8:
        k_cache[blk, off] = (k[valid].float() / k_scale).clamp(-FP8_MAX, FP8_MAX).to(FP8)
        v_cache[blk, off] = (v[valid].float() / v_scale).clamp(-FP8_MAX, FP8_MAX).to(FP8)
    else:
        k_cache[blk, off] = k[valid].to(k_cache.dtype)
        v_cache[blk, off] = v[valid].to(v_cache.dtype)
    return q


def map_norm_kv_write(q, k, v, positions, rope_cache, rotary_dim, k_cache, v_cache, slot_mapping, q_norm_w, k_norm_w, eps: float):
    """See ``ops.map_norm_kv_write``; everything up to the result in fp32."""
    T, H, _, n = q.shape
    G, dv, D = k.shape[1], v.shape[2], k_cache.shape[3]

    def turned(x, w):
        x = x.float() * torch.rsqrt(x.float().pow(2).mean(-1, keepdim=True) + eps) * w.float()
        return apply_rope(x.reshape(T, -1, n), positions, rope_cache, rotary_dim)
    qf, kf = turned(q, q_norm_w).view(T, H, 2, n), turned(k, k_norm_w).reshape(T, G, 2 * n)
    ok = slot_mapping >= 0
    slots, bs = slot_mapping[ok].long(), k_cache.shape[1]
    k_cache[slots // bs, slots % bs, :, :2 * n] = kf[ok].to(k_cache.dtype)
    v_cache[slots // bs, slots % bs, :, :dv] = v[ok].to(v_cache.dtype)
    rows = torch.zeros(T, H, 2, D, dtype=q.dtype, device=q.device)
    rows[:, :, 0, :n], rows[:, :, 1, n:2 * n] = qf[:, :, 0].to(q.dtype), qf[:, :, 1].to(q.dtype)
    return rows.view(T, 2 * H, D)


def map_difference(a, dv: int, lam: float, rest: float, eps: float, gate=None):
    """See ``ops.map_difference``."""
    T = a.shape[0]
    o = a.float().view(T, -1, 2, a.shape[2])[..., :dv]
    o = o[:, :, 0] - lam * o[:, :, 1]
    o = (o * torch.rsqrt(o.pow(2).mean(-1, keepdim=True) + eps) * rest).reshape(T, -1)
    return (o if gate is None else o * torch.sigmoid(gate.float())).to(a.dtype)


def qk_row_norm_kv_write(q, k, v, positions, rope_cache, rotary_dim, k_cache, v_cache, slot_mapping, seq_positions, q_norm_w, k_norm_w,
                         eps: float, nq: int, nk: int, temp: float, temp_every: int, sums=None):
    """See ``ops.qk_row_norm_kv_write``; everything up to the result in fp32."""
    def unit(x, w, n, ss):
        ss = x.float().square().sum((1, 2)) if ss is None else ss
        return x.float() * torch.rsqrt(ss / n + eps)[:, None, None] * w.float().view(x.shape[1:])
    qf = unit(q, q_norm_w, nq, None if sums is None else sums[:, 0])
    kf = unit(k, k_norm_w, nk, None if sums is None else sums[:, 1])
    qf, kf = (apply_rope(t, positions, rope_cache, rotary_dim) for t in (qf, kf))
    steps = torch.div(seq_positions + 1, temp_every, rounding_mode="floor") + 1
    qf = qf * (1.0 + temp * torch.log(steps.float()))[:, None, None]
    ok = slot_mapping >= 0
    slots, bs = slot_mapping[ok].long(), k_cache.shape[1]
    k_cache[slots // bs, slots % bs] = kf[ok].to(k_cache.dtype)
    v_cache[slots // bs, slots % bs] = v[ok].to(v_cache.dtype)
    return qf.to(q.dtype)


# ----------------------------------------------------------------------------- attention
def paged_attention(q: torch.Tensor, k_cache: torch.Tensor, v_cache: torch.Tensor,
                    block_tables: torch.Tensor, seq_lens: torch.Tensor, query_start_loc: torch.Tensor,
                    scale: float, k_scale: float = 1.0, v_scale: float = 1.0,
                    sliding_window: Optional[int] = None, chunk: int = 0,
                    sinks: Optional[torch.Tensor] = None, softcap: float = 0.0,
                    distance: Optional[torch.Tensor] = None) -> torch.Tensor:
    """Causal attention of new query rows over the paged cache (prefill chunks and decode alike).

    ``chunk`` > 0 limits a row to keys of its own ``chunk``-token block (counted from the sequence's first token);
    ``sinks [Hq]`` adds ``exp(sink)`` to every row's softmax denominator; ``softcap`` > 0 bounds the scores; ``distance
    [Hq, n]`` is added to them by the key's distance, its last column from there on.

    Sequence ``b`` owns query rows ``query_start_loc[b]:query_start_loc[b+1]``; its last row sits
    at position ``seq_lens[b]-1``.  ``q [T,Hq,D]`` -> ``out [T,Hq,D]``.
    """
    T, Hq, D = q.shape
    nb, bs, Hkv, _ = k_cache.shape
    G = Hq // Hkv
    out = torch.zeros_like(q)
    qsl = query_start_loc.tolist()
    sl = seq_lens.tolist()
    for b in range(len(sl)):
        q0, q1 = qsl[b], qsl[b + 1]
        ql, L = q1 - q0, sl[b]
        if ql <= 0 or L <= 0:
            continue
        nblk = (L + bs - 1) // bs
        blocks = block_tables[b, :nblk].long()
        kk = k_cache[blocks].reshape(nblk * bs, Hkv, D)[:L].float() * k_scale
        vv = v_cache[blocks].reshape(nblk * bs, Hkv, D)[:L].float() * v_scale
        qq = q[q0:q1].float().view(ql, Hkv, G, D)
        s = torch.einsum("qhgd,khd->hgqk", qq, kk) * scale
        if softcap:
            s = softcap * torch.tanh(s / softcap)
        qpos = torch.arange(L - ql, L, device=q.device)[:, None]
        kpos = torch.arange(L, device=q.device)[None, :]
        if distance is not None:
            back = (qpos - kpos).clamp(0, distance.shape[1] - 1)
            s = s + distance.view(Hkv, G, -1)[:, :, back]
        mask = kpos <= qpos
        if sliding_window:
            mask &= kpos > qpos - sliding_window
        if chunk:
            mask &= torch.div(kpos, chunk, rounding_mode="floor") == torch.div(qpos, chunk, rounding_mode="floor")
        s = s.masked_fill(~mask[None, None], float("-inf"))
        if sinks is not None:
            s = torch.cat([s, sinks.float().view(Hkv, G, 1, 1).expand(Hkv, G, ql, 1)], -1)
        p = torch.softmax(s, dim=-1)[..., :L]
        o = torch.einsum("hgqk,khd->qhgd", p, vv).reshape(ql, Hq, D)
        out[q0:q1] = o.to(q.dtype)
    return out


# ----------------------------------------------------------------------------- residual streams, WKV
def hyper_norm(streams, delta, read, norm_w, eps):
    """See ``ops.hyper_norm``; everything in fp32, the result in the dtype of ``delta.y``."""
    y = delta.y.float()
    if delta.conn is None:
        x = (y * delta.scale)[:, None, :].expand(-1, read.shape[0], -1).clone()
    else:
        if delta.y2 is not None:
            unit = lambda t: t * torch.rsqrt(t.pow(2).mean(-1, keepdim=True) + eps)
            y = 0.5 * (unit(y) * delta.w1.float() + unit(delta.y2.float()) * delta.w2.float())
        c = delta.conn
        x = torch.einsum("st,nsw->ntw", c.mix, streams) + c.write[None, :, None] * y[:, None, :]
    u = torch.einsum("s,nsw->nw", read.float(), x)
    h = u * torch.rsqrt(u.pow(2).mean(-1, keepdim=True) + eps) * norm_w.float()
    return h.to(delta.y.dtype), x


def token_shift_mix(x: torch.Tensor, prev: torch.Tensor, mu: torch.Tensor) -> torch.Tensor:
    """``x + (prev - x) * mu_s`` for every row of ``mu [S, W]``: ``[S, T, W]``."""
    xf, pf = x.float(), prev.float()
    return (xf[None] + (pf - xf)[None] * mu.float()[:, None, :]).to(x.dtype)


def wkv_scan(r, k, v, decay, u, h):
    """Sequential WKV recurrence.  ``r, k, v, decay [T, H, D]`` fp32, ``u [H, D]``, ``h [H, V, K]`` -> ``(o [T, H, V], h)``."""
    out = []
    for t in range(r.shape[0]):
        kv = v[t][:, :, None] * k[t][:, None, :]
        out.append(((h + u.float()[:, None, :] * kv) * r[t][:, None, :]).sum(-1))
        h = h * decay[t][:, None, :] + kv
    return torch.stack(out), h


def group_norm_gate(y, z, w, group: int, eps: float, gate_first: bool, gate: str = "silu", den=None):
    """``norm(y * gate(z)) * w`` or ``norm(y) * w * gate(z)``, RMS over groups of ``group`` channels, each divided by ``den`` first."""
    gz = (torch.sigmoid if gate == "sigmoid" else F.silu)(z.float())
    v = y.float() * gz if gate_first else y.float()
    g = v.reshape(*v.shape[:-1], -1, group)
    if den is not None:
        g = g / den[..., None]
    v = (g * torch.rsqrt(g.pow(2).mean(-1, keepdim=True) + eps)).reshape(v.shape) * w.float()
    return (v if gate_first else v * gz).to(y.dtype)


# ----------------------------------------------------------------------------- mLSTM, latent attention, normed outputs
MLSTM_EPS = 1e-6            # joins the denominator of the memory's output


def mlstm_gates(raw, bias, cap: float, m):
    """Raw gates ``[T, 2 H]`` (input, forget) -> per row the log factors on the old state and on the new token, and the running
    maximum: ``la = f + m_prev - m <= 0``, ``lb = i - m <= 0``, ``m`` (all ``[T, H]``).  ``m`` carries on from ``m [H]``."""
    z = cap * torch.tanh((raw.float() + bias) / cap)
    i, f = z.chunk(2, -1)
    f = F.logsigmoid(f)
    la, lb, ms = [], [], []
    for t in range(raw.shape[0]):
        new = torch.maximum(f[t] + m, i[t])
        la.append(f[t] + m - new)
        lb.append(i[t] - new)
        ms.append(new)
        m = new
    return torch.stack(la), torch.stack(lb), torch.stack(ms)


def mlstm_scan(q, k, v, la, lb, h):
    """Sequential memory.  ``q`` (scaled), ``k [T, H, D]``, ``v [T, H, V]``, ``h [H, V + 1, D]`` (last row: the normaliser) ->
    ``(S q [T, H, V], n . q [T, H], h)``."""
    one = torch.ones(v.shape[1], 1, dtype=v.dtype, device=v.device)
    out = []
    for t in range(k.shape[0]):
        new = torch.cat([v[t], one], -1)[:, :, None] * k[t][:, None, :]
        h = h * torch.exp(la[t])[:, None, None] + torch.exp(lb[t])[:, None, None] * new
        out.append((h * q[t][:, None, :]).sum(-1))
    o = torch.stack(out)
    return o[..., :-1], o[..., -1], h


def latent_rows(ckv, q_rope, norm_w, rank: int, rp: int, ep: int, positions, rope_cache, rotary: int, eps: float):
    """``(cache rows [T, rp + ep], rotated query parts [T, H, ep])`` of a step, fp32, zero-padded to the cache row's widths."""
    c = ckv[:, :rank].float()
    c = c * torch.rsqrt(c.pow(2).mean(-1, keepdim=True) + eps) * norm_w
    turn = (lambda x: apply_rope(x.float(), positions, rope_cache, rotary)) if rotary else (lambda x: x.float())
    r = turn(ckv[:, None, rank:])[:, 0]
    pad = lambda x, n: F.pad(x, (0, n - x.shape[-1]))
    return torch.cat([pad(c, rp), pad(r, ep)], -1), pad(turn(q_rope), ep)


def latent_attention(q, cache, rp: int, block_tables, seq_lens, query_start_loc, scale: float, window: Optional[int] = None):
    """Absorbed form: ``q [T, H, rp + ep]`` against cache rows of the same width, values the rows' first ``rp`` numbers."""
    out = torch.zeros(*q.shape[:2], rp, dtype=torch.float32, device=q.device)
    qsl, sl, bs = query_start_loc.tolist(), seq_lens.tolist(), cache.shape[1]
    for b, L in enumerate(sl):
        q0, q1 = qsl[b], qsl[b + 1]
        n = q1 - q0
        if n <= 0 or L <= 0:
            continue
        rows = cache[block_tables[b, :(L + bs - 1) // bs].long()].reshape(-1, cache.shape[-1])[:L].float()
        s = torch.einsum("qhw,kw->hqk", q[q0:q1].float(), rows) * scale
        qpos, kpos = torch.arange(L - n, L, device=q.device)[:, None], torch.arange(L, device=q.device)[None, :]
        see = kpos <= qpos
        if window:
            see &= kpos > qpos - window
        p = torch.softmax(s.masked_fill(~see, float("-inf")), -1)
        out[q0:q1] = torch.einsum("hqk,kr->qhr", p, rows[:, :rp])
    return out


def add_normed(stream, delta, eps: float, plus_one: bool, out_norm, write: bool, step=None, out_bias=None):
    """See ``ops.add_normed``."""
    if hasattr(delta.y, "slot_of"):
        e = delta.y
        T, k = e.w.shape
        slots = e.slot_of.view(T, k).long()
        picked = e.y.float()[slots.clamp_min(0)] * (slots >= 0)[..., None]
        y, dtype = (picked * e.w[..., None]).sum(1), e.y.dtype
        y = y if e.extra is None else y + e.extra.float()
    else:
        y, dtype = delta.y.float(), delta.y.dtype
    if delta.gate is not None:
        y = y * torch.sigmoid(delta.gate.float())

    def unit(t, w, b):
        t = t if b is None else t - t.mean(-1, keepdim=True)
        t = t * torch.rsqrt(t.pow(2).mean(-1, keepdim=True) + eps) * (w.float() + 1.0 if plus_one else w.float())
        return t if b is None else t + b.float()
    if stream is None:
        x = y * delta.scale
    else:
        x = stream + (y if delta.norm is None else unit(y, delta.norm, delta.bias))
    x = x if step is None else x + step
    if delta.depth is not None:
        d, entry = delta.depth, x
        if d.factors is not None:
            x = entry * d.factors[d.index]
            for j in range(d.index):
                x = x + d.history[j] * d.factors[j]
        if write or stream is None:
            d.history[d.index] = entry
    if write and stream is not None:
        stream.copy_(x)
    h = x if out_norm is None else unit(x, out_norm, out_bias)
    return h.to(dtype), (x.clone() if stream is None else stream)      # the stream changes in place, h does not


def gelu_embedding(z, table, ids, first: int, n: int):
    """See ``ops.gelu_embedding``."""
    out = torch.zeros_like(z)
    out[:, :n] = (F.gelu(z[:, :n].float(), approximate="tanh") * table[ids.long(), first:first + n].float()).to(z.dtype)
    return out


# ----------------------------------------------------------------------------- activations
def gated_unit(gate_up: torch.Tensor, unit: Tuple[float, float, float], paired: bool = False) -> torch.Tensor:
    """See ``ops.gated_unit_act``."""
    limit, alpha, shift = unit
    i = gate_up.shape[-1] // 2
    g, u = (gate_up[..., 0::2], gate_up[..., 1::2]) if paired else (gate_up[..., :i], gate_up[..., i:])
    g, u = g.float().clamp(max=limit), u.float().clamp(-limit, limit)
    return (g * torch.sigmoid(alpha * g) * (u + shift)).to(gate_up.dtype)


def silu_mul(gate_up: torch.Tensor) -> torch.Tensor:
    """``[T, 2I]`` (gate | up) -> ``silu(gate) * up`` ``[T, I]``."""
    i = gate_up.shape[-1] // 2
    g, u = gate_up[..., :i].float(), gate_up[..., i:].float()
    return (F.silu(g) * u).to(gate_up.dtype)


def gelu_tanh_mul(gate_up: torch.Tensor) -> torch.Tensor:
    i = gate_up.shape[-1] // 2
    g, u = gate_up[..., :i].float(), gate_up[..., i:].float()
    return (F.gelu(g, approximate="tanh") * u).to(gate_up.dtype)


def silu_mul_quant_fp8(gate_up: torch.Tensor, group: int = 128):
    y = silu_mul(gate_up)
    return per_token_group_quant_fp8(y, group)


# ----------------------------------------------------------------------------- MoE
def quant_nvfp4_rowwise(x: torch.Tensor) -> torch.Tensor:
    """What the W4A4 path's activation quantiser stands for, as an fp32 matrix: per row a second-level scale
    ``g = amax / (6 * 448)``, per 16 values an e4m3 scale factor against ``g``, values rounded to e2m1."""
    from ..quant import E2M1_MAX, _e2m1_lut, _round_to_e2m1_code
    xf = x.float()
    T, K = xf.shape
    amax = xf.abs().amax(-1, keepdim=True)
    g = torch.where(amax > 0, amax / (E2M1_MAX * FP8_MAX), torch.ones_like(amax))
    grp = xf.view(T, K // 16, 16)
    s8 = (grp.abs().amax(-1) / (E2M1_MAX * g)).clamp(max=FP8_MAX).to(FP8).float()
    s = s8 * g
    inv = torch.where(s > 0, 1.0 / s, torch.zeros_like(s))
    codes = _round_to_e2m1_code(grp * inv[..., None])
    vals = _e2m1_lut(x.device)[codes.long()]
    return (vals * s[..., None]).view(T, K)


def route_scores(logits: torch.Tensor, scoring: str) -> torch.Tensor:
    lf = logits.float()
    if scoring == "sigmoid":
        return torch.sigmoid(lf)
    if scoring == "sqrtsoftplus":
        return torch.sqrt(F.softplus(lf))
    return torch.softmax(lf, -1)


def moe_route(logits: torch.Tensor, top_k: int, norm_topk: bool, scoring: str = "softmax", bias: Optional[torch.Tensor] = None,
              n_group: int = 0, topk_group: int = 0, scale: float = 1.0, hash_table: Optional[torch.Tensor] = None,
              token_ids: Optional[torch.Tensor] = None):
    """Router scores -> (weights ``[T,k]`` fp32, expert ids ``[T,k]`` int32); ties pick the lower id.

    ``bias`` biases the SELECTION only (weights come from the unbiased scores).  ``n_group`` / ``topk_group``: a group
    scores the sum of its two best biased scores and only the best ``topk_group`` groups stay eligible.  ``hash_table
    [vocab, k]`` replaces selection by a lookup on ``token_ids``.  ``scale`` multiplies the final weights.
    """
    probs = route_scores(logits, scoring)
    if hash_table is not None:
        ids = hash_table.to(logits.device)[token_ids.long()].long().clamp(0, probs.shape[-1] - 1)
        w = probs.gather(-1, ids)
        if norm_topk:
            w = w / (w.sum(-1, keepdim=True) + 1e-20)
        return w * scale, ids.to(torch.int32)
    sel = probs if bias is None else probs + bias.float()
    if n_group > 1 and 0 < topk_group < n_group:
        T, E = sel.shape
        g = sel.view(T, n_group, E // n_group)
        gs = g.topk(min(2, g.shape[-1]), dim=-1).values.sum(-1)
        keep = torch.zeros_like(gs, dtype=torch.bool).scatter_(1, _topk_low_ties(gs, topk_group), True)
        sel = g.masked_fill(~keep[..., None], float("-inf")).view(T, E)
    ids = _topk_low_ties(sel, top_k)
    w = probs.gather(-1, ids)
    if norm_topk:
        w = w / w.sum(-1, keepdim=True).clamp_min(1e-20)
    return w * scale, ids.to(torch.int32)


def _topk_low_ties(x: torch.Tensor, k: int) -> torch.Tensor:
    """Indices of the k largest along the last dim, descending, ties to the lower index (a stable sort gives that)."""
    return torch.sort(x, dim=-1, descending=True, stable=True).indices[..., :k]


def expert_act(h: torch.Tensor, activation: str, unit: Optional[Tuple[float, float, float]] = None) -> torch.Tensor:
    """``silu_glu``: silu(gate) * up of ``[gate | up]``; ``relu2``: squared relu of a single up projection; ``clamped_glu``: the
    gated unit ``(limit, alpha, shift)`` of alternating gate and up columns."""
    if activation == "relu2":
        return torch.relu(h).square()
    if activation == "clamped_glu":
        return gated_unit(h, unit, paired=True)
    i = h.shape[-1] // 2
    return F.silu(h[..., :i]) * h[..., i:]


def moe_experts(x: torch.Tensor, w13: torch.Tensor, w2: torch.Tensor, topk_w: torch.Tensor,
                topk_ids: torch.Tensor, expert_lo: int = 0, activation: str = "silu_glu",
                unit: Optional[Tuple[float, float, float]] = None) -> torch.Tensor:
    """Dense-math MoE over local experts ``[expert_lo, expert_lo+E_local)``.

    ``w13 [E,2I,H]`` (gate rows then up rows; ``relu2``: ``[E,I,H]``; ``clamped_glu``: alternating), ``w2 [E,H,I]`` already dequantized.
    Tokens routed to non-local experts contribute zero (their owner rank adds them).
    """
    T, H = x.shape
    E = w13.shape[0]
    out = torch.zeros(T, H, dtype=torch.float32, device=x.device)
    xf = x.float()
    for e in range(E):
        sel = (topk_ids == (e + expert_lo))
        tok = sel.any(-1).nonzero(as_tuple=True)[0]
        if tok.numel() == 0:
            continue
        wgt = (topk_w * sel).sum(-1)[tok]
        h = xf[tok] @ w13[e].float().t()
        a = expert_act(h, activation, unit).to(x.dtype).float()
        y = a @ w2[e].float().t()
        out.index_add_(0, tok, y * wgt[:, None])
    return out.to(x.dtype)


# ----------------------------------------------------------------------------- Gated DeltaNet
def causal_conv1d(x: torch.Tensor, conv_state: torch.Tensor, weight: torch.Tensor,
                  bias: Optional[torch.Tensor] = None, activation: bool = True):
    """Depthwise causal conv over one sequence chunk.

    ``x [L,C]``, ``conv_state [C,W-1]`` (previous inputs, oldest first), ``weight [C,W]``.
    Returns ``(y [L,C], new_state [C,W-1])``.
    """
    L, C = x.shape
    W = weight.shape[-1]
    full = torch.cat([conv_state.float().t(), x.float()], dim=0)      # [W-1+L, C]
    win = full.unfold(0, W, 1)                                         # [L, C, W]
    y = (win * weight.float()[None]).sum(-1)
    if bias is not None:
        y = y + bias.float()
    if activation:
        y = F.silu(y)
    new_state = full[full.shape[0] - (W - 1):].t().contiguous().to(conv_state.dtype)
    return y.to(x.dtype), new_state


def rglru_gates(u, zr, zi, lam):
    """RG-LRU: decay ``a`` and drive ``sqrt(1 - a^2) i u`` of every row and channel in fp32, from the raw gates ``zr`` / ``zi``
    (biases included): ``log a = -8 sigmoid(zr) softplus(lam)``, ``i = sigmoid(zi)``."""
    log_a = -8.0 * torch.sigmoid(zr.float()) * F.softplus(lam.float())
    return torch.exp(log_a), torch.sqrt(-torch.expm1(2.0 * log_a)) * torch.sigmoid(zi.float()) * u.float()


def linear_recurrence(a, drive, h):
    """``h_t = a_t h_(t-1) + drive_t`` row by row: every state ``[T, C]`` (the last one carries on)."""
    out = []
    for t in range(a.shape[0]):
        h = a[t] * h + drive[t]
        out.append(h)
    return torch.stack(out)


def gdn_gates(a: torch.Tensor, b: torch.Tensor, A_log: torch.Tensor, dt_bias: torch.Tensor):
    """``g = -exp(A_log) * softplus(a + dt_bias)`` (log decay, fp32), ``beta = sigmoid(b)``."""
    g = -A_log.float().exp() * F.softplus(a.float() + dt_bias.float())
    return g, torch.sigmoid(b.float())


def gdn_recurrent(q, k, v, g, beta, h0: torch.Tensor, scale: Optional[float] = None):
    """Token-by-token gated delta rule over one sequence.

    ``q,k [L,H,Dk]`` (already l2-normalised), ``v [L,H,Dv]``, ``g,beta [L,H]``, ``h0 [H,Dk,Dv]`` fp32.
    ``h_t = exp(g_t) h_{t-1} + k_t (x) ((v_t - h_{t-1}'^T k_t) beta_t)``, ``o_t = h_t^T q_t * scale``.
    Returns ``(o [L,H,Dv], h_L, h_all [L,H,Dk,Dv])``.
    """
    L, H, Dk = q.shape
    scale = scale if scale is not None else Dk ** -0.5
    h = h0.float().clone()
    outs, hs = [], []
    for t in range(L):
        h = h * g[t].float().exp()[:, None, None]
        kt, vt = k[t].float(), v[t].float()
        mem = torch.einsum("hkv,hk->hv", h, kt)
        delta = (vt - mem) * beta[t].float()[:, None]
        h = h + kt[:, :, None] * delta[:, None, :]
        outs.append(torch.einsum("hkv,hk->hv", h, q[t].float() * scale))
        hs.append(h.clone())
    o = torch.stack(outs).to(v.dtype) if L else torch.zeros(0, H, v.shape[-1], dtype=v.dtype, device=v.device)
    return o, h, (torch.stack(hs) if L else h[None][:0])


def gdn_chunked(q, k, v, g, beta, h0: torch.Tensor, chunk: int = 64, scale: Optional[float] = None):
    """Chunk-parallel form of :func:`gdn_recurrent` (WY/UT transform inside a chunk, state pass between).

    Mirrors what the chunked scan kernel computes; used to test that formulation against the
    sequential recurrence.  Reference: ``kernels/gb10/common/gated_delta_rule_fla.cu`` (CHUNK=64).
    """
    L, H, Dk = q.shape
    Dv = v.shape[-1]
    scale = scale if scale is not None else Dk ** -0.5
    h = h0.float().clone()
    out = torch.zeros(L, H, Dv, dtype=torch.float32, device=q.device)
    for c0 in range(0, L, chunk):
        c1 = min(L, c0 + chunk)
        n = c1 - c0
        qc = q[c0:c1].float().transpose(0, 1) * scale       # [H,n,Dk]
        kc = k[c0:c1].float().transpose(0, 1)
        vc = v[c0:c1].float().transpose(0, 1)
        bc = beta[c0:c1].float().transpose(0, 1)            # [H,n]
        gc = g[c0:c1].float().transpose(0, 1).cumsum(-1)    # cumulative log decay inside chunk
        tril = torch.tril(torch.ones(n, n, dtype=torch.bool, device=q.device), -1)
        tril0 = torch.tril(torch.ones(n, n, dtype=torch.bool, device=q.device))
        decay = (gc[:, :, None] - gc[:, None, :]).masked_fill(~tril0, 0.0)   # [H,n,n] log(G_i/G_j), i>=j
        kk = torch.einsum("hik,hjk->hij", kc, kc)
        A = -(kk * decay.exp() * bc[:, :, None]).masked_fill(~tril, 0.0)   # strictly lower
        # (I - A)^{-1} by forward substitution
        Tm = torch.eye(n, device=q.device).expand(H, n, n).clone()
        for i in range(1, n):
            Tm[:, i, :i] = torch.einsum("hj,hjk->hk", A[:, i, :i], Tm[:, :i, :i])
        u = torch.einsum("hij,hjv->hiv", Tm, vc * bc[:, :, None])
        w = torch.einsum("hij,hjk->hik", Tm, kc * (bc * gc.exp())[:, :, None])
        v_new = u - torch.einsum("hik,hkv->hiv", w, h)
        qk = torch.einsum("hik,hjk->hij", qc, kc)
        attn = (qk * decay.exp()).masked_fill(~tril0, 0.0)
        o = torch.einsum("hik,hkv->hiv", qc * gc.exp()[:, :, None], h) + torch.einsum("hij,hjv->hiv", attn, v_new)
        out[c0:c1] = o.transpose(0, 1)
        glast = gc[:, -1]
        h = h * glast.exp()[:, None, None] + torch.einsum(
            "hik,hiv->hkv", kc * (glast[:, None] - gc).exp()[:, :, None], v_new)
    return out.to(v.dtype), h


# ----------------------------------------------------------------------------- sampling
def argmax_first(logits: torch.Tensor) -> torch.Tensor:
    """Greedy argmax; ties resolve to the lowest index (reference: ``sampler.rs:512``)."""
    lf = logits.float()
    mx = lf.max(-1, keepdim=True).values
    idx = torch.arange(lf.shape[-1], device=lf.device).expand_as(lf)
    big = torch.full_like(idx, lf.shape[-1])
    return torch.where(lf == mx, idx, big).min(-1).values.to(torch.int64)


def apply_penalties(logits: torch.Tensor, token_counts: Optional[torch.Tensor], prompt_mask: Optional[torch.Tensor],
                    repetition: torch.Tensor, presence: torch.Tensor, frequency: torch.Tensor) -> torch.Tensor:
    """OpenAI presence/frequency penalties over generated counts + HF repetition penalty over seen tokens."""
    lf = logits.float()
    if token_counts is None:
        return lf
    seen = token_counts > 0
    if prompt_mask is not None:
        seen_rep = seen | prompt_mask
    else:
        seen_rep = seen
    rp = repetition[:, None]
    lf = torch.where(seen_rep, torch.where(lf > 0, lf / rp, lf * rp), lf)
    lf = lf - frequency[:, None] * token_counts.float() - presence[:, None] * seen.float()
    return lf


def sample(logits: torch.Tensor, temperature: torch.Tensor, top_k: torch.Tensor, top_p: torch.Tensor,
           min_p: torch.Tensor, uniform: torch.Tensor) -> torch.Tensor:
    """Temperature / top-k / top-p / min-p sampling with caller-provided uniforms (one per row).

    Rows with ``temperature == 0`` are greedy.  The filter order is top-k, top-p, min-p over the
    temperature-scaled distribution sorted descending (ties by lower id), then inverse-CDF with
    ``uniform[row]``.
    """
    lf = logits.float()
    B, V = lf.shape
    greedy = argmax_first(lf)
    t = temperature.clamp_min(1e-6)[:, None]
    probs = torch.softmax(lf / t, -1)
    sp, si = torch.sort(probs, dim=-1, descending=True, stable=True)
    rank = torch.arange(V, device=lf.device)[None, :]
    k = torch.where(top_k <= 0, torch.full_like(top_k, V), top_k)[:, None]
    keep = rank < k
    csum = sp.cumsum(-1)
    keep &= (csum - sp) < top_p[:, None]
    keep &= sp >= (min_p[:, None] * sp[:, :1])
    keep[:, 0] = True
    sp = torch.where(keep, sp, torch.zeros_like(sp))
    sp = sp / sp.sum(-1, keepdim=True)
    cdf = sp.cumsum(-1)
    pick = (cdf < uniform[:, None] * (1 - 1e-7)).sum(-1).clamp(max=V - 1)
    sampled = si.gather(1, pick[:, None]).squeeze(1)
    return torch.where(temperature <= 0, greedy, sampled)


def spec_verify_greedy(draft_tokens: torch.Tensor, target_argmax: torch.Tensor):
    """Greedy speculative acceptance.

    ``draft_tokens [B,K]`` proposed tokens, ``target_argmax [B,K+1]`` the target's argmax after
    consuming ``[last, d_0..d_{K-1}]``.  Returns ``(num_accepted [B], out_tokens [B,K+1])`` where
    ``out_tokens[:, :n+1]`` are the tokens to emit (accepted drafts then the bonus/correction).
    """
    B, K = draft_tokens.shape
    match = (draft_tokens == target_argmax[:, :K]).to(torch.int64)
    n_acc = match.cumprod(-1).sum(-1)
    return n_acc, target_argmax.clone()


def spec_verify_sample(draft_tokens, draft_probs, target_probs, uniform, resample_uniform):
    """Rejection-sampling acceptance (Leviathan et al.): accept ``d_i`` iff ``u_i < p(d_i)/q(d_i)``;
    on the first rejection resample from ``norm(max(p - q, 0))``; if all accepted sample the bonus from ``p_K``.

    ``draft_probs [B,K,V]``, ``target_probs [B,K+1,V]``, ``uniform [B,K]``, ``resample_uniform [B]``.
    """
    B, K = draft_tokens.shape
    V = target_probs.shape[-1]
    out = torch.zeros(B, K + 1, dtype=torch.int64, device=draft_tokens.device)
    n_acc = torch.zeros(B, dtype=torch.int64, device=draft_tokens.device)
    for b in range(B):
        n = 0
        for i in range(K):
            d = int(draft_tokens[b, i])
            p, qd = float(target_probs[b, i, d]), float(draft_probs[b, i, d])
            if qd > 0 and float(uniform[b, i]) < min(1.0, p / qd):
                out[b, i] = d
                n += 1
            else:
                break
        if n < K:
            resid = (target_probs[b, n].float() - draft_probs[b, n].float()).clamp_min(0)
            if float(resid.sum()) <= 0:
                resid = target_probs[b, n].float()
        else:
            resid = target_probs[b, K].float()
        cdf = (resid / resid.sum()).cumsum(-1)
        out[b, n] = int((cdf < float(resample_uniform[b]) * (1 - 1e-7)).sum().clamp(max=V - 1))
        n_acc[b] = n
    return n_acc, out
