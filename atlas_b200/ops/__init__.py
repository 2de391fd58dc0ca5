"""Op front-end: every call goes to the sm_100a kernel library when the tensors live on a GPU and to
the plain-PyTorch restatement (``ops.reference``) otherwise.

On a machine with a GPU the kernel library is mandatory: importing this package there without a
built ``libatlas_b200_kernels.so`` raises instead of silently running eager PyTorch.
"""
from __future__ import annotations

from dataclasses import dataclass
import os
from typing import List, Optional, Tuple

import torch

from .. import quant as Q
from . import reference as ref

_cuda = None
FORCE_REFERENCE = False     # run the plain-PyTorch restatement even for GPU tensors (oracle for end-to-end tests)


def on_gpu(t: torch.Tensor) -> bool:
    """True when ``t`` should go to the sm_100a kernels."""
    return t.is_cuda and not FORCE_REFERENCE


def cuda_ops():
    """The ctypes binding module for the kernel library (loaded on first GPU use)."""
    global _cuda
    if _cuda is None:
        from . import cuda as _c
        _c.load()
        _cuda = _c
    return _cuda


# ----------------------------------------------------------------------------- weights / activations
@dataclass
class LinearWeight:
    """One (possibly quantized) ``[N,K]`` projection.

    kind ``dense``: ``weight [N,K]`` in the model dtype.
    kind ``fp8_block``: ``weight [N,K]`` e4m3, ``scale [ceil(N/128), ceil(K/128)]`` fp32.
    kind ``nvfp4``: ``weight [N,K/2]`` packed E2M1, ``scale [N,K/16]`` e4m3, ``gscale`` fp32, ``[1]`` or one per output row ``[N]``.
    """
    kind: str
    weight: torch.Tensor
    scale: Optional[torch.Tensor] = None
    gscale: Optional[torch.Tensor] = None
    bias: Optional[torch.Tensor] = None
    _dense_cache: Optional[torch.Tensor] = None

    @property
    def out_features(self) -> int:
        return self.weight.shape[0]

    @property
    def in_features(self) -> int:
        return self.weight.shape[1] * (2 if self.kind == "nvfp4" else 1)

    def dequantized(self) -> torch.Tensor:
        if self.kind == "dense":
            return self.weight
        if self.kind == "fp8_block":
            return Q.dequantize_fp8_block(self.weight, self.scale)
        return Q.dequantize_nvfp4(self.weight, self.scale, self.gscale)

    @staticmethod
    def from_dense(w: torch.Tensor, kind: str, bias=None) -> "LinearWeight":
        if kind in ("dense", "none"):
            return LinearWeight("dense", w.contiguous(), bias=bias)
        if kind == "fp8_block":
            q, s = Q.quantize_fp8_block(w)
            return LinearWeight("fp8_block", q, s, bias=bias)
        if kind == "nvfp4":
            p, s, g = Q.quantize_nvfp4(w)
            return LinearWeight("nvfp4", p, s, g, bias=bias)
        raise ValueError(kind)


@dataclass
class Act:
    """Activation handle: plain ``x [T,K]`` and/or its FP8 group-quantized form ``(q, s)``."""
    x: Optional[torch.Tensor] = None
    q: Optional[torch.Tensor] = None
    s: Optional[torch.Tensor] = None
    dtype: Optional[torch.dtype] = None      # dtype of the tensor the quantised form was made from
    # rows still arriving from other ranks (sequence-parallel all-gather): (flags address, epoch address, wait cycles);
    # the consuming GEMM polls the flags tile by tile (parallel/seqpar.py)
    ready: Optional[tuple] = None
    # deferred RMSNorm factor: ``(q, s)`` hold ``residual * norm_weight`` and every row still has to be multiplied by
    # rsqrt(sum over parts of sums[part, row] / H + eps); tuple ``(sums [parts, rows_pad] fp32, parts, H, eps)``.  The
    # factor commutes with a linear layer, so the consuming GEMM applies it to its output rows.
    row_ss: Optional[tuple] = None

    @property
    def out_dtype(self) -> torch.dtype:
        return self.x.dtype if self.x is not None else (self.dtype or torch.bfloat16)

    def plain(self) -> torch.Tensor:
        if self.x is None:
            x = (self.q.float().view(self.q.shape[0], -1, 128) * self.s[..., None]).view(self.q.shape)
            if self.row_ss is not None:
                sums, parts, h, eps = self.row_ss
                x = x * torch.rsqrt(sums[:parts, :x.shape[0]].sum(0) / h + eps)[:, None]
            self.x = x.to(self.out_dtype)
        return self.x

    def fp8(self) -> Tuple[torch.Tensor, torch.Tensor]:
        if self.q is None:
            self.q, self.s = quant_fp8(self.x)
        return self.q, self.s


@dataclass
class StreamDelta:
    """What the last sublayer leaves for the residual streams (``layers/hyper.py``).

    Start of the model (``conn`` is None): every stream becomes ``y * scale``.  Otherwise the streams are rewritten with the
    sublayer's connection ``conn`` and its output ``y``, or, with ``y2``, half the sum of ``y`` and ``y2`` after an RMS norm
    each with the weights ``w1`` / ``w2``."""
    y: torch.Tensor
    conn: Optional[object] = None            # layers.hyper.HyperConnection
    scale: float = 1.0
    y2: Optional[torch.Tensor] = None
    w1: Optional[torch.Tensor] = None
    w2: Optional[torch.Tensor] = None


def hyper_norm(streams: Optional[torch.Tensor], delta: StreamDelta, read: torch.Tensor, norm_w: torch.Tensor, eps: float,
               write: bool = True) -> Tuple[torch.Tensor, torch.Tensor]:
    """Apply ``delta`` to ``streams [T, S, W]`` (fp32, in place; None at the start), read ``u = sum_s read[s] * streams[s]``
    and return ``(rmsnorm(u) * norm_w, streams)``.  ``write=False`` leaves the streams as they are (last read of a step)."""
    if on_gpu(delta.y):
        return cuda_ops().hyper_norm(streams, delta, read, norm_w, eps, write)
    return ref.hyper_norm(streams, delta, read, norm_w, eps)


@dataclass
class ExpertRows:
    """Expert outputs before their weighted sum: ``y`` holds one row per (token, choice) pair, ``slot_of [T * k]`` the row of each
    pair (-1: nothing to add), ``w [T, k]`` its weight; ``extra [T, W]`` joins the sum as it is (shared expert)."""
    y: torch.Tensor
    slot_of: torch.Tensor
    w: torch.Tensor
    extra: Optional[torch.Tensor] = None


@dataclass
class DepthSum:
    """Weighted sums over the results of all layers: the stream that a delta leaves becomes entry ``index`` of ``history
    [entries, T, W]`` (fp32), and what goes on is ``sum_j factors[j] * history[j]``, ``j = 0 .. index``, or, without ``factors``, the
    entry as it is."""
    history: torch.Tensor
    index: int
    factors: Optional[torch.Tensor] = None   # fp32 [index + 1]


@dataclass
class NormDelta:
    """What the last sublayer leaves for an fp32 residual stream: ``stream += rmsnorm(y) * norm``, or ``stream += y`` without
    ``norm``, with ``y`` given as it is or as :class:`ExpertRows`.  Start of the model (no stream yet): the stream is
    ``y * scale``.  With ``bias`` the norm is a layer norm (mean taken off, bias added); ``gate [T, W]`` multiplies ``y`` by its
    sigmoid first; ``depth`` replaces the new stream by a sum over the layers' results."""
    y: object
    norm: Optional[torch.Tensor] = None
    scale: float = 1.0
    bias: Optional[torch.Tensor] = None
    gate: Optional[torch.Tensor] = None
    depth: Optional[DepthSum] = None


def add_normed(stream: Optional[torch.Tensor], delta: NormDelta, eps: float, plus_one: bool, out_norm: Optional[torch.Tensor] = None,
               write: bool = True, step: Optional[torch.Tensor] = None, out_bias: Optional[torch.Tensor] = None) -> Tuple[torch.Tensor, torch.Tensor]:
    """Apply ``delta`` and then the vector ``step`` (fp32 ``[W]``) to ``stream [T, W]`` (fp32, in place; None at the start) and
    return ``(h, stream)``: ``h`` is the stream in the activations' dtype, normed with ``out_norm`` where one is given (a layer norm
    with ``out_bias``).  ``write=False`` leaves the stream, and the history of a :class:`DepthSum`, as they are."""
    y = delta.y.y if isinstance(delta.y, ExpertRows) else delta.y
    if on_gpu(y):
        return cuda_ops().add_normed(stream, delta, eps, plus_one, out_norm, write, step, out_bias)
    return ref.add_normed(stream, delta, eps, plus_one, out_norm, write, step, out_bias)


# ----------------------------------------------------------------------------- elementwise / norm
def quant_fp8(x: torch.Tensor, group: int = 128):
    if on_gpu(x):
        return cuda_ops().quant_fp8(x, group)
    return Q.per_token_group_quant_fp8(x, group)


def rmsnorm(x, w, eps, residual=None, plus_one=False):
    if on_gpu(x):
        return cuda_ops().rmsnorm(x, w, eps, residual, plus_one, quant=False)
    return ref.rmsnorm(x, w, eps, residual, plus_one)


def rmsnorm_act(x, w, eps, residual=None, plus_one=False, want_fp8=False) -> Tuple[Act, Optional[torch.Tensor]]:
    """Residual add + RMSNorm, emitting FP8 group-quantized activations when the consumer is an FP8 GEMM."""
    if want_fp8 and x.shape[-1] % 128 == 0:
        if on_gpu(x):
            q, s, r = cuda_ops().rmsnorm(x, w, eps, residual, plus_one, quant=True)
        else:
            q, s, r = ref.rmsnorm_quant_fp8(x, w, eps, residual, plus_one)
        return Act(q=q, s=s, dtype=x.dtype), r
    y, r = rmsnorm(x, w, eps, residual, plus_one)
    return Act(x=y), r


def relu_squared(x: torch.Tensor) -> torch.Tensor:
    """``relu(x) ** 2`` (the activation of Nemotron-H's two-projection MLP)."""
    if on_gpu(x) and x.dtype == torch.bfloat16 and x.stride(-1) == 1:
        return cuda_ops().relu_squared(x)
    return torch.relu(x).square()


def glu_act(gate_up: torch.Tensor, want_fp8=False, kind: str = "silu") -> Act:
    """``act(gate) * up`` with ``kind`` in {silu, gelu_tanh}."""
    if kind == "silu":
        return silu_mul_act(gate_up, want_fp8)
    inter = gate_up.shape[-1] // 2
    gpu = on_gpu(gate_up) and gate_up.dtype == torch.bfloat16
    if want_fp8 and inter % 128 == 0:
        if gpu:
            q, s = cuda_ops().gelu_tanh_mul(gate_up, quant=True)
        else:
            q, s = Q.per_token_group_quant_fp8(ref.gelu_tanh_mul(gate_up), 128)
        return Act(q=q, s=s, dtype=gate_up.dtype)
    return Act(x=cuda_ops().gelu_tanh_mul(gate_up) if gpu else ref.gelu_tanh_mul(gate_up))


SILU_UNIT = (float("inf"), 1.0, 0.0)        # silu(gate) * up as a gated unit


def gated_unit_act(gate_up: torch.Tensor, unit: Tuple[float, float, float], paired: bool = False) -> Act:
    """``g * sigmoid(alpha * g) * (u + shift)`` with ``unit = (limit, alpha, shift)``, ``g = min(gate, limit)`` and ``u = clamp(up,
    -limit, limit)`` of ``[gate | up]``, or with ``paired`` of alternating gate and up columns."""
    if on_gpu(gate_up):
        return Act(x=cuda_ops().gated_unit(gate_up, unit, paired))
    return Act(x=ref.gated_unit(gate_up, unit, paired))


def linear_gated_unit(a, w: LinearWeight, unit: Tuple[float, float, float]) -> Act:
    """:func:`gated_unit_act` of a projection whose gate and up rows alternate; one kernel for unquantised bf16 weights."""
    x = a.plain() if isinstance(a, Act) else a
    if w.kind == "dense" and w.bias is None and on_gpu(x) and x.dtype == torch.bfloat16 and x.shape[1] % 8 == 0:
        return Act(x=cuda_ops().gemm_bf16(x, w.weight, unit=unit))
    return gated_unit_act(linear(a, w), unit, paired=True)


def linear_gated_unit_tail(a, w: LinearWeight, unit: Tuple[float, float, float], n_main: int) -> Tuple[Act, torch.Tensor]:
    """:func:`linear_gated_unit` of the first ``n_main`` rows and, from the same product, the others as fp32 sums (bf16 weights on a
    GPU, ``n_main`` a multiple of 16)."""
    y, tail = cuda_ops().gemm_bf16(a.plain() if isinstance(a, Act) else a, w.weight, unit=unit, n_main=n_main)
    return Act(x=y), tail


def tanh_(x: torch.Tensor) -> torch.Tensor:
    """``tanh`` in place."""
    if on_gpu(x):
        return cuda_ops().tanh_(x)
    return x.tanh_()


def group_norm_gate(y: torch.Tensor, z: torch.Tensor, w: torch.Tensor, group: int, eps: float, gate_first: bool, gate: str = "silu",
                    den: Optional[torch.Tensor] = None) -> torch.Tensor:
    """RMS norm over groups of ``group`` channels joined with a gate: ``norm(y * gate(z)) * w`` with ``gate_first`` (Mamba-2),
    ``norm(y) * w * gate(z)`` otherwise (WKV, mLSTM); ``gate`` is silu or sigmoid.  ``z`` may be a column slice.  ``den [T, groups]``
    (fp32) divides every group of ``y`` first."""
    if on_gpu(y):
        return cuda_ops().group_norm_gate(y, z, w, group, eps, gate_first, gate, den)
    return ref.group_norm_gate(y, z, w, group, eps, gate_first, gate, den)


def head_gate(x: torch.Tensor, g: torch.Tensor) -> torch.Tensor:
    """``x [T, H, D]`` times ``sigmoid(g [T, H])`` (fp32 gate numbers; in place on the GPU)."""
    if on_gpu(x):
        return cuda_ops().head_gate(x, g)
    return (x.float() * torch.sigmoid(g.float())[..., None]).to(x.dtype)


def silu_mul_act(gate_up: torch.Tensor, want_fp8=False) -> Act:
    inter = gate_up.shape[-1] // 2
    if want_fp8 and inter % 128 == 0:
        if on_gpu(gate_up):
            q, s = cuda_ops().silu_mul(gate_up, quant=True)
        else:
            q, s = ref.silu_mul_quant_fp8(gate_up)
        return Act(q=q, s=s, dtype=gate_up.dtype)
    if on_gpu(gate_up):
        if gate_up.dtype == torch.float32 or inter % 8:
            return gated_unit_act(gate_up, SILU_UNIT)
        return Act(x=cuda_ops().silu_mul(gate_up, quant=False))
    return Act(x=ref.silu_mul(gate_up))


# ----------------------------------------------------------------------------- GEMM
def linear(a, w: LinearWeight, out: Optional[torch.Tensor] = None) -> torch.Tensor:
    """``y = a @ W^T (+ bias)``; ``a`` is a tensor or an :class:`Act`."""
    act = a if isinstance(a, Act) else Act(x=a)
    dev_cuda = on_gpu(act.x if act.x is not None else act.q)
    if w.kind == "fp8_block" and act.row_ss is not None and dev_cuda:
        y = cuda_ops().gemm_fp8_fused(act.q, act.s, w.weight, w.scale, mode=0, out=out, ss_in=act.row_ss, ready=act.ready)
    elif w.kind == "fp8_block":
        if act.row_ss is not None:
            act = Act(x=act.plain())
        q, s = act.fp8()
        if dev_cuda:
            y = cuda_ops().gemm_fp8_block(q, s, w.weight, w.scale, out=out, ready=act.ready)
        else:
            y = Q.fp8_block_gemm_ref(q, s, w.weight, w.scale, out_dtype=act.out_dtype)
    elif w.kind == "nvfp4":
        x = act.plain()
        w4a4 = NVFP4_ACTIVATIONS and x.shape[-1] % 64 == 0
        if dev_cuda and w4a4:
            from . import cuda_fp4
            y = cuda_fp4.linear_w4a4(x, w, out=out)
        elif dev_cuda:
            y = cuda_ops().gemm_nvfp4(x, w.weight, w.scale, w.gscale, out=out)
        elif w4a4:
            y = (ref.quant_nvfp4_rowwise(x) @ w.dequantized().t()).to(x.dtype)
        else:
            y = (x.float() @ w.dequantized().t()).to(x.dtype)
    else:
        x = act.plain()
        if dev_cuda and x.dtype == torch.bfloat16 and w.weight.dtype == torch.bfloat16:
            return cuda_ops().gemm_bf16(x, w.weight, out=out, bias=w.bias)
        return torch.nn.functional.linear(x, w.weight, w.bias)
    if w.bias is not None:
        y = y + w.bias
    return y


def linear_relu2(a, w: LinearWeight, n_act: Optional[int] = None) -> torch.Tensor:
    """``a @ W^T (+ bias)`` with the first ``n_act`` columns (all of them by default) as ``relu(.) ** 2``; one kernel for unquantised bf16
    weights with a bias."""
    x = a.plain() if isinstance(a, Act) else a
    n_act = w.weight.shape[0] if n_act is None else n_act
    if w.kind == "dense" and w.bias is not None and on_gpu(x) and x.dtype == torch.bfloat16 and x.shape[1] % 8 == 0:
        return cuda_ops().gemm_bf16(x, w.weight, bias=w.bias, relu2_cols=n_act)
    y = linear(a, w)
    if n_act == y.shape[1]:
        return relu_squared(y)
    return torch.cat([torch.relu(y[:, :n_act]).square(), y[:, n_act:]], 1)


def linear_tail(a, w: LinearWeight, n_main: int) -> Tuple[torch.Tensor, torch.Tensor]:
    """``a @ W^T (+ bias)`` of an unquantised weight in two parts: the first ``n_main`` columns in the activations' dtype, the others as
    the fp32 sums that the product forms.  Returns ``(main, tail)``."""
    x = a.plain() if isinstance(a, Act) else a
    assert w.kind == "dense"
    if on_gpu(x) and x.dtype == torch.bfloat16:
        return cuda_ops().linear_tail(x, w.weight, n_main, w.bias)
    y = torch.nn.functional.linear(x.float(), w.weight.float(), None if w.bias is None else w.bias.float())
    return y[:, :n_main].to(x.dtype), y[:, n_main:]


# NVFP4 weights: quantise the activations to NVFP4 too and run the block-scaled FP4 x FP4 tensor-core GEMM (what an
# "NVFP4" ModelOpt checkpoint is calibrated for); off = weight-only (activations stay bf16)
NVFP4_ACTIVATIONS = os.environ.get("ATLAS_NVFP4_W4A4", "0") == "1"

FUSED_EPILOGUES = True      # tests switch this off to compare against the unfused kernel sequence


def swiglu_fusable(a, w: LinearWeight) -> bool:
    """The gate|up GEMM can apply SiLU * mul and the FP8 quantisation of its output in its own epilogue."""
    act = a if isinstance(a, Act) else Act(x=a)
    probe = act.x if act.x is not None else act.q
    return (FUSED_EPILOGUES and on_gpu(probe) and w.kind == "fp8_block" and w.bias is None and w.weight.shape[0] % 256 == 0
            and (w.weight.shape[0] // 2) % 128 == 0)


def linear_swiglu(a, w: LinearWeight) -> Act:
    """``silu(gate) * up`` of the stacked gate|up projection as FP8 group-quantised activations (one kernel)."""
    act = a if isinstance(a, Act) else Act(x=a)
    if act.row_ss is None:
        q, s = act.fp8()
    else:
        q, s = act.q, act.s
    qo, so = cuda_ops().gemm_fp8_fused(q, s, w.weight, w.scale, mode=1, ss_in=act.row_ss, ready=act.ready)
    return Act(q=qo, s=so, dtype=act.out_dtype)


def residual_norm_fusable(residual: torch.Tensor, w: LinearWeight) -> bool:
    """The projection ``w`` can add its output to ``residual`` and emit the normalised FP8 activations of the sum in its
    own epilogue.  (The projection's input never carries a deferred 1/rms factor: it is an attention output or an
    activation product, not a norm output.)"""
    return (FUSED_EPILOGUES and on_gpu(residual) and w.kind == "fp8_block" and w.bias is None and w.weight.shape[0] % 128 == 0
            and residual.dtype == torch.bfloat16 and residual.is_contiguous())


def linear_residual_norm(a, w: LinearWeight, residual: torch.Tensor, norm_w: torch.Tensor, eps: float, plus_one: bool):
    """``residual += a @ W^T`` (in place) and the FP8 form of ``residual * norm_w`` with the row's 1/rms factor left to
    the consumer (``Act.row_ss``): projection, residual add, RMSNorm and quantisation in one kernel."""
    act = a if isinstance(a, Act) else Act(x=a)
    q, s = act.fp8()
    qo, so, (sums, parts) = cuda_ops().gemm_fp8_fused(q, s, w.weight, w.scale, mode=2, residual=residual, norm_w=norm_w,
                                                      plus_one=plus_one, ready=act.ready)
    return Act(q=qo, s=so, dtype=residual.dtype, row_ss=(sums, parts, w.weight.shape[0], eps)), residual


# ----------------------------------------------------------------------------- attention
def qk_norm_rope_kv_write(q, k, v, positions, rope_cache, rotary_dim, k_cache, v_cache, slot_mapping,
                          k_scale=1.0, v_scale=1.0, q_norm_w=None, k_norm_w=None, eps=1e-6, norm_plus_one=False, rotate=False, norm_dim=0):
    """``rotate``: every q / k / v head goes through the orthonormal Walsh-Hadamard transform after RoPE, so the cache
    holds rotated keys and values (the "turbo8" cache: rotation + FP8) and the attention output comes out rotated too
    (``head_rotate`` takes it back).  ``norm_dim``: channels of a head that its norm counts (0 = all; the rest is zero padding)."""
    if on_gpu(q):
        return cuda_ops().qk_norm_rope_kv_write(q, k, v, positions, rope_cache, rotary_dim, k_cache, v_cache,
                                                slot_mapping, k_scale, v_scale, q_norm_w, k_norm_w, eps, norm_plus_one, rotate, norm_dim)
    return ref.qk_norm_rope_kv_write(q, k, v, positions, rope_cache, rotary_dim, k_cache, v_cache, slot_mapping,
                                     k_scale, v_scale, q_norm_w, k_norm_w, eps, norm_plus_one, rotate, norm_dim)


def qk_row_norm_kv_write(q, k, v, positions, rope_cache, rotary_dim, k_cache, v_cache, slot_mapping, seq_positions, q_norm_w, k_norm_w,
                         eps: float, nq: int, nk: int, temp: float = 0.0, temp_every: int = 1, sums: Optional[torch.Tensor] = None):
    """RMS norm of each row of ``q [T, Hq, D]`` and of ``k [T, Hkv, D]`` over all heads (``nq`` / ``nk`` channels, the rest is zero
    padding) with fp32 weights, rotation, queries times ``1 + temp * ln(floor((seq_positions + 1) / temp_every) + 1)``, paged
    cache write.  ``sums [T, 2]``: the rows' sums of squares where other ranks hold some of the heads."""
    if on_gpu(q):
        return cuda_ops().qk_row_norm_kv_write(q, k, v, positions, rope_cache, rotary_dim, k_cache, v_cache, slot_mapping, seq_positions,
                                               q_norm_w, k_norm_w, eps, nq, nk, temp, temp_every, sums)
    return ref.qk_row_norm_kv_write(q, k, v, positions, rope_cache, rotary_dim, k_cache, v_cache, slot_mapping, seq_positions, q_norm_w,
                                    k_norm_w, eps, nq, nk, temp, temp_every, sums)


def map_norm_kv_write(q, k, v, positions, rope_cache, rotary_dim, k_cache, v_cache, slot_mapping, q_norm_w, k_norm_w, eps: float):
    """Two maps per head: RMS norm (fp32 weights) and rotation of every map of ``q [T, H, 2, dim]`` and ``k [T, G, 2, dim]``.  Both maps'
    keys go side by side into one cache row, ``v [T, G, vdim]`` beside them; returns the query rows ``[T, 2 H, D]`` of the cache width
    ``D``: map 1 of head ``h`` in row ``2 h`` ahead of zeros, map 2 in row ``2 h + 1`` behind zeros, so that a row's product with a cache
    row is its own map's score."""
    if on_gpu(q):
        return cuda_ops().map_norm_kv_write(q, k, v, positions, rope_cache, rotary_dim, k_cache, v_cache, slot_mapping, q_norm_w, k_norm_w, eps)
    return ref.map_norm_kv_write(q, k, v, positions, rope_cache, rotary_dim, k_cache, v_cache, slot_mapping, q_norm_w, k_norm_w, eps)


def map_difference(a: torch.Tensor, dv: int, lam: float, rest: float, eps: float, gate: Optional[torch.Tensor] = None) -> torch.Tensor:
    """``a [T, 2 H, D]``, the outputs of two maps per head in their first ``dv`` columns -> ``[T, H * dv]``: ``o = a_1 - lam a_2``, RMS norm
    without a weight over a head's ``dv`` numbers, times ``rest`` and, with ``gate [T, H * dv]``, its sigmoid."""
    if on_gpu(a):
        return cuda_ops().map_difference(a, dv, lam, rest, eps, gate)
    return ref.map_difference(a, dv, lam, rest, eps, gate)


def gelu_embedding(z: torch.Tensor, table: torch.Tensor, ids: torch.Tensor, first: int, n: int) -> torch.Tensor:
    """``gelu_tanh(z[:, :n]) * table[ids, first : first + n]``, zeros in the columns of ``z`` from ``n`` on."""
    if on_gpu(z):
        return cuda_ops().gelu_embedding(z, table, ids, first, n)
    return ref.gelu_embedding(z, table, ids, first, n)


def head_rotate(x: torch.Tensor) -> torch.Tensor:
    """Orthonormal Walsh-Hadamard transform along the last (head) dimension of ``x [T, H, D]``; its own inverse."""
    if on_gpu(x) and x.shape[-1] == 128 and x.dtype == torch.bfloat16 and x.stride(2) == 1 and x.stride(1) == 128:
        return cuda_ops().wht_d128(x)
    return ref.head_rotate(x)


def paged_attention(q, k_cache, v_cache, batch, scale, k_scale=1.0, v_scale=1.0, sliding_window=None, chunk=0,
                    sinks=None, softcap=0.0, distance=None) -> torch.Tensor:
    """Attention of the step's query rows over the paged cache. ``batch`` is a ``ForwardBatch``.  ``chunk`` > 0: a token sees
    only keys of its own ``chunk``-token block of the sequence; ``sinks [Hq]``: ``exp(sink)`` joins the softmax denominator;
    ``softcap`` > 0: scores become ``softcap * tanh(score / softcap)``; ``distance [Hq, n]`` (fp32): column ``min(i - j, n - 1)``
    joins the scaled score of query ``i`` and key ``j``."""
    if on_gpu(q):
        return cuda_ops().paged_attention(q, k_cache, v_cache, batch, scale, k_scale, v_scale, sliding_window, chunk, sinks, softcap, distance)
    return ref.paged_attention(q, k_cache, v_cache, batch.block_tables, batch.seq_lens, batch.query_start_loc,
                               scale, k_scale, v_scale, sliding_window, chunk, sinks, softcap, distance)


def paged_attention_fp8_out(q, k_cache, v_cache, batch, scale, k_scale=1.0, v_scale=1.0, sliding_window=None) -> Optional[Act]:
    """Decode attention that hands its output over already group-quantised for an FP8 output projection (one kernel
    less per layer); None when the step / cache / head size is not covered and the caller takes the bf16 path."""
    if not (FUSED_EPILOGUES and on_gpu(q)):
        return None
    r = cuda_ops().paged_attention_q8(q, k_cache, v_cache, batch, scale, k_scale, v_scale, sliding_window)
    return None if r is None else Act(q=r[0], s=r[1], dtype=q.dtype)


# ----------------------------------------------------------------------------- MoE
def moe_route(logits, top_k, norm_topk, scoring="softmax", bias=None, n_group=0, topk_group=0, scale=1.0, hash_table=None,
              token_ids=None):
    if on_gpu(logits):
        return cuda_ops().moe_route(logits, top_k, norm_topk, scoring, bias, n_group, topk_group, scale, hash_table, token_ids)
    return ref.moe_route(logits, top_k, norm_topk, scoring, bias, n_group, topk_group, scale, hash_table, token_ids)


# ----------------------------------------------------------------------------- sampling
def argmax(logits: torch.Tensor, with_value: bool = False):
    if on_gpu(logits):
        return cuda_ops().argmax(logits, with_value)
    idx = ref.argmax_first(logits)
    if with_value:
        return idx, logits.float().gather(-1, idx[:, None])[:, 0]
    return idx


def sample(logits, temperature, top_k, top_p, min_p, uniform):
    if on_gpu(logits):
        return cuda_ops().sample(logits, temperature, top_k, top_p, min_p, uniform)
    return ref.sample(logits, temperature, top_k, top_p, min_p, uniform)


def logit_edits(logits: torch.Tensor, edits: torch.Tensor) -> None:
    """In-place sparse edits of fp32 ``logits [B, V]``.  ``edits`` is an int32 ``[n, 6]`` tensor of records
    ``(row, token, add, rep, sub, flags)`` with the three floats stored as their bit patterns; a (row, token) pair
    appears at most once.  Per record: ``x += add``; ``x = x / rep if x > 0 else x * rep``; ``x -= sub``; bit 0 of
    ``flags`` sets ``x = -inf``."""
    if edits.shape[0] == 0:
        return
    if on_gpu(logits):
        cuda_ops().logit_edits(logits, edits)
        return
    rows, toks = edits[:, 0].long(), edits[:, 1].long()
    add, rep, sub = (edits[:, i].view(torch.float32) for i in (2, 3, 4))
    x = logits[rows, toks] + add
    x = torch.where(rep != 1.0, torch.where(x > 0, x / rep, x * rep), x) - sub
    x = torch.where((edits[:, 5] & 1).bool(), torch.full_like(x, float("-inf")), x)
    logits[rows, toks] = x


def spec_accept(draft: torch.Tensor, target: torch.Tensor) -> torch.Tensor:
    """Greedy draft acceptance: ``draft [B, K]`` (-1 pads), ``target [B, K+1]`` -> accepted draft count per row."""
    if on_gpu(draft):
        return cuda_ops().spec_accept(draft, target)
    B, K = draft.shape
    ok = (draft == target[:, :K]) & (draft >= 0)
    return ok.long().cumprod(1).sum(1).to(torch.int32)
