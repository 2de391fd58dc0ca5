"""Sizes, models and kernel table of ``bench.py --design bisudra``.

Four layers of Bisudra (differential attention, a dense feed-forward and experts in turn) beside four attention layers of Kenovik with
the same feed-forward kinds, experts, projections of the same size (a head's two maps of 64 against one of 128, values of 128) and the
same cache bytes per token.  What Bisudra's gates cost in parameters goes to the other model's dense feed-forward.
"""
from __future__ import annotations

from types import SimpleNamespace
from typing import List

import torch

# attn: heads, kv heads, map size, value size; moe: experts, per token, hidden size; ff: Bisudra's dense hidden size
SIZES = {
    "2048": dict(width=2048, attn=(16, 4, 64, 128), moe=(64, 6, 1408), ff=9216),
    "4096": dict(width=4096, attn=(32, 8, 64, 128), moe=(64, 6, 2048), ff=18432),
}
VOCAB, WINDOW, TAPS, SIDE, PATTERN = 32768, 4096, 4, 128, "dede"


def bisudra(size: str):
    from ..config import _bisudra
    s = SIZES[size]
    h, g, d, dv = s["attn"]
    return _bisudra(VOCAB, s["width"], PATTERN, (h, g, d, dv, d, WINDOW), s["ff"], s["moe"], TAPS, SIDE, "bfloat16")


def beside(size: str):
    from ..config import kenovik_config
    s = SIZES[size]
    W, (h, g, _, dv), (E, top, I) = s["width"], s["attn"], s["moe"]
    mixer = {"heads": h, "kv_heads": g, "dim": dv, "vdim": dv, "scale": dv ** -0.5, "rot": {"base": 5e5, "dims": dv}}
    moe = {"kind": "moe", "expert": {"ff": I, "limit": 7.0}, "shared": None, "router": {"experts": E, "top": top, "scale": 1.0}}
    dense = {"kind": "dense", "ff": s["ff"] * 2 // 3 + 2 * W}
    return kenovik_config({"vocab": VOCAB, "width": W, "norm": {"eps": 1e-6}, "embedding": {"scale": W ** 0.5}, "dtype": "bfloat16", "loop": None,
                           "layers": [{"type": "attention", "mixer": mixer, "mlp": dense if ch == "d" else moe} for ch in PATTERN]})


def kernel_table(size: str, timer, peaks) -> List[dict]:
    """Time and fraction of the roofline (bytes the kernels must move at the measured copy bandwidth, or their products at the
    measured bf16 rate, the slower of both) of every kernel of the new layers, each beside the like kernel of the other model."""
    from .. import ops
    from ..layers import DenseMLP, InputConvolution, MoE, ParallelCtx, TokenSide
    from ..models import ForwardBatch
    from ..ops import Act, cuda as K, cuda_recurrent as R, reference as ref
    s = SIZES[size]
    W = s["width"]
    dev, bf = "cuda", torch.bfloat16
    gen = torch.Generator(device=dev).manual_seed(0)
    rn = lambda *sh, dt=bf, std=1.0: (torch.randn(*sh, generator=gen, device=dev) * std).to(dt)
    ours, theirs = bisudra(size), beside(size)
    p = ParallelCtx()
    rows: List[dict] = []

    def add(pair: str, who: str, shape: str, fn, nbytes: float, flops: float = 0.0):
        us = timer.time(fn) * 1e3
        ideal = max(nbytes / peaks["hbm_gbs"] / 1e3, flops / peaks["bf16_tflops"] / 1e6)
        rows.append({"pair": pair, "kernel": who, "shape": shape, "us": round(us, 1), "roofline": round(ideal / us, 3)})

    (h, g, dm, dv), (E, top, I), F = s["attn"], s["moe"], s["ff"]
    moe_a, moe_b = MoE(ours.for_layer(1), p, "dense", "dense"), MoE(theirs.for_layer(1), p, "dense", "dense")
    mlp_a, mlp_b = DenseMLP(ours.for_layer(0), p, "dense"), DenseMLP(theirs.for_layer(0), p, "dense", paired=True)
    for m in (moe_a, moe_b, mlp_a, mlp_b):
        m.init_random(gen, 0.02, bf, dev)
    moe_b.fuse_inputs()
    Fb = theirs.for_layer(0).intermediate_size
    conv, side = InputConvolution(W, TAPS), TokenSide(W, SIDE, 1, "dense")
    conv.init_random(gen, bf, dev)
    side.init_random(gen, 0.02, bf, dev)
    side.table = rn(VOCAB, 4 * SIDE)
    fused = ops.LinearWeight("dense", torch.cat([mlp_a.gate_up.weight, rn(W, W, std=0.02)], 0).contiguous(), bias=torch.zeros(F + W, device=dev))
    routed = ops.LinearWeight("dense", torch.cat([rn(W, W, std=0.02), moe_a.router.weight], 0).contiguous(), bias=torch.zeros(E + W, device=dev))
    plain = ops.LinearWeight("dense", fused.weight)
    for T, nseq in ((8192, 8), (8192, 1), (128, 128), (1, 1)):
        decode = T == nseq
        shape, lens = f"{T} rows, {nseq} seq", [T // nseq] * nseq
        b = SimpleNamespace(query_lens_host=lens, state_slots_host=list(range(nseq)), has_state_host=[True] * nseq, snapshot_plan={}, spec_verify=False)
        used = min(E, T * top)
        # ---- residual and norms
        y, z, x = rn(T, W), rn(T, W), rn(T, W, dt=torch.float32)
        nw, nb, hist, fac = torch.ones(W, device=dev), torch.zeros(W, device=dev), rn(5, T, W, dt=torch.float32), torch.full((5,), 0.2, device=dev)
        act = Act(x=y)
        add("norm", "gate, layer norm on the residual", shape, lambda: ops.add_normed(x, ops.NormDelta(y, nw, bias=nb, gate=z), 1e-6, False), T * W * 14)
        add("norm", "rms norm, sum over five results", shape, lambda: ops.add_normed(x, ops.NormDelta(y, nw, depth=ops.DepthSum(hist, 4, fac)), 1e-6, False), T * W * 32)
        add("norm", "add_normed (existing)", shape, lambda: ops.add_normed(x, ops.NormDelta(y), 1e-6, False, nw), T * W * 12)
        pr, slots, pw = rn(T * top, W), torch.randperm(T * top, generator=gen, device=dev).to(torch.int32), torch.rand(T, top, device=dev)
        er = ops.ExpertRows(pr, slots, pw)
        add("norm", "gate, layer norm of expert rows", shape, lambda: ops.add_normed(x, ops.NormDelta(er, nw, bias=nb, gate=z), 1e-6, False), T * W * (12 + 2 * top))
        add("norm", "add_normed of expert rows (existing)", shape, lambda: ops.add_normed(x, ops.NormDelta(er), 1e-6, False, nw), T * W * (10 + 2 * top))
        # ---- convolution
        st, meta, out = conv.alloc_state(nseq, dev, bf), R.step_meta(b, dev), torch.empty_like(y)
        win = st["inputs"]
        add("convolution", "input convolution, window", shape, lambda: conv.forward(y, b, st), T * W * 4 + nseq * W * (TAPS - 1) * 4)

        def plain_conv():
            K._check(R._lib().atlas_conv1d_bias_silu(y.data_ptr(), W, conv.w.data_ptr(), None, W, TAPS, win.data_ptr(), meta.seq_of.data_ptr(), meta.qsl.data_ptr(),
                                                     meta.slots.data_ptr(), meta.has.data_ptr(), out.data_ptr(), W, T, 1, 0, K._stream()), "conv1d")
            R._input_conv_state(conv, y, meta, win)
        add("convolution", "conv1d, silu, window (existing)", shape, plain_conv, T * W * 4 + nseq * W * (TAPS - 1) * 4)
        # ---- products
        pb, pf = T * W * 2 + 2 * (F + W) * W + T * (F + W) * 2, 2.0 * T * W * (F + W)
        add("projection", "up (squared relu) and gate, biases", shape, lambda: ops.linear_relu2(act, fused, F), pb, pf)
        add("projection", "linear (existing)", shape, lambda: ops.linear(act, plain), pb, pf)
        add("feed-forward", "squared relu, biases", shape, lambda: mlp_a.forward(act), T * W * 4 + 4 * W * F, 4.0 * T * W * F)
        add("feed-forward", "silu, unit in the product (existing)", shape, lambda: mlp_b.forward(act), T * W * 4 + 6 * W * Fb, 6.0 * T * W * Fb)
        add("router", "gate and fp32 logits with bias, softmax", shape, lambda: ops.moe_route(ops.linear_tail(act, routed, W)[1], top, True),
            T * W * 4 + (E + W) * W * 2, 2.0 * T * W * (E + W))
        add("router", "fp32 logits, sigmoid (existing)", shape,
            lambda: ops.moe_route(ops.linear_tail(act, moe_b.router, 0)[1], top, True, "sigmoid", moe_b.router_bias, 1, 1, 1.0), T * W * 2 + E * W * 2)
        eb, ef = T * W * 2 + used * 6 * I * W + T * top * W * 2, 6.0 * T * top * W * I
        add("experts", "router, silu experts, rows", shape, lambda: moe_a.forward(act, rows_ok=True), eb, ef)
        add("experts", "router, clamped experts, rows (existing)", shape, lambda: moe_b.forward(act, rows_ok=True), eb, ef)
        ids = torch.randint(0, VOCAB, (T,), generator=gen, device=dev)
        zz = rn(T, SIDE)
        add("token input", "gate product, gelu x embedding, product", shape, lambda: side.forward(act, ids), T * W * 4 + 4 * SIDE * W + T * SIDE * 2, 4.0 * T * W * SIDE)
        ga, gb = side.gate, side.proj
        add("token input", "two products of that size (existing)", shape, lambda: ops.linear(ops.linear(act, ga), gb), T * W * 4 + 4 * SIDE * W, 4.0 * T * W * SIDE)
        add("token input", "gelu x embedding", shape, lambda: ops.gelu_embedding(zz, side.table, ids, SIDE, SIDE), T * SIDE * 6)
        # ---- attention
        ctx = 2048 if decode else 0
        per = (ctx + lens[0] + 15) // 16
        fb = ForwardBatch.build([[0] * lens[0]] * nseq, [ctx] * nseq, [list(range(i * per, (i + 1) * per)) for i in range(nseq)], 16, device=dev)
        L = ctx + lens[0]
        seen = lambda w: min(L, w) if decode else (w * w / 2 + (L - w) * w) / L if w < L else L / 2        # keys per row, on average
        nq, nk, nv = 2 * h * dm, 2 * g * dm, g * dv
        qkvg = rn(T, nq + nk + nv + h * dv)
        q, k, v, gate = qkvg.split([nq, nk, nv, h * dv], 1)
        kc, vc = K.alloc_kv_cache(per * nseq, 16, g, dv, bf, dev)
        table = ref.build_rope_cache(dm, 16384, 5e5, None, dev)
        wide = ref.build_rope_cache(dv, 16384, 5e5, None, dev)
        qw, hw = torch.ones(dm, device=dev), torch.zeros(dv, device=dev, dtype=bf)
        add("cache write", "map norms, rotation, packed keys", shape,
            lambda: ops.map_norm_kv_write(q.view(T, h, 2, dm), k.view(T, g, 2, dm), v.view(T, g, dv), fb.positions, table, dm, kc, vc, fb.slot_mapping, qw, qw, 1e-6),
            T * (3 * nq + 2 * nk + 2 * nv) * 2 + T * dm * 4)
        add("cache write", "head norms, rotation (existing)", shape,
            lambda: ops.qk_norm_rope_kv_write(q.view(T, h, dv), k.view(T, g, dv), v.view(T, g, dv), fb.positions, wide, dv, kc, vc, fb.slot_mapping, 1.0, 1.0, hw, hw, 1e-6, True),
            T * (2 * nq + 2 * nk + 2 * nv) * 2 + T * dv * 4)
        qa, qb = rn(T, 2 * h, dv), rn(T, h, dv)
        cache = nseq * g * dv * 4 * L
        add("attention", "two maps per head", shape, lambda: ops.paged_attention(qa, kc, vc, fb, dm ** -0.5, sliding_window=WINDOW), T * 2 * h * dv * 4 + cache,
            T * seen(WINDOW) * h * (4.0 * dm + 4.0 * dv))
        add("attention", "two maps per head, window 256", shape, lambda: ops.paged_attention(qa, kc, vc, fb, dm ** -0.5, sliding_window=256),
            T * 2 * h * dv * 4 + (cache if not decode else nseq * g * dv * 4 * 256), T * seen(256) * h * (4.0 * dm + 4.0 * dv))
        add("attention", "causal (existing)", shape, lambda: ops.paged_attention(qb, kc, vc, fb, dv ** -0.5), T * h * dv * 4 + cache, T * seen(L) * h * 4.0 * dv)
        a, hg = rn(T, 2 * h, dv), rn(T, h, dt=torch.float32)
        add("output gate", "difference, norm, gate", shape, lambda: ops.map_difference(a, dv, 0.5, 0.7, 1e-6, gate), T * h * dv * 8)
        add("output gate", "head gate (existing)", shape, lambda: ops.head_gate(qb, hg), T * h * dv * 4)
        del kc, vc, qa, qb, qkvg, pr, er, a, hist
        torch.cuda.empty_cache()
    return rows
