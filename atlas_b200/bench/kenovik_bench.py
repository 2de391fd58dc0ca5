"""Sizes, models and kernel table of ``bench.py --design kenovik``.

Four layers of Kenovik (RG-LRU, attention with a fixed sink, attention with a distance bias, RG-LRU; the first one with a dense
feed-forward, the others with experts and a shared expert) beside four layers of Qwen3-Next with the same heads, experts and
recurrent channels: Gated DeltaNet whose value channels are the RG-LRU's, plain attention on a bf16 cache, SwiGLU experts.
"""
from __future__ import annotations

from types import SimpleNamespace
from typing import List

import torch

# lru: channels, blocks; gdn: key heads, value heads, head size (value channels = lru channels); attn: heads, kv heads, size;
# moe: experts, per token, hidden size
SIZES = {
    "2048": dict(width=2048, lru=(2560, 10), gdn=(10, 20, 128), attn=(16, 2, 128), moe=(64, 6, 1408), ff=6144),
    "4096": dict(width=4096, lru=(4096, 16), gdn=(16, 32, 128), attn=(32, 8, 128), moe=(64, 6, 2048), ff=12288),
}
VOCAB, REACH, ROWS, GROUPS, KEEP = 32768, 1024, 32, 8, 4


def kenovik(size: str):
    from ..config import _kenovik
    s = SIZES[size]
    hq, hkv, d = s["attn"]
    return _kenovik(VOCAB, s["width"], "Radr", s["lru"], (hq, hkv, d, d, d // 2), (hq, hkv, d, d, REACH), s["ff"], s["moe"] + (GROUPS, KEEP), None, "bfloat16")


def beside(size: str):
    from ..config import ModelConfig, QuantConfig
    s = SIZES[size]
    (hq, hkv, d), (hk, hv, dk), (E, top, I) = s["attn"], s["gdn"], s["moe"]
    return ModelConfig(model_type="qwen3_next", family="hybrid", vocab_size=VOCAB, hidden_size=s["width"], intermediate_size=s["ff"],
                       num_hidden_layers=4, num_attention_heads=hq, num_key_value_heads=hkv, head_dim=d, rope_theta=1e7, tie_word_embeddings=True,
                       partial_rotary_factor=0.5, qk_norm=True, attn_output_gate=False, norm_plus_one=True, num_experts=E,
                       num_experts_per_tok=top, moe_intermediate_size=I, shared_expert_intermediate_size=I, norm_topk_prob=True, mlp_only_layers=[0],
                       layer_types=["linear_attention", "full_attention", "full_attention", "linear_attention"], linear_num_key_heads=hk,
                       linear_num_value_heads=hv, linear_key_head_dim=dk, linear_value_head_dim=dk, quant=QuantConfig(kv_cache_dtype="bf16"))


def kernel_table(size: str, timer, peaks) -> List[dict]:
    """Time and fraction of the roofline (bytes the kernels must move at the measured copy bandwidth, or their products at the
    measured bf16 rate, the slower of both) of every kernel of the new layers, each beside the like kernel of the other model."""
    from .. import ops
    from ..layers import DenseMLP, GatedDeltaNet, MoE, ParallelCtx, RGLRUMixer
    from ..layers.attention import distance_table
    from ..models import ForwardBatch
    from ..ops import Act, cuda as K, reference as ref
    s = SIZES[size]
    W = s["width"]
    dev, bf = "cuda", torch.bfloat16
    gen = torch.Generator(device=dev).manual_seed(0)
    rn = lambda *sh, dt=bf, std=1.0: (torch.randn(*sh, generator=gen, device=dev) * std).to(dt)
    ours, qwen = kenovik(size), beside(size)
    p = ParallelCtx()
    rows: List[dict] = []

    def add(pair: str, who: str, shape: str, fn, nbytes: float, flops: float = 0.0):
        us = timer.time(fn) * 1e3
        ideal = max(nbytes / peaks["hbm_gbs"] / 1e3, flops / peaks["bf16_tflops"] / 1e6)
        rows.append({"pair": pair, "kernel": who, "shape": shape, "us": round(us, 1), "roofline": round(ideal / us, 3)})

    (C, blocks), (hk, hv, dk), (E, top, I), ff = s["lru"], s["gdn"], s["moe"], s["ff"]
    n = C // blocks
    lru, gd = RGLRUMixer(ours.for_layer(0), 0, p, "dense"), GatedDeltaNet(qwen, 0, p, "dense")
    moe_a, moe_b = MoE(ours.for_layer(1), p, "dense", "dense"), MoE(qwen, p, "dense", "dense")
    mlp_a, mlp_b = DenseMLP(ours.for_layer(0), p, "dense", paired=True), DenseMLP(qwen, p, "dense", activation="silu_glu")
    for m in (lru, gd, moe_a, moe_b, mlp_a, mlp_b):
        m.init_random(gen, 0.02, bf, dev)
    moe_a.fuse_inputs()
    for T, nseq in ((8192, 8), (8192, 1), (128, 128), (1, 1)):
        decode = T == nseq
        shape, lens = f"{T} rows, {nseq} seq", [T // nseq] * nseq
        b = SimpleNamespace(query_lens_host=lens, state_slots_host=list(range(nseq)), has_state_host=[True] * nseq, snapshot_plan={}, spec_verify=False)
        act, used = None, min(E, T * top)
        # ---- residual and norm
        y, x, nw, step = rn(T, W), rn(T, W, dt=torch.float32), torch.ones(W, device=dev), torch.zeros(W, device=dev)
        act = Act(x=y)
        add("norm", "add_normed", shape, lambda: ops.add_normed(x, ops.NormDelta(y), 1e-6, False, nw), T * W * 12)
        add("norm", "add_normed with a step vector", shape, lambda: ops.add_normed(x, ops.NormDelta(y), 1e-6, False, nw, step=step), T * W * 12)
        pr, slots, pw = rn(T * top, W), torch.randperm(T * top, generator=gen, device=dev).to(torch.int32), torch.rand(T, top, device=dev)
        sh = rn(T, W)
        er = ops.ExpertRows(pr, slots, pw, sh)
        add("norm", "add_normed of expert and shared rows", shape, lambda: ops.add_normed(x, ops.NormDelta(er), 1e-6, False, nw), T * W * (12 + 2 * top))
        nwb, out, res = nw.to(bf), torch.empty(T, W, dtype=bf, device=dev), rn(T, W)
        add("norm", "rmsnorm + residual (existing)", shape, lambda: ops.rmsnorm(y, nwb, 1e-6, res, True), T * W * 8)

        def combine_then_norm():
            K._check(K.lib().atlas_moe_combine(pr.data_ptr(), W, slots.data_ptr(), pw.data_ptr(), T, top, W, None, 0, out.data_ptr(), W, K._stream()), "moe_combine")
            K.shared_expert_blend(out, sh, y, moe_b.shared_gate)
            ops.rmsnorm(out, nwb, 1e-6, res, True)
        add("norm", "combine, blend, rmsnorm + residual (existing)", shape, combine_then_norm, T * W * (12 + 2 * top))
        # ---- recurrence: convolution, gates, scan, output gate, window
        yx = rn(T, 2 * C)
        st = lru.alloc_state(nseq, dev, bf)
        add("recurrence", "rglru conv + gates + scan + window", shape, lambda: K.rglru_forward(lru, yx[:, :C], yx[:, C:], b, st, True),
            T * C * 6 + nseq * C * (8 + 12) + 4 * C * n, 4.0 * T * C * n)
        Cg = gd.conv_dim
        proj = rn(T, Cg + 2 * hv)
        gs = gd.alloc_state(nseq, dev, bf)
        gflops = T * hv * (4.0 * 64 * dk + 2.0 * 64 * dk + 6.0 * dk * dk) if not decode else 0.0
        add("recurrence", "gdn conv + memory + window (existing)", shape,
            lambda: K.gdn_forward(gd, proj[:, :Cg], proj[:, Cg:Cg + hv], proj[:, Cg + hv:], b, gs, True), T * (Cg * 6 + hv * dk * 2) + nseq * hv * dk * dk * 8, gflops)
        del proj
        # ---- products
        wi = lru.in_proj
        add("projection", "linear with bias (RG-LRU in)", shape, lambda: ops.linear(y, wi), T * W * 2 + 4 * C * W + T * C * 4, 4.0 * T * W * C)
        plain = ops.LinearWeight("dense", wi.weight)
        add("projection", "linear (existing)", shape, lambda: ops.linear(y, plain), T * W * 2 + 4 * C * W + T * C * 4, 4.0 * T * W * C)
        add("feed-forward", "silu mlp, unit in the product", shape, lambda: mlp_a.forward(act), T * W * 4 + 6 * W * ff, 6.0 * T * W * ff)
        add("feed-forward", "silu mlp (existing)", shape, lambda: mlp_b.forward(act), T * W * 4 + 6 * W * ff, 6.0 * T * W * ff)

        def route(m, grouped):
            lg = ops.linear_tail(y, m.router, 0)[1] if grouped else ops.linear(y, m.router)
            if grouped:
                ops.moe_route(lg, top, True, "sigmoid", m.router_bias, GROUPS, KEEP, 2.5)
            else:
                ops.moe_route(lg, top, True)
        add("router", "fp32 logits, sigmoid, groups", shape, lambda: route(moe_a, True), T * W * 2 + E * W * 2)
        add("router", "bf16 logits, softmax (existing)", shape, lambda: route(moe_b, False), T * W * 2 + E * W * 2)
        eb, ef = T * W * 4 + (used + 1) * 6 * I * W, 6.0 * T * (top + 1) * W * I
        add("experts", "router, clamped experts + shared, rows", shape, lambda: moe_a.forward(act, rows_ok=True), eb + T * top * W * 2, ef)
        add("experts", "router, swiglu experts + shared (existing)", shape, lambda: moe_b.forward(act), eb, ef)
        # ---- attention
        (hq, hkv, d), ctx = s["attn"], 2048 if decode else 0
        per = (ctx + lens[0] + 15) // 16
        fb = ForwardBatch.build([[0] * lens[0]] * nseq, [ctx] * nseq, [list(range(i * per, (i + 1) * per)) for i in range(nseq)], 16, device=dev)
        L = ctx + lens[0]
        keys = L if decode else lens[0] / 2
        qkv = rn(T, (hq + 2 * hkv) * d)
        q, k, v = (t.view(T, -1, d) for t in qkv.split([hq * d, hkv * d, hkv * d], 1))
        kc, vc = K.alloc_kv_cache(per * nseq, 16, hkv, d, bf, dev)
        table = ref.build_rope_cache(d, 16384, 5e5, None, dev)
        qw, kw, hw = torch.ones(hq * d, device=dev), torch.ones(hkv * d, device=dev), torch.zeros(d, device=dev, dtype=bf)
        wb = T * (2 * hq + 4 * hkv) * d * 2
        add("cache write", "norm over all heads, temperature", shape,
            lambda: ops.qk_row_norm_kv_write(q, k, v, fb.positions, table[:, :0], 0, kc, vc, fb.slot_mapping, fb.positions, qw, kw, 1e-6, hq * d, hkv * d, 0.1, 8192), wb)
        add("cache write", "head norms, rotation (existing)", shape,
            lambda: ops.qk_norm_rope_kv_write(q, k, v, fb.positions, table, d, kc, vc, fb.slot_mapping, 1.0, 1.0, hw, hw, 1e-6, True), wb + T * d * 4)
        nb, fl = T * hq * d * 4 + nseq * hkv * d * 4 * L, 4.0 * T * keys * hq * d
        dist, sinks = distance_table(rn(ROWS, hq, dt=torch.float32), REACH), torch.zeros(hq, device=dev)
        qa = rn(T, hq, d)
        add("attention", "bf16 cache, distance bias", shape, lambda: ops.paged_attention(qa, kc, vc, fb, d ** -0.5, distance=dist), nb, fl)
        add("attention", "bf16 cache, fixed sink", shape, lambda: ops.paged_attention(qa, kc, vc, fb, d ** -0.5, sinks=sinks), nb, fl)
        add("attention", "bf16 cache, causal (existing)", shape, lambda: ops.paged_attention(qa, kc, vc, fb, d ** -0.5), nb, fl)
        del kc, vc, qa, qkv, pr, er, yx
        torch.cuda.empty_cache()
    return rows
