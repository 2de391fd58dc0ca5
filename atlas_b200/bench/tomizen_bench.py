"""Sizes, models and kernel table of ``bench.py --design tomizen``.

Four layers of Tomizen (mLSTM, latent attention, attention, mLSTM, each with experts) beside four layers of Qwen3-Next with the same
work: Gated DeltaNet with the same recurrent state, gated attention, experts with the same number of weights.  The latent layer's
kernels stand beside those of the DeepSeek layer (latent attention on expanded heads) and, where the kernel is an attention
kernel, beside causal attention on a bf16 cache.
"""
from __future__ import annotations

from types import SimpleNamespace
from typing import List

import torch

# mlstm: heads, key size, value size; latent: heads, unrotated, rotated, value, rank; attn: heads, kv heads, size; moe: experts, per
# token, hidden size (two matrices here, three in the other model: a hidden size of two thirds there)
SIZES = {
    "2048": dict(width=2048, mlstm=(16, 128, 256), gdn=(16, 32, 128), latent=(16, 64, 64, 128, 512), attn=(16, 2, 128), moe=(64, 6, 1408), glu=960),
    "4096": dict(width=4096, mlstm=(32, 128, 256), gdn=(32, 64, 128), latent=(32, 64, 64, 128, 512), attn=(32, 8, 128), moe=(64, 6, 2048), glu=1344),
}
VOCAB, WINDOW, CAP = 32768, 4096, 30.0


def tomizen(size: str):
    from ..config import _tomizen
    s = SIZES[size]
    return _tomizen(VOCAB, s["width"], "mlam", s["mlstm"], s["latent"] + (WINDOW,), s["attn"], s["moe"], "bfloat16")


def beside(size: str):
    from ..config import ModelConfig, QuantConfig
    s = SIZES[size]
    (hq, hkv, d), (hk, hv, dk), (E, top, _) = s["attn"], s["gdn"], s["moe"]
    return ModelConfig(model_type="qwen3_next", family="hybrid", vocab_size=VOCAB, hidden_size=s["width"], intermediate_size=s["glu"],
                       num_hidden_layers=4, num_attention_heads=hq, num_key_value_heads=hkv, head_dim=d, rope_theta=1e7,
                       partial_rotary_factor=0.25, qk_norm=True, attn_output_gate=True, norm_plus_one=True, num_experts=E,
                       num_experts_per_tok=top, moe_intermediate_size=s["glu"], norm_topk_prob=True,
                       layer_types=["linear_attention", "full_attention", "full_attention", "linear_attention"], linear_num_key_heads=hk,
                       linear_num_value_heads=hv, linear_key_head_dim=dk, linear_value_head_dim=dk, quant=QuantConfig(kv_cache_dtype="bf16"))


def _deepseek(size: str):
    from ..config import ModelConfig, QuantConfig
    s = SIZES[size]
    H, dn, dr, dv, rank = s["latent"]
    need = max(dn + dr, dv)
    head = next(d for d in (64, 128, 256) if d >= need)
    return ModelConfig(model_type="deepseek_v2", family="moe", hidden_size=s["width"], num_attention_heads=H, num_key_value_heads=H, head_dim=head,
                       partial_rotary_factor=dr / head, kv_lora_rank=rank, qk_nope_head_dim=dn, qk_rope_head_dim=dr, v_head_dim=dv,
                       quant=QuantConfig(kv_cache_dtype="bf16"))


def kernel_table(size: str, timer, peaks) -> List[dict]:
    """Time and fraction of the roofline (bytes the kernels must move at the measured copy bandwidth, or their products at the
    measured bf16 rate, the slower of both) of every kernel of the new layers, each beside the like kernel of the other model."""
    from .. import ops
    from ..layers import GatedDeltaNet, LatentAttention, MLAttention, MLSTMMixer, MoE, ParallelCtx
    from ..models import ForwardBatch
    from ..ops import Act, cuda as K, cuda_latent as KL, reference as ref
    s = SIZES[size]
    W = s["width"]
    dev, bf = "cuda", torch.bfloat16
    gen = torch.Generator(device=dev).manual_seed(0)
    rn = lambda *sh, dt=bf, std=1.0: (torch.randn(*sh, generator=gen, device=dev) * std).to(dt)
    ours, qwen, ds = tomizen(size), beside(size), _deepseek(size)
    p = ParallelCtx()
    rows: List[dict] = []

    def add(pair: str, who: str, shape: str, fn, nbytes: float, flops: float = 0.0):
        us = timer.time(fn) * 1e3
        ideal = max(nbytes / peaks["hbm_gbs"] / 1e3, flops / peaks["bf16_tflops"] / 1e6)
        rows.append({"pair": pair, "kernel": who, "shape": shape, "us": round(us, 1), "roofline": round(ideal / us, 3)})

    (H, D, V), (hk, hv, dk) = s["mlstm"], s["gdn"]
    (E, top, I), glu = s["moe"], s["glu"]
    ml, gd = MLSTMMixer(ours.for_layer(0), 0, p, "dense"), GatedDeltaNet(qwen, 0, p, "dense")
    moe_a, moe_b = MoE(ours.for_layer(0), p, "dense", "dense"), MoE(qwen, p, "dense", "dense")
    la, mla = LatentAttention(ours.for_layer(1), 1, p, "dense"), MLAttention(ds, 0, p, "dense")
    for m in (ml, gd, moe_a, moe_b, la, mla):
        m.init_random(gen, 0.02, bf, dev)
    for T, nseq in ((8192, 8), (8192, 1), (128, 128), (1, 1)):
        decode = T == nseq
        shape, lens = f"{T} rows, {nseq} seq", [T // nseq] * nseq
        b = SimpleNamespace(query_lens_host=lens, state_slots_host=list(range(nseq)), has_state_host=[True] * nseq, snapshot_plan={}, spec_verify=False)
        # ---- residual and norm
        y, x = rn(T, W), rn(T, W, dt=torch.float32)
        nw = torch.zeros(W, device=dev)
        add("norm", "add_normed", shape, lambda: ops.add_normed(x, ops.NormDelta(y, nw), 1e-6, True), T * W * 12)
        pr, slots, pw = rn(T * top, W), torch.randperm(T * top, generator=gen, device=dev).to(torch.int32), torch.rand(T, top, device=dev)
        er = ops.ExpertRows(pr, slots, pw)
        add("norm", "add_normed of expert rows", shape, lambda: ops.add_normed(x, ops.NormDelta(er, nw), 1e-6, True), T * W * (10 + 2 * top))
        nwb, out, res = nw.to(bf), torch.empty(T, W, dtype=bf, device=dev), rn(T, W)
        add("norm", "rmsnorm + residual (existing)", shape, lambda: ops.rmsnorm(y, nwb, 1e-6, res, True), T * W * 8)

        def combine_then_norm():
            K._check(K.lib().atlas_moe_combine(pr.data_ptr(), W, slots.data_ptr(), pw.data_ptr(), T, top, W, None, 0, out.data_ptr(), W, K._stream()), "moe_combine")
            ops.rmsnorm(out, nwb, 1e-6, res, True)
        add("norm", "moe_combine, rmsnorm + residual (existing)", shape, combine_then_norm, T * W * (8 + 2 * top))
        # ---- recurrence
        q, k, v, raw = rn(T, H * D), rn(T, H * D), rn(T, H * V), rn(T, 2 * H, dt=torch.float32)
        st = ml.alloc_state(nseq, dev, bf)
        state = nseq * H * (V + 1) * D * 8
        chunk_flops = T * H * (2.0 * 64 * D + 2.0 * 64 * V + 4.0 * D * V) if not decode else 0.0
        add("recurrence", "mlstm gates + memory", shape, lambda: K.mlstm_forward(ml, q, k, v, raw, b, st, True), T * H * (4 * D + 4 * V + 8) + state, chunk_flops)
        C = gd.conv_dim
        proj = rn(T, C + 2 * hv)
        gs = gd.alloc_state(nseq, dev, bf)
        gstate = nseq * hv * dk * dk * 8
        gflops = T * hv * (4.0 * 64 * dk + 2.0 * 64 * dk + 6.0 * dk * dk) if not decode else 0.0
        add("recurrence", "gdn conv + memory + window (existing)", shape,
            lambda: K.gdn_forward(gd, proj[:, :C], proj[:, C:C + hv], proj[:, C + hv:], b, gs, True), T * (C * 6 + hv * dk * 2) + gstate, gflops)
        num, z, den, gw = rn(T, H * V), rn(T, H * V), torch.rand(T, H, device=dev) + 1, torch.ones(H * V, device=dev)
        add("gated norm", "group_norm_gate (sigmoid, den)", shape, lambda: ops.group_norm_gate(num, z, gw, V, 1e-6, False, "sigmoid", den), T * H * V * 6)
        z3, n3, gw2 = rn(T, hv, dk), rn(T, hv, dk), torch.ones(dk, device=dev, dtype=bf)
        add("gated norm", "gated_rmsnorm (existing)", shape, lambda: K.gated_rmsnorm(n3, z3, gw2, 1e-6), T * hv * dk * 6)
        del num, z, z3, n3, proj, q, k, v
        # ---- products with an fp32 tail, experts
        n = ml.in_proj.w.weight.shape[0]
        add("projection", "linear_tail (mLSTM in)", shape, lambda: ml.in_proj(y), T * W * 2 + n * W * 2 + T * n * 2, 2.0 * T * W * n)
        n2 = gd.in_proj.weight.shape[0]
        add("projection", "linear (GDN in, existing)", shape, lambda: ops.linear(y, gd.in_proj), T * W * 2 + n2 * W * 2 + T * n2 * 2, 2.0 * T * W * n2)

        def route(m, cfg, f32):
            lg = ops.linear_tail(y, m.router, 0)[1] if f32 else ops.linear(y, m.router)
            ops.moe_route(lg, top, cfg.norm_topk_prob)
        add("router", "fp32 logits + top k", shape, lambda: route(moe_a, ours.for_layer(0), True), T * W * 2 + E * W * 2)
        add("router", "bf16 logits + top k (existing)", shape, lambda: route(moe_b, qwen, False), T * W * 2 + E * W * 2)
        act, used = Act(x=y), min(E, T * top)
        add("experts", "relu2 experts, rows", shape, lambda: moe_a.forward(act, rows_ok=True), T * W * 4 + used * 2 * I * W * 2 + T * top * W * 2, 4.0 * T * top * W * I)
        add("experts", "swiglu experts, combined (existing)", shape, lambda: moe_b.forward(act), T * W * 4 + used * 3 * glu * W * 2, 6.0 * T * top * W * glu)
        # ---- attention
        (hq, hkv, d), ctx = s["attn"], 2048 if decode else 0
        per = (ctx + lens[0] + 15) // 16
        fb = ForwardBatch.build([[0] * lens[0]] * nseq, [ctx] * nseq, [list(range(i * per, (i + 1) * per)) for i in range(nseq)], 16, device=dev)
        L = ctx + lens[0]
        keys = L if decode else lens[0] / 2
        qa = rn(T, hq, d)
        kc, vc = K.alloc_kv_cache(per * nseq, 16, hkv, d, bf, dev)
        nb, fl = T * hq * d * 4 + nseq * hkv * d * 4 * L, 4.0 * T * keys * hq * d
        add("attention", "bf16 cache, bounded scores", shape, lambda: ops.paged_attention(qa, kc, vc, fb, d ** -0.5, softcap=CAP), nb, fl)
        add("attention", "bf16 cache, causal (existing)", shape, lambda: ops.paged_attention(qa, kc, vc, fb, d ** -0.5), nb, fl)
        g1, g2, o2 = rn(T, hq, dt=torch.float32), rn(T, hq * d), rn(T, hq * d)
        add("output gate", "head_gate", shape, lambda: ops.head_gate(qa, g1), T * hq * d * 4)
        add("output gate", "sigmoid_gate_mul (existing)", shape, lambda: K.sigmoid_gate_mul(o2, g2), T * hq * d * 6)
        del kc, vc, qa, o2, g2
        # ---- latent attention: the whole block between the projections' input and the output projection
        lh, dn, dr, lv, rank = s["latent"]
        table = ref.build_rope_cache(dr, 16384, 5e5, None, dev)
        cache, _ = la.alloc_kv(per * nseq, 16, bf, dev)
        kx, vx = K.alloc_kv_cache(per * nseq, 16, lh, mla.d, bf, dev)
        vis = min(L, WINDOW)
        vkeys = vis if decode else min(lens[0] / 2, WINDOW)
        pw_flops = 2.0 * T * W * (lh * (dn + dr) + rank + dr)
        core = 2.0 * T * vkeys * lh * (dn + dr + lv)
        expand = 2.0 * T * rank * lh * (dn + lv)
        wb = W * (lh * (dn + dr) + rank + dr) * 2 + rank * lh * (dn + lv) * 2
        io = T * W * 2 + T * lh * lv * 2
        add("latent block", "latent cache", shape, lambda: la.mix(act, fb, (cache, None), table), wb + io + nseq * vis * (rank + dr) * 2, pw_flops + core + expand)
        add("latent block", "expanded cache (existing)", shape, lambda: mla.mix(act, fb, (kx, vx, 1.0, 1.0), table),
            wb + io + nseq * L * lh * (dn + dr + lv) * 2, pw_flops + core + expand)
        if decode:
            mt = KL.row_tiles(la)
            qq, lat = rn(T, lh, la.width), torch.empty(T, lh, la.rp, dtype=bf, device=dev)
            splits = KL.decode_splits(nseq, lh, mt, vis, K._num_sms[K._dev(qq)])
            po, pml = torch.empty(T * lh * splits * la.rp, device=dev), torch.empty(T * lh * splits * 2, device=dev)
            KL._lib()

            def absorbed():
                K._check(K.lib().atlas_latent_attn(qq.data_ptr(), cache.data_ptr(), lat.data_ptr(), po.data_ptr(), pml.data_ptr(), fb.block_tables.data_ptr(),
                                                   fb.block_tables.stride(0), fb.seq_lens.data_ptr(), fb.query_start_loc.data_ptr(), None, None, None, 0, T, T,
                                                   lh, la.rp, la.ep, 16, WINDOW, splits, mt, 0.1, K._stream()), "latent_attn")
            add("latent kernel", "absorbed decode", shape, absorbed, nseq * vis * la.width * 2 + T * lh * (2 * la.rp + la.ep) * 2,
                2.0 * T * vis * lh * (la.width + la.rp))
            qx = rn(T, lh, mla.d)
            add("latent kernel", "expanded decode (existing)", shape, lambda: ops.paged_attention(qx, kx, vx, fb, 0.1),
                T * lh * mla.d * 4 + nseq * L * lh * mla.d * 4, 4.0 * T * L * lh * mla.d)
            add("latent kernel", "head_gemm (W_uk)", shape,
                lambda: KL._head_gemm(qx, lh * mla.d, mla.d, la.uk, qq, lh * la.width, la.width, T), la.uk.numel() * 2 + T * lh * (dn + la.rp) * 2,
                2.0 * T * la.uk.numel())
            wd = ops.LinearWeight("dense", rn(la.rp * lh // 2, 2 * dn))
            add("latent kernel", "linear of the same weights (existing)", shape, lambda: ops.linear(qx.view(T, -1)[:, :2 * dn].contiguous(), wd),
                wd.weight.numel() * 2 + T * (2 * dn + wd.weight.shape[0]) * 2, 2.0 * T * wd.weight.numel())
        del kx, vx, cache, pr, er
        torch.cuda.empty_cache()
    return rows
