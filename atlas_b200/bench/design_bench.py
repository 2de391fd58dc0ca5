"""Prefill and decode throughput of a design's layers beside the closest other model at equal size, and the rooflines of their
kernels.

    python bench.py --design papidra|tomizen|kenovik|bisudra    # or: python -m atlas_b200.bench.design_bench --design ...

``papidra`` beside Nemotron-H: the same width, feed-forward size, attention heads, Mamba-2 heads, vocabulary and cache dtype.  One
period is, for Papidra, a WKV layer and a layer with attention beside Mamba-2 plus a feed-forward; for Nemotron-H the blocks with
the same work: Mamba-2, attention, Mamba-2, MLP.

``tomizen`` (tomizen_bench.py) beside Qwen3-Next, and its latent attention beside DeepSeek's; ``kenovik`` (kenovik_bench.py) beside
Qwen3-Next; ``bisudra`` (bisudra_bench.py) beside Kenovik's attention layers.

All with random bf16 weights.  Steps are timed with CUDA events around a captured step (L2 flushed in between), kernels the same
way one by one.
"""
from __future__ import annotations

import argparse
import json
from typing import Dict, List, Optional

import torch

SIZES = {
    "2048": dict(width=2048, ff=7168, attn=(16, 4, 128), mamba=(64, 64, 128, 8), wkv=(32, 64)),
    "4096": dict(width=4096, ff=14336, attn=(32, 8, 128), mamba=(128, 64, 128, 8), wkv=(64, 64)),
}
PERIODS, VOCAB, CHUNK, STREAMS = 2, 32768, 4096, 4


def papidra(size: str):
    from ..config import _papidra
    s = SIZES[size]
    return _papidra(VOCAB, s["width"], s["ff"], "wp" * PERIODS, STREAMS, s["wkv"], s["attn"], s["mamba"], CHUNK, "bfloat16")


def nemotron(size: str):
    from ..config import ModelConfig, QuantConfig
    s = SIZES[size]
    (hq, hkv, d), (mh, mp, mn, mg) = s["attn"], s["mamba"]
    blocks = ["mamba", "attention", "mamba", "mlp"] * PERIODS
    return ModelConfig(model_type="nemotron_h", family="hybrid", vocab_size=VOCAB, hidden_size=s["width"], intermediate_size=s["ff"],
                       num_hidden_layers=len(blocks), num_attention_heads=hq, num_key_value_heads=hkv, head_dim=d,
                       partial_rotary_factor=0.0, rms_norm_eps=1e-5, block_types=blocks, mamba_num_heads=mh, mamba_head_dim=mp,
                       ssm_state_size=mn, mamba_n_groups=mg, mlp_activation="relu2", quant=QuantConfig(kv_cache_dtype="bf16"))


def _step(model, cache, nseq: int, rows: int, ctx: int):
    """A closure over one step: ``rows`` new tokens of ``nseq`` sequences that hold ``ctx`` tokens."""
    from ..models import ForwardBatch
    bs = cache.block_size
    per = (ctx + rows + bs - 1) // bs
    g = torch.Generator().manual_seed(0)
    toks = [torch.randint(0, VOCAB, (rows,), generator=g).tolist() for _ in range(nseq)]
    fb = ForwardBatch.build(toks, [ctx] * nseq, [list(range(i * per, (i + 1) * per)) for i in range(nseq)], bs, device=model.device,
                            state_slots=list(range(nseq)), has_state=[ctx > 0] * nseq)
    last = (fb.query_start_loc[1:] - 1).long()
    return lambda: model.compute_logits(model.forward(fb, cache), last)


def throughput(cfg, timer, prefill=((1, 8192), (8, 1024)), decode=(1, 32, 128), ctx: int = 2048) -> Dict[str, float]:
    from ..models import build_model
    cfg.max_position_embeddings = 16384
    model = build_model(cfg, device="cuda").init_random(0, max_pos=16384)
    bs = 16
    blocks = max([n * ((r + bs - 1) // bs) for n, r in prefill] + [max(decode) * ((ctx + bs) // bs + 1)]) + 8
    cache = model.alloc_cache(blocks, bs, torch.bfloat16, state_slots=max(list(decode) + [n for n, _ in prefill]) + 1)
    out = {}
    for n, r in prefill:
        ms = timer.time(_step(model, cache, n, r, 0), iters=5)
        out[f"prefill {n}x{r}"] = {"ms": round(ms, 3), "tok_s": round(n * r / ms * 1e3)}
    for n in decode:
        ms = timer.time(_step(model, cache, n, 1, ctx), iters=7)
        out[f"decode {n} @ {ctx}"] = {"ms": round(ms, 4), "tok_s": round(n / ms * 1e3)}
    del model, cache
    torch.cuda.empty_cache()
    return out


# ----------------------------------------------------------------------------- kernels
def kernel_table(size: str, timer, peaks) -> List[dict]:
    """Every kernel of the new layers beside the like kernel of the existing model: time and fraction of the roofline (bytes the
    kernel must move at the measured copy bandwidth, or attention's products at the measured bf16 rate, the slower of both)."""
    from types import SimpleNamespace

    from .. import ops
    from ..layers import HyperConnection
    from ..models import ForwardBatch
    from ..ops import cuda as K
    s = SIZES[size]
    W, I = s["width"], s["ff"]
    (hq, hkv, d), (mh, mp, mn, mg), (wh, wd) = s["attn"], s["mamba"], s["wkv"]
    dev, bf = "cuda", torch.bfloat16
    gen = torch.Generator(device=dev).manual_seed(0)
    rn = lambda *sh, dt=bf: torch.randn(*sh, generator=gen, device=dev).to(dt)
    rows: List[dict] = []

    def add(pair: str, who: str, shape: str, fn, nbytes: float, flops: float = 0.0):
        us = timer.time(fn) * 1e3
        ideal = max(nbytes / peaks["hbm_gbs"] / 1e3, flops / peaks["bf16_tflops"] / 1e6)
        rows.append({"pair": pair, "kernel": who, "shape": shape, "us": round(us, 1), "roofline": round(ideal / us, 3)})

    for T, nseq in ((8192, 8), (8192, 1), (128, 128), (1, 1)):
        decode = T == nseq
        shape = f"{T} rows, {nseq} seq"
        lens = [T // nseq] * nseq
        b = SimpleNamespace(query_lens_host=lens, state_slots_host=list(range(nseq)), has_state_host=[True] * nseq, snapshot_plan={})
        y, y2, x = rn(T, W), rn(T, W), rn(T, STREAMS, W, dt=torch.float32)
        nw = torch.ones(W, device=dev)
        conn = HyperConnection(STREAMS)
        conn.init_random(gen, dev)
        add("norm", "hyper_norm", shape, lambda: ops.hyper_norm(x, ops.StreamDelta(y, conn), conn.read, nw, 1e-5), T * W * (8 * STREAMS + 4))
        add("norm", "hyper_norm, two outputs", shape, lambda: ops.hyper_norm(x, ops.StreamDelta(y, conn, y2=y2, w1=nw, w2=nw), conn.read, nw, 1e-5),
            T * W * (8 * STREAMS + 6))
        nwb = nw.to(bf)
        add("norm", "rmsnorm + residual (existing)", shape, lambda: ops.rmsnorm(y, nwb, 1e-5, y2), T * W * 8)
        mu, shift = torch.rand(5, W, device=dev), rn(nseq, W)
        add("shift", "token_shift_mix", shape, lambda: K.token_shift_mix(y, mu, b, shift), T * W * 12)
        gu = rn(T, 2 * I)
        add("activation", "clamped_glu", shape, lambda: ops.clamped_glu_act(gu, 7.0, 1.702), T * I * 6)
        up = rn(T, I)
        add("activation", "relu2 (existing)", shape, lambda: ops.relu_squared(up), T * I * 4)
        n = wh * wd
        r, k, v, raw = (rn(T, n) for _ in range(4))
        lay = SimpleNamespace(w0=torch.linspace(-6, -1, n, device=dev), u=torch.rand(wh, wd, device=dev), inner=n, h=wh, d=wd)
        st = {"h": torch.zeros(nseq, wh, wd, wd, device=dev), "shift": shift}
        state = nseq * wh * wd * wd * 8
        add("recurrence", "wkv_scan", shape, lambda: K.wkv_forward(lay, y, r, k, v, raw, b, st, True), T * n * 10 + state)
        di, C = mh * mp, mh * mp + 2 * mg * mn
        proj = rn(T, C + mh)
        ml = SimpleNamespace(conv_w=rn(C, 4), conv_b=rn(C), W=4, d_inner=di, A_log=torch.zeros(mh, device=dev), D=torch.ones(mh, device=dev),
                             dt_bias=torch.zeros(mh, device=dev), cfg=SimpleNamespace(mamba_dt_min=0.0), h=mh, p=mp, n=mn, g=mg)
        ms = {"h": torch.zeros(nseq, mh, mp, mn, device=dev), "conv": torch.zeros(nseq, C, 3, dtype=bf, device=dev)}
        mstate = nseq * mh * mp * mn * 8
        add("recurrence", "mamba2 conv + scan + window (shared)", shape, lambda: K.mamba2_forward(ml, proj[:, :C], proj[:, C:], b, ms, True),
            T * (C * 4 + C * 2 + di * 2 + mh * 2) + mstate)
        z, gw = rn(T, n), torch.ones(n, device=dev)
        add("gated norm", "group_norm_gate (WKV)", shape, lambda: ops.group_norm_gate(r, z, gw, wd, 1e-5, False), T * n * 6)
        yo, zo, gd = rn(T, di), rn(T, di), torch.ones(di, device=dev)
        add("gated norm", "group_norm_gate (Mamba-2, shared)", shape, lambda: ops.group_norm_gate(yo, zo, gd, di // mg, 1e-5, True), T * di * 6)
        del x, gu, up, proj
        ctx = 2048 if decode else 0
        per = (ctx + lens[0] + 15) // 16
        fb = ForwardBatch.build([[0] * lens[0]] * nseq, [ctx] * nseq, [list(range(i * per, (i + 1) * per)) for i in range(nseq)], 16, device=dev)
        q = rn(T, hq, d)
        L = ctx + lens[0]
        keys = min(L, CHUNK) if decode else min(lens[0], CHUNK) / 2
        flops = 4.0 * T * keys * hq * d
        kvb = nseq * hkv * d * 2 * (L if not decode else min(L, CHUNK))
        sinks = torch.zeros(hq, device=dev)
        kc, vc = K.alloc_kv_cache(per * nseq, 16, hkv, d, bf, dev)
        add("attention", "bf16 cache, chunks + sinks", shape, lambda: ops.paged_attention(q, kc, vc, fb, d ** -0.5, chunk=CHUNK, sinks=sinks),
            T * hq * d * 4 + kvb * 2, flops)
        keys_all = L if decode else lens[0] / 2
        add("attention", "bf16 cache, causal (existing)", shape, lambda: ops.paged_attention(q, kc, vc, fb, d ** -0.5),
            T * hq * d * 4 + nseq * hkv * d * 4 * L, 4.0 * T * keys_all * hq * d)
        kf, vf = K.alloc_kv_cache(per * nseq, 16, hkv, d, torch.float8_e4m3fn, dev)
        add("attention", "fp8 cache, causal (existing)", shape, lambda: ops.paged_attention(q, kf, vf, fb, d ** -0.5),
            T * hq * d * 4 + nseq * hkv * d * 2 * L, 4.0 * T * keys_all * hq * d)
        del kc, vc, kf, vf, q
        torch.cuda.empty_cache()
    return rows


def designs() -> dict:
    """name -> (name of the model beside it, sizes, configuration of both by size, kernel table, layers)"""
    from . import bisudra_bench as B, kenovik_bench as V, tomizen_bench as T
    return {"papidra": ("nemotron_h", SIZES, papidra, nemotron, kernel_table, f"{PERIODS} periods"),
            "tomizen": ("qwen3_next", T.SIZES, T.tomizen, T.beside, T.kernel_table, "4 layers"),
            "kenovik": ("qwen3_next", V.SIZES, V.kenovik, V.beside, V.kernel_table, "4 layers"),
            "bisudra": ("kenovik", B.SIZES, B.bisudra, B.beside, B.kernel_table, "4 layers")}


def run(sizes: Optional[List[str]] = None, kernels: bool = True, design: str = "papidra") -> dict:
    from ..ops import cuda as K
    from .microbench import Timer, load_peaks
    K.load()
    timer, peaks = Timer(), load_peaks()
    other, all_sizes, mine, theirs, table, layers = designs()[design]
    out: dict = {"design": design, "beside": other, "dtype": "bf16 weights and KV cache", "data": "synthetic: random weights and tokens",
                 "l2": "flushed between timed steps", "peaks": peaks, "sizes": {}}
    with torch.inference_mode():
        for s in sizes or list(all_sizes):
            a, b = mine(s), theirs(s)
            out["sizes"][s] = {design: throughput(a, timer), other: throughput(b, timer), "layers": layers,
                               "params_m": [round(c.param_count() / 1e6, 1) for c in (a, b)]}
            if kernels:
                out["sizes"][s]["kernels"] = table(s, timer, peaks)
    assert K.check_status() == 0
    return out


def report(res: dict) -> str:
    lines, (a, b) = [], (res["design"], res["beside"])
    for s, r in res["sizes"].items():
        lines.append(f"width {s}, {r['layers']}, parameters (M) {r['params_m'][0]} / {r['params_m'][1]}")
        for key, v in r[a].items():
            w = r[b][key]
            lines.append(f"  {key:<18} {a} {v['ms']:>9} ms {v['tok_s']:>9} tok/s    {b} {w['ms']:>9} ms {w['tok_s']:>9} tok/s")
        for k in r.get("kernels", ()):
            lines.append(f"  {k['pair']:<12} {k['kernel']:<46} {k['shape']:<20} {k['us']:>9} us  {k['roofline']:.3f} of roofline")
    return "\n".join(lines)


def main(argv=None) -> int:
    ap = argparse.ArgumentParser()
    ap.add_argument("--design", default="papidra", choices=["papidra", "tomizen", "kenovik", "bisudra"])
    ap.add_argument("--sizes", default="", help="widths (default: all of the design)")
    ap.add_argument("--no-kernels", action="store_true")
    ap.add_argument("--out")
    a = ap.parse_args(argv)
    res = run([s for s in a.sizes.split(",") if s], not a.no_kernels, a.design)
    print(report(res))
    if a.out:
        with open(a.out, "w") as f:
            json.dump(res, f, indent=1)
    return 0


if __name__ == "__main__":
    raise SystemExit(main())
