"""Small Kenovik configurations with random weights, shared by the CPU and GPU tests."""
import json
import os

import torch

from papidra_cases import feed_alone, feed_together, portions, spread, tokens  # noqa: F401


def sink(heads, kv, dim, vdim, dims, mlp=None, scale=None, base=1e4, factor=3.0):
    scaling = {"factor": factor} if factor else None
    return {"type": "attention", "mixer": {"heads": heads, "kv_heads": kv, "dim": dim, "vdim": vdim, "scale": scale or dim ** -0.5,
                                           "rot": {"dims": dims, "base": base, "scaling": scaling}}, "mlp": mlp}


def distance(heads, kv, dim, vdim, reach, mlp=None, scale=None, coef=0.4, every=16, rows=8):
    return {"type": "attention_2", "rows": rows,
            "mixer": {"heads": heads, "kv_heads": kv, "dim": dim, "vdim": vdim, "scale": scale or dim ** -0.5, "bias_max": reach,
                      "q_temp": {"coef": coef, "every": every}}, "mlp": mlp}


def rglru(width, blocks, conv, mlp=None):
    return {"type": "rglru", "mixer": {"width": width, "blocks": blocks, "conv": conv}, "mlp": mlp}


def dense(ff):
    return {"kind": "dense", "ff": ff}


def moe(experts, top, ff, count, keep, limit=1.2, scale=1.7, shared=None):
    """``shared``: (hidden size, limit) of the shared expert."""
    return {"kind": "moe", "expert": {"ff": ff, "limit": limit}, "shared": shared and {"ff": shared[0], "limit": shared[1]},
            "router": {"experts": experts, "top": top, "scale": scale, "groups": {"count": count, "keep": keep}}}


def model(vocab, width, layers, loop=None, eps=1e-5, scale=1.5):
    return {"architecture": "Kenovik", "vocab": vocab, "width": width, "norm": {"eps": eps}, "embedding": {"scale": scale}, "layers": layers,
            "loop": loop and dict(zip(("start", "stop", "times"), loop))}


CASES = {
    # layers of each kind with each feed-forward and without one, padded heads, a loop in the middle that runs three times
    "mixed": model(131, 96, [sink(6, 2, 24, 40, 16), distance(4, 2, 40, 24, 37, moe(6, 3, 40, 3, 2, shared=(24, 0.8))),
                             rglru(60, 3, 4, dense(72)), sink(3, 1, 48, 32, 48, moe(8, 2, 24, 4, 3)), rglru(96, 2, 3),
                             distance(6, 3, 32, 32, 90, dense(40), rows=12)], (1, 4, 3)),
    # everything that can be one is one
    "ones": model(64, 64, [rglru(8, 1, 1, moe(1, 1, 8, 1, 1, shared=(8, 1.0))), sink(1, 1, 2, 1, 2, factor=1.0), distance(1, 1, 1, 1, 2, dense(1), every=1, rows=2)],
                  (1, 2, 1), scale=1.0),
    # more heads than a tile holds, sizes off the vector sizes, blocks wider than a tile, many groups, an odd number of rows
    "wide": model(77, 100, [distance(20, 1, 72, 130, 60, moe(24, 5, 36, 6, 2, shared=(50, 2.0)), rows=9), rglru(3 * 139, 3, 7, dense(37)),
                            sink(20, 1, 72, 40, 40, moe(5, 3, 50, 5, 4))], (0, 3, 2)),
    # sizes that every tensor-core path takes; the distance table outgrows shared memory
    "aligned": model(96, 128, [rglru(256, 2, 4, moe(8, 2, 64, 4, 2, shared=(64, 1.0))), distance(8, 1, 128, 128, 4000, moe(8, 4, 128, 2, 1), rows=32),
                               sink(8, 2, 64, 64, 64, dense(128), factor=None), rglru(128, 1, 4)], (0, 2, 2)),
    # everything divides by two (tensor parallelism)
    "even": model(96, 64, [rglru(32, 2, 4, dense(64)), sink(4, 2, 16, 24, 8, moe(4, 2, 16, 2, 1, shared=(16, 1.0))), distance(4, 2, 32, 48, 25, moe(4, 2, 32, 2, 2))],
                  (1, 3, 2)),
    # no loop, no groups worth the name, no feed-forward at the end
    "plain": model(61, 90, [distance(3, 3, 20, 12, 11, moe(7, 2, 45, 7, 5), rows=6), rglru(45, 9, 2, dense(30)), sink(3, 3, 9, 11, 6)]),
}


def weights(cfg, seed=0):
    """Random weights (rounded to bf16, like a checkpoint): peaked attention, distances that matter, decays from short to long,
    scores around zero beside the fixed sink, corrections of both signs.  The routers read channels of the residual that no
    sublayer writes, so that hardly a choice of an expert turns on rounding."""
    g = torch.Generator().manual_seed(seed)
    W = cfg["width"]
    kept = W - max(4, min(16, W // 4))
    out = {}

    def put(name, *shape, std=None, mean=0.0, uniform=None):
        if uniform:
            t = torch.rand(*shape, generator=g) * (uniform[1] - uniform[0]) + uniform[0]
        else:
            t = torch.randn(*shape, generator=g) * (std if std is not None else shape[-1] ** -0.5) + mean
        out[name] = t.to(torch.bfloat16)

    def writes(name, *shape):
        put(name, *shape)
        out[name][kept:] = 0.0

    def unit(pre, ff):
        put(pre + "gate", ff, W)
        put(pre + "up", ff, W)
        writes(pre + "down", W, ff)
    put("embed", cfg["vocab"], W, std=1.0)
    put("final.norm", W, std=0.2, mean=1.0)
    if cfg["loop"]:
        put("loop.step", cfg["loop"]["times"], W, std=0.7)
    for i, l in enumerate(cfg["layers"]):
        p, m = f"l{i}.", l["mixer"]
        put(p + "norm1", W, std=0.2, mean=1.0)
        x = p + "mix."
        if l["type"] == "rglru":
            C, n = m["width"], m["width"] // m["blocks"]
            for s in "yx":
                put(x + s, C, W)
                put(x + s + ".b", C, std=0.3)
            put(x + "conv", C, m["conv"], std=0.6)
            put(x + "conv.b", C, std=0.3)
            for s in ("ra", "ri"):
                put(x + s, m["blocks"], n, n)
                put(x + s + ".b", m["blocks"], n, std=1.0)
            put(x + "lam", C, uniform=(-7.0, 1.0))
            writes(x + "o", W, C)
        else:
            H, G = m["heads"], m["kv_heads"]
            for s, n in (("q", H * m["dim"]), ("k", G * m["dim"]), ("v", G * m["vdim"])):
                put(x + s, n, W, std=(1.5 if s != "v" else 1.0) * W ** -0.5)
                if l["type"] == "attention":
                    put(x + s + ".b", n, std=0.5)
            if l["type"] == "attention_2":
                put(x + "q.norm", H * m["dim"], std=0.3, mean=1.6)
                put(x + "k.norm", G * m["dim"], std=0.3, mean=1.4)
                put(x + "rel", l["rows"], H, std=1.5)
            writes(x + "o", W, H * m["vdim"])
        f = l["mlp"]
        if f is None:
            continue
        put(p + "norm2", W, std=0.2, mean=1.0)
        if f["kind"] == "dense":
            unit(p + "mlp.", f["ff"])
            continue
        E = f["router"]["experts"]
        put(p + "mlp.router", E, W, std=2.0 * (W - kept) ** -0.5)
        out[p + "mlp.router"][:, :kept] = 0.0
        put(p + "mlp.correction", E, std=0.5, mean=-0.6)
        for e in range(E):
            unit(f"{p}mlp.e{e}.", f["expert"]["ff"])
        if f["shared"]:
            unit(p + "mlp.shared.", f["shared"]["ff"])
    return out


def write(folder, name, seed=0):
    """Configuration and checkpoint of case ``name`` under ``folder``; returns ``(cfg, weights)``."""
    from safetensors.torch import save_file
    cfg = CASES[name]
    w = weights(cfg, seed)
    os.makedirs(folder, exist_ok=True)
    plain = {**cfg, "layers": [{k: v for k, v in l.items() if k != "rows"} for l in cfg["layers"]]}
    with open(os.path.join(folder, "config.json"), "w") as f:
        json.dump(plain, f)
    save_file({k: v.contiguous() for k, v in w.items()}, os.path.join(folder, "model.safetensors"))
    return cfg, w
