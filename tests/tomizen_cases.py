"""Small Tomizen configurations with random weights, shared by the CPU and GPU tests."""
import json
import os

import torch

from papidra_cases import feed_alone, feed_together, portions, spread, tokens  # noqa: F401


def mlstm(heads, dim, vdim, cap, mlp=None):
    return {"type": "mlstm", "mixer": {"heads": heads, "dim": dim, "vdim": vdim, "gate_cap": cap}, "mlp": mlp}


def latent(heads, dim, rot, vdim, rank, size, mlp=None, scale=None, scaling=True, base=1e4):
    sc = {"factor": 3.0, "original": 64, "fast": 8.0, "slow": 1.0} if scaling else None
    return {"type": "latent_attention", "mixer": {"heads": heads, "dim": dim, "rot_dim": rot, "vdim": vdim, "kv_rank": rank,
                                                  "scale": scale or (dim + rot) ** -0.5, "mask": {"size": size} if size else None,
                                                  "rot": {"base": base, "dims": rot, "scaling": sc}}, "mlp": mlp}


def attention(heads, kv, dim, vdim, cap, mlp=None, scale=None):
    return {"type": "attention", "mixer": {"heads": heads, "kv_heads": kv, "dim": dim, "vdim": vdim, "scale": scale or dim ** -0.5, "softcap": cap},
            "mlp": mlp}


def moe(experts, top, ff):
    return {"kind": "moe", "expert": {"ff": ff}, "router": {"experts": experts, "top": top}}


def model(vocab, width, layers, eps=1e-5):
    return {"architecture": "Tomizen", "vocab": vocab, "width": width, "norm": {"eps": eps}, "layers": layers}


CASES = {
    # different layers of each kind, one of each without a feed-forward, padded heads, windows that end inside pages
    "mixed": model(131, 96, [mlstm(3, 24, 40, 7.0, moe(6, 3, 40)), latent(6, 20, 12, 28, 40, 21, moe(5, 2, 64)),
                             attention(6, 2, 40, 24, 5.0, moe(9, 4, 24)), latent(3, 32, 32, 64, 96, 50, None, scaling=False),
                             attention(4, 4, 64, 64, 30.0, None, scale=0.2), mlstm(2, 48, 16, 15.0)]),
    # everything that can be one is one
    "ones": model(64, 64, [latent(1, 8, 2, 8, 8, 1, moe(1, 1, 8)), mlstm(1, 8, 8, 3.0, moe(2, 1, 8)), attention(1, 1, 64, 64, 2.0)]),
    # more heads than a tile holds, key sizes above 64 and 128, widths off the vector sizes
    "wide": model(77, 100, [latent(20, 72, 20, 130, 136, 33, moe(20, 5, 36)), attention(20, 1, 72, 40, 4.0, moe(3, 3, 50)),
                            mlstm(2, 136, 72, 9.0)]),
    # sizes that every tensor-core path takes; a latent layer that sees everything
    "aligned": model(96, 128, [mlstm(2, 64, 128, 12.0, moe(8, 2, 64)), latent(4, 32, 32, 64, 64, 40, moe(4, 2, 128)),
                               attention(8, 1, 64, 64, 10.0, moe(4, 1, 64)), latent(2, 64, 64, 128, 256, 0)]),
    # everything divides by two (tensor parallelism)
    "even": model(96, 64, [mlstm(2, 16, 24, 5.0, moe(4, 2, 16)), latent(4, 16, 8, 16, 24, 18), attention(4, 2, 32, 48, 6.0, moe(4, 2, 32))]),
    "odd": model(61, 90, [attention(3, 3, 20, 12, 3.0, moe(7, 2, 45)), mlstm(3, 10, 14, 2.0, moe(3, 2, 30)), latent(3, 9, 6, 11, 13, 19)]),
}


def weights(cfg, seed=0):
    """Random weights (rounded to bf16, like a checkpoint), scaled so that attention is peaked, scores meet their bound and memories
    are short and long.  The routers read channels of the embedding that no sublayer writes (their norm weights are zero there),
    so that no choice of an expert turns on rounding."""
    g = torch.Generator().manual_seed(seed)
    W = cfg["width"]
    out = {}

    def put(name, *shape, std=None, mean=0.0, uniform=None):
        if uniform:
            t = torch.rand(*shape, generator=g) * (uniform[1] - uniform[0]) + uniform[0]
        else:
            t = torch.randn(*shape, generator=g) * (std if std is not None else shape[-1] ** -0.5) + mean
        out[name] = t.to(torch.bfloat16)
    kept = W - max(4, min(16, W // 4))
    put("embed", cfg["vocab"], W, std=1.0)
    put("final.norm", W, std=0.2)
    put("head", cfg["vocab"], W)
    for i, l in enumerate(cfg["layers"]):
        p, m = f"l{i}.", l["mixer"]
        put(p + "norm1", W, std=0.2)
        out[p + "norm1"][kept:] = -1.0
        x = p + "mix."
        H = m["heads"]
        if l["type"] == "mlstm":
            for s, n in (("q", m["dim"]), ("k", m["dim"]), ("v", m["vdim"]), ("g", m["vdim"])):
                put(x + s, H * n, W)
            put(x + "norm", H * m["vdim"], std=0.2, mean=1.0)
            put(x + "i", H, W)
            put(x + "f", H, W)
            put(x + "i.b", H, uniform=(-2.0, 1.0))
            put(x + "f.b", H, uniform=(0.0, 5.0))
            put(x + "o", W, H * m["vdim"])
        elif l["type"] == "latent_attention":
            put(x + "q", H * (m["dim"] + m["rot_dim"]), W, std=2.0 * W ** -0.5)
            put(x + "dkv", m["kv_rank"] + m["rot_dim"], W)
            put(x + "dkv.norm", m["kv_rank"], std=0.2, mean=1.0)
            put(x + "uk", H * m["dim"], m["kv_rank"])
            put(x + "uv", H * m["vdim"], m["kv_rank"])
            put(x + "o", W, H * m["vdim"])
        else:
            put(x + "q", H * m["dim"], W)
            put(x + "k", m["kv_heads"] * m["dim"], W)
            put(x + "v", m["kv_heads"] * m["vdim"], W)
            put(x + "q.norm", m["dim"], std=0.3, mean=2.0)
            put(x + "k.norm", m["dim"], std=0.3, mean=1.5)
            put(x + "g", H, W)
            put(x + "o", W, H * m["vdim"])
        if l["mlp"] is not None:
            put(p + "norm2", W, std=0.2)
            out[p + "norm2"][kept:] = -1.0
            n = l["mlp"]["expert"]["ff"]
            put(p + "mlp.router", l["mlp"]["router"]["experts"], W, std=(W - kept) ** -0.5)
            out[p + "mlp.router"][:, :kept] = 0.0
            for e in range(l["mlp"]["router"]["experts"]):
                put(f"{p}mlp.e{e}.up", n, W)
                put(f"{p}mlp.e{e}.down", W, n)
    return out


def write(folder, name, seed=0):
    """Configuration and checkpoint of case ``name`` under ``folder``; returns ``(cfg, weights)``."""
    from safetensors.torch import save_file
    cfg = CASES[name]
    w = weights(cfg, seed)
    os.makedirs(folder, exist_ok=True)
    with open(os.path.join(folder, "config.json"), "w") as f:
        json.dump(cfg, f)
    save_file({k: v.contiguous() for k, v in w.items()}, os.path.join(folder, "model.safetensors"))
    return cfg, w
