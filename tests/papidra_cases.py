"""Small Papidra configurations with random weights, shared by the CPU and GPU tests."""
import json
import os

import torch


def attn(heads, kv, dim, vdim, size, rot_dims, scale=None, scaling=True, base=1e4):
    sc = {"factor": 3.0, "original": 64, "fast": 8.0, "slow": 1.0} if scaling else None
    return {"heads": heads, "kv_heads": kv, "dim": dim, "vdim": vdim, "scale": scale or dim ** -0.5, "mask": {"size": size},
            "rot": {"base": base, "dims": rot_dims, "scaling": sc}}


def mamba(heads, vdim, state, groups, norm_groups, conv):
    return {"heads": heads, "vdim": vdim, "state": state, "groups": groups, "norm_groups": norm_groups, "conv": conv}


def wkv_layer(heads, dim, mlp=None):
    return {"type": "wkv", "mixer": {"heads": heads, "dim": dim}, "mlp": mlp}


def par_layer(left, right, mlp=None):
    return {"type": "parallel", "mixer": {"left": left, "right": right}, "mlp": mlp}


def ff(n, limit):
    return {"kind": "dense", "ff": n, "limit": limit}


def model(vocab, width, streams, layers, eps=1e-5, scale=3.5):
    return {"architecture": "Papidra", "vocab": vocab, "width": width, "streams": streams, "norm": {"eps": eps},
            "embedding": {"scale": scale}, "layers": layers}


# name -> (configuration, rank of the decay's low-rank pair)
CASES = {
    # different layers of each kind, feed-forward on a WKV layer, none on one parallel layer, padded heads of 32 / 48
    "mixed": (model(131, 96, 2, [par_layer(attn(4, 2, 32, 48, 24, 16), mamba(6, 24, 24, 3, 2, 3)),
                                 wkv_layer(3, 16, ff(80, 0.8)),
                                 par_layer(attn(6, 3, 64, 64, 40, 64), mamba(4, 32, 32, 1, 1, 4), ff(112, 2.0)),
                                 wkv_layer(2, 48)]), 16),
    # everything that can be one is one
    "ones": (model(64, 64, 1, [wkv_layer(1, 8), par_layer(attn(1, 1, 64, 64, 17, 2, scaling=False), mamba(1, 8, 8, 1, 1, 1), ff(24, 1.0))]), 8),
    # more query heads per kv head than one tile holds, wide state, five streams, five taps, sizes off the vector widths
    "wide": (model(77, 100, 5, [par_layer(attn(20, 1, 72, 40, 33, 36), mamba(2, 20, 136, 2, 1, 5), ff(36, 1.5)),
                                wkv_layer(2, 72)]), 12),
    # everything divides by two (tensor parallelism)
    "even": (model(96, 64, 2, [wkv_layer(2, 16), par_layer(attn(4, 2, 32, 48, 24, 16), mamba(4, 24, 24, 2, 2, 3), ff(256, 1.0))]), 8),
    "odd": (model(61, 90, 3, [wkv_layer(3, 10), par_layer(attn(3, 3, 20, 12, 19, 6), mamba(3, 14, 13, 1, 3, 2), ff(45, 0.7))]), 5),
}


def weights(cfg, rank, seed=0):
    """Random weights (rounded to bf16, like a checkpoint) scaled so that attention is peaked, sinks matter, decays span
    short and long memories and the gated unit meets its limits."""
    g = torch.Generator().manual_seed(seed)
    W = cfg["width"]
    out = {}

    def put(name, *shape, std=None, mean=0.0, uniform=None):
        if uniform:
            t = torch.rand(*shape, generator=g) * (uniform[1] - uniform[0]) + uniform[0]
        else:
            t = torch.randn(*shape, generator=g) * (std if std is not None else shape[-1] ** -0.5) + mean
        out[name] = t.to(torch.bfloat16)
    put("embed", cfg["vocab"], W, std=1.0)
    put("final.norm", W, std=0.2, mean=1.0)
    S = cfg["streams"]
    for i, l in enumerate(cfg["layers"]):
        p, m = f"l{i}.", l["mixer"]
        for q in (1, 2) if l["mlp"] is not None else (1,):
            put(f"{p}norm{q}", W, std=0.2, mean=1.0)
            put(f"{p}hc{q}.in", S, std=0.3, mean=1.0 / S)
            put(f"{p}hc{q}.out", S, std=0.3, mean=1.0)
            put(f"{p}hc{q}.mix", S, S, std=0.2)
            out[f"{p}hc{q}.mix"] = (out[f"{p}hc{q}.mix"].float() + 0.8 * torch.eye(S)).to(torch.bfloat16)
        if l["type"] == "wkv":
            n = m["heads"] * m["dim"]
            for s in "rkvgw":
                put(f"{p}mix.mu.{s}", W, uniform=(0.0, 1.0))
            for s in "rkvg":
                put(f"{p}mix.{s}", n, W)
            put(f"{p}mix.w1", rank, W)
            put(f"{p}mix.w2", n, rank)
            put(f"{p}mix.w0", n, uniform=(-6.0, 0.5))
            put(f"{p}mix.u", m["heads"], m["dim"], std=0.5)
            put(f"{p}mix.norm", n, std=0.2, mean=1.0)
            put(f"{p}mix.o", W, n)
        else:
            a, b = m["left"], m["right"]
            put(f"{p}mix.left.q", a["heads"] * a["dim"], W, std=2.0 * W ** -0.5)
            put(f"{p}mix.left.k", a["kv_heads"] * a["dim"], W, std=2.0 * W ** -0.5)
            put(f"{p}mix.left.v", a["kv_heads"] * a["vdim"], W)
            put(f"{p}mix.left.sink", a["heads"], std=1.5, mean=1.0)
            put(f"{p}mix.left.o", W, a["heads"] * a["vdim"])
            inner, gn = b["heads"] * b["vdim"], b["groups"] * b["state"]
            put(f"{p}mix.right.in", 2 * inner + 2 * gn + b["heads"], W)
            put(f"{p}mix.right.conv", inner + 2 * gn, b["conv"], std=0.6)
            put(f"{p}mix.right.conv.b", inner + 2 * gn, std=0.2)
            put(f"{p}mix.right.dt_bias", b["heads"], uniform=(-3.0, 0.0))
            put(f"{p}mix.right.A_log", b["heads"], uniform=(-2.0, 1.0))
            put(f"{p}mix.right.D", b["heads"], std=0.5, mean=1.0)
            put(f"{p}mix.right.norm", inner, std=0.2, mean=1.0)
            put(f"{p}mix.right.o", W, inner)
            put(f"{p}mix.left.out", W, std=0.2, mean=1.0)
            put(f"{p}mix.right.out", W, std=0.2, mean=1.0)
        if l["mlp"] is not None:
            n = l["mlp"]["ff"]
            put(f"{p}mlp.gate", n, W)
            put(f"{p}mlp.up", n, W)
            put(f"{p}mlp.down", W, n)
    return out


def write(folder, name, seed=0):
    """Configuration and checkpoint of case ``name`` under ``folder``; returns ``(cfg, weights)``."""
    from safetensors.torch import save_file
    cfg, rank = CASES[name]
    w = weights(cfg, rank, seed)
    os.makedirs(folder, exist_ok=True)
    with open(os.path.join(folder, "config.json"), "w") as f:
        json.dump(cfg, f)
    save_file({k: v.contiguous() for k, v in w.items()}, os.path.join(folder, "model.safetensors"))
    return cfg, w


def tokens(cfg, n, seed):
    return torch.randint(0, cfg["vocab"], (n,), generator=torch.Generator().manual_seed(1000 + seed)).tolist()


def portions(total, sizes):
    """Cut ``total`` into portions whose lengths cycle through ``sizes``."""
    out, at, i = [], 0, 0
    while at < total:
        n = min(sizes[i % len(sizes)], total - at)
        out.append(n)
        at += n
        i += 1
    return out


def feed_alone(engine, rid, toks, cuts):
    """Logits of every position of one request fed in portions, released at the end."""
    rows, at = [], 0
    for n in cuts:
        last = at + n == len(toks)
        rows.append(engine.feed([(rid, toks[at:at + n], list(range(n)))], [rid] if last else [])[0])
        at += n
    return torch.cat(rows)


def feed_together(engine, plans):
    """``plans``: ``{id: (tokens, cuts, first step)}``, all fed in common steps; logits of every position per id."""
    at = {r: 0 for r in plans}
    left = {r: list(c) for r, (_, c, _) in plans.items()}
    rows = {r: [] for r in plans}
    step = 0
    while any(left.values()):
        entries, end = [], []
        for r, (toks, _, start) in plans.items():
            if step < start or not left[r]:
                continue
            n = left[r].pop(0)
            entries.append((r, toks[at[r]:at[r] + n], list(range(n))))
            at[r] += n
            if not left[r]:
                end.append(r)
        for (r, _, _), lg in zip(entries, engine.feed(entries, end) if entries else []):
            rows[r].append(lg)
        step += 1
    return {r: torch.cat(v) for r, v in rows.items()}


def spread(a, b):
    """Largest difference of logits, means taken off, relative to the spread of ``b``."""
    d = (a.double() - b.double())
    d = d - d.mean(-1, keepdim=True)
    return (d.pow(2).mean(-1).sqrt().max() / b.double().std()).item()
