"""Small Bisudra configurations with random weights, shared by the CPU and GPU tests."""
import json
import os

import torch

from papidra_cases import feed_alone, feed_together, portions, spread, tokens  # noqa: F401


def attention(heads, kv, dim, vdim, size, rot, mlp=None, diff=0.3, scale=None, base=1e4):
    return {"type": "attention", "mixer": {"heads": heads, "kv_heads": kv, "dim": dim, "vdim": vdim, "diff": diff, "scale": scale or dim ** -0.5,
                                           "mask": {"size": size}, "rot": {"base": base, "dims": rot}}, "mlp": mlp}


def ff(n):
    return {"kind": "dense", "ff": n}


def moe(experts, top, n):
    return {"kind": "moe", "expert": {"ff": n}, "router": {"experts": experts, "top": top}}


def model(vocab, width, taps, side, layers, eps=1e-5):
    return {"architecture": "Bisudra", "vocab": vocab, "width": width, "norm": {"eps": eps}, "canon": {"taps": taps}, "token_side": {"dim": side},
            "layers": layers}


CASES = {
    # layers that differ in everything, one without a feed-forward, windows that end inside pages, values wider and narrower than maps
    "mixed": model(131, 96, 4, 20, [attention(6, 2, 20, 36, 21, 12, ff(72), 0.2), attention(4, 1, 32, 24, 50, 32, moe(9, 4, 24), 0.55),
                                    attention(3, 3, 8, 40, 33, 4, None, 0.1, scale=0.5, base=500.0), attention(8, 2, 16, 16, 17, 8, moe(5, 2, 40), 0.7)]),
    # everything that can be one is one
    "ones": model(64, 64, 1, 1, [attention(1, 1, 8, 8, 1, 2, moe(1, 1, 8)), attention(1, 1, 32, 64, 40, 2, ff(1)), attention(1, 1, 2, 1, 7, 2, None)]),
    # cached keys and values of 256, many query rows on one key / value head, widths off the vector sizes
    "wide": model(77, 100, 2, 13, [attention(20, 1, 70, 130, 33, 70, moe(20, 5, 36)), attention(9, 1, 33, 50, 60, 20, ff(50), 0.4),
                                   attention(2, 2, 128, 256, 45, 64, moe(3, 3, 50))]),
    # sizes that every tensor-core path takes; a window over the whole sequence
    "aligned": model(96, 128, 4, 32, [attention(4, 2, 32, 64, 40, 16, ff(128)), attention(8, 1, 64, 128, 500, 64, moe(8, 2, 64)),
                                      attention(4, 1, 64, 64, 48, 64, moe(4, 1, 128), 0.6)]),
    # everything divides by two (tensor parallelism)
    "even": model(96, 64, 3, 10, [attention(4, 2, 16, 24, 18, 16, ff(256)), attention(2, 1, 16, 32, 30, 8, moe(4, 2, 16), 0.5), attention(4, 4, 8, 16, 9, 8, ff(48))]),
    "odd": model(61, 90, 7, 7, [attention(3, 3, 10, 12, 19, 6, moe(7, 2, 45)), attention(5, 1, 15, 9, 26, 14, ff(33), 0.45)], eps=1e-3),
}


def weights(cfg, seed=0):
    """Random weights (rounded to bf16, like a checkpoint), scaled so that attention is peaked, the maps differ, gates open and close and
    every layer's result counts in every later sum.  The routers read channels of the embedding that no sublayer writes (their norm
    weights and biases are zero there, and every layer hands them on as they are), so that no choice of an expert turns on rounding."""
    g = torch.Generator().manual_seed(seed)
    W, taps, side = cfg["width"], cfg["canon"]["taps"], cfg["token_side"]["dim"]
    out = {}

    def put(name, *shape, std=None, mean=0.0):
        t = torch.randn(*shape, generator=g) * (std if std is not None else shape[-1] ** -0.5) + mean
        out[name] = t.to(torch.bfloat16)
    kept = W - max(4, min(16, W // 4))

    def norm(name):
        put(name, W, std=0.2, mean=1.0)
        put(name + ".b", W, std=0.2)
        out[name][kept:] = 0.0
        out[name + ".b"][kept:] = 0.0
    put("embed", cfg["vocab"], W, std=1.0)
    put("side.embed", cfg["vocab"], side * len(cfg["layers"]), std=1.0)
    put("final.norm", W, std=0.2, mean=1.0)
    put("final.norm.b", W, std=0.2)
    for i, l in enumerate(cfg["layers"]):
        p, m = f"l{i}.", l["mixer"]
        H, G, D, V = m["heads"], m["kv_heads"], m["dim"], m["vdim"]
        norm(p + "norm1")
        x = p + "mix."
        put(x + "q", H * 2 * D, W)
        put(x + "k", G * 2 * D, W)
        put(x + "v", G * V, W)
        put(x + "q.norm", D, std=0.3, mean=1.4)
        put(x + "k.norm", D, std=0.3, mean=1.3)
        for n in ("lq1", "lk1", "lq2", "lk2"):
            put(x + n, D, std=0.6 * D ** -0.25)
        put(x + "g", H * V, W, std=2 * W ** -0.5)
        put(x + "o", W, H * V)
        put(p + "canon1", W, taps, std=0.5)
        put(p + "rg1", W, W, std=2 * W ** -0.5)
        put(p + "rg1.b", W, std=1.0)
        put(p + "side.gate", side, W)
        put(p + "side.proj", W, side)
        put(p + "side.norm", W, std=0.2, mean=0.5)
        out[p + "side.norm"][kept:] = 0.0
        share = torch.rand(i + 2, generator=g) * 0.6 - 0.2
        share[-1] += 0.7
        out[p + "dwa"] = share.to(torch.bfloat16)
        if l["mlp"] is None:
            continue
        norm(p + "norm2")
        put(p + "rg2", W, W, std=2 * W ** -0.5)
        put(p + "rg2.b", W, std=1.0)
        if l["mlp"]["kind"] == "dense":
            n = l["mlp"]["ff"]
            put(p + "mlp.up", n, W)
            put(p + "mlp.up.b", n, std=0.5)
            put(p + "mlp.down", W, n)
            put(p + "mlp.down.b", W, std=0.5)
            continue
        n, E = l["mlp"]["expert"]["ff"], l["mlp"]["router"]["experts"]
        put(p + "mlp.router", E, W, std=3 * (W - kept) ** -0.5)
        out[p + "mlp.router"][:, :kept] = 0.0
        put(p + "mlp.router.b", E, std=0.7)
        for e in range(E):
            put(f"{p}mlp.e{e}.gate", n, W)
            put(f"{p}mlp.e{e}.up", n, W)
            put(f"{p}mlp.e{e}.down", W, n)
    return out


def write(folder, name, seed=0):
    """Configuration and checkpoint of case ``name`` under ``folder``; returns ``(cfg, weights)``."""
    return write_model(folder, CASES[name], seed)


def write_model(folder, cfg, seed=0, change=None):
    """``change(weights)`` may alter the weights before they are written."""
    from safetensors.torch import save_file
    w = weights(cfg, seed)
    if change is not None:
        change(w)
    os.makedirs(folder, exist_ok=True)
    with open(os.path.join(folder, "config.json"), "w") as f:
        json.dump(cfg, f)
    save_file({k: v.contiguous() for k, v in w.items()}, os.path.join(folder, "model.safetensors"))
    return cfg, w


# ------------------------------------------------------------------------------------------------- one key that stands out
def standing_out(device, dtype, heads, kv, dim, vdim, size, rot, total, rows, key, map_index, seed=0):
    """Attention of the last ``rows`` positions of a sequence of ``total`` tokens through the package's map and attention operations on
    scattered pages, with one loud pair: the last query and the key at position ``key`` point the same way in one map, so that this
    key takes nearly all of the weight where it is visible.  Returns ``(got, want)`` ``[rows, heads, 2, vdim]``."""
    import bisudra_oracle as O
    from atlas_b200 import ops
    from atlas_b200.config import padded_head_width
    from atlas_b200.models import ForwardBatch
    from atlas_b200.models.decoder import alloc_kv
    from atlas_b200.ops import reference as ref
    g = torch.Generator().manual_seed(seed)
    D, bs = padded_head_width(2 * dim, vdim), 16
    table = torch.randperm((total + bs - 1) // bs + 3, generator=g).tolist()
    q, k, v = (torch.randn(total, *s, generator=g).to(dtype) for s in ((heads, 2, dim), (kv, 2, dim), (kv, vdim)))
    eps, qn, kn = 1e-6, torch.full((dim,), 1.0), torch.full((dim,), 1.0)
    turns = {"base": 1e4, "dims": rot}
    pos = torch.arange(total)
    unit = lambda x, p: O.rotate_pairs(O.unit_rms(x.double(), eps), turns, p)
    # the query that the loud key answers: its rotation taken off again, so that the rotated ones agree
    loud = unit(k[key:key + 1], pos[key:key + 1])[0, 0, map_index]
    back = O.rotate_pairs(loud.view(1, 1, dim), turns, -pos[-1:])[0, 0]
    q[-1, :, map_index] = back.to(dtype)
    scale = 40.0 / dim
    order = torch.cat([torch.arange(0, rot, 2), torch.arange(1, rot, 2), torch.arange(rot, dim)])      # half-split pairs
    kc, vc = alloc_kv(len(table), bs, kv, D, dtype, device)
    rope = ref.build_rope_cache(rot, total, turns["base"], None, device)
    got = []
    for lo, hi in ((0, total - rows), (total - rows, total)):
        if lo == hi:
            continue
        fb = ForwardBatch.build([[0] * (hi - lo)], [lo], [table], bs, device=device)
        part = lambda x, o: (x[lo:hi] if o is None else x[lo:hi][..., o]).contiguous().to(device)
        rq = ops.map_norm_kv_write(part(q, order), part(k, order), part(v, None), fb.positions, rope, rot, kc, vc, fb.slot_mapping, qn.to(device),
                                   kn.to(device), eps)
        got = ops.paged_attention(rq, kc, vc, fb, scale, sliding_window=size or None)
    got = got.view(rows, heads, 2, D)[..., :vdim].cpu().double()
    held = lambda x: unit(x, pos).to(dtype).double()                  # queries and cached keys are held in the activations' dtype
    want = O.map_outputs(held(q), held(k), v.double(), scale, O.window(total, size))[-rows:]
    return got, want
