"""Plain fp64 statement of the Kenovik decoder, one function per mechanism.

Everything works on one whole sequence, token by token where the mechanism is a recurrence, and shares no code with the
package.  ``weights`` is a flat ``name -> tensor`` dict with the checkpoint's names, ``cfg`` the parsed ``config.json``
dictionary.
"""
import math

import torch


def rms_norm(x, w, eps):
    return x / torch.sqrt((x * x).mean(-1, keepdim=True) + eps) * w


def sigmoid(x):
    return 1.0 / (1.0 + torch.exp(-x))


def softplus(x):
    return torch.clamp(x, min=0) + torch.log1p(torch.exp(-x.abs()))


def gelu_tanh(z):
    return 0.5 * z * (1.0 + torch.tanh(math.sqrt(2.0 / math.pi) * (z + 0.044715 * z ** 3)))


# ------------------------------------------------------------------------------------------------- positions
def rotate_pairs(x, rot, positions):
    """x [T, heads, dim]; the first ``dims`` dimensions turn in pairs (2i, 2i + 1) by position times a frequency that a linear
    scaling divides."""
    n, base = rot["dims"], float(rot["base"])
    factor = float((rot.get("scaling") or {}).get("factor", 1.0))
    out = x.clone()
    for i in range(n // 2):
        a = positions.double() * (base ** (-2.0 * i / n) / factor)
        c, s = torch.cos(a)[:, None], torch.sin(a)[:, None]
        u, v = x[..., 2 * i], x[..., 2 * i + 1]
        out[..., 2 * i], out[..., 2 * i + 1] = u * c - v * s, v * c + u * s
    return out


def query_temperature(positions, temp):
    return torch.tensor([1.0 + temp["coef"] * math.log((p + 1) // temp["every"] + 1) for p in positions.tolist()], dtype=torch.float64)


def distance_bucket(n, rows, reach):
    """Row of the distance table for a key ``n`` tokens back: one row per distance for the near half, logarithmic beyond."""
    half = rows // 2
    if n < half:
        return n
    return min(rows - 1, half + math.floor(math.log(n / half) / math.log(reach / half) * (rows - half) + 1e-9))


def distance_bias(table, count, reach):
    """[heads, count, count]: what query i adds to its score of key j <= i."""
    rows = table.shape[0]
    per = torch.stack([table[distance_bucket(n, rows, reach)] for n in range(count)])          # [distance, heads]
    i = torch.arange(count)
    return per[(i[:, None] - i[None, :]).clamp(min=0)].permute(2, 0, 1)


# ------------------------------------------------------------------------------------------------- attention
def attend(q, k, v, scale, bias=None, one_more=False):
    """q [T, H, d], k / v [T, G, *]: causal softmax; ``one_more`` adds one to every denominator."""
    T, H = q.shape[:2]
    group = H // k.shape[1]
    outs = []
    seen = torch.arange(T)[None, :] <= torch.arange(T)[:, None]
    for h in range(H):
        s = q[:, h] @ k[:, h // group].t() * scale
        if bias is not None:
            s = s + bias[h]
        s = s.masked_fill(~seen, -math.inf)
        top = s.max(-1, keepdim=True).values
        if one_more:
            top = top.clamp(min=0.0)
        e = torch.exp(s - top)
        den = e.sum(-1, keepdim=True) + (torch.exp(-top) if one_more else 0.0)
        outs.append(e / den @ v[:, h // group])
    return torch.stack(outs, 1)


def sink_attention(h, m, w, pre):
    T = h.shape[0]
    pos = torch.arange(T)
    lin = lambda n: h @ w[pre + n].t() + w[pre + n + ".b"]
    q = rotate_pairs(lin("q").view(T, m["heads"], m["dim"]), m["rot"], pos)
    k = rotate_pairs(lin("k").view(T, m["kv_heads"], m["dim"]), m["rot"], pos)
    v = lin("v").view(T, m["kv_heads"], m["vdim"])
    return attend(q, k, v, m["scale"], one_more=True).reshape(T, -1) @ w[pre + "o"].t()


def distance_attention(h, m, w, pre, eps):
    T = h.shape[0]
    q = rms_norm(h @ w[pre + "q"].t(), w[pre + "q.norm"], eps) * query_temperature(torch.arange(T), m["q_temp"])[:, None]
    k = rms_norm(h @ w[pre + "k"].t(), w[pre + "k.norm"], eps)
    v = h @ w[pre + "v"].t()
    o = attend(q.view(T, m["heads"], m["dim"]), k.view(T, m["kv_heads"], m["dim"]), v.view(T, m["kv_heads"], m["vdim"]), m["scale"],
               bias=distance_bias(w[pre + "rel"], T, m["bias_max"]))
    return o.reshape(T, -1) @ w[pre + "o"].t()


# ------------------------------------------------------------------------------------------------- recurrence
def causal_conv(x, taps, bias):
    """x [T, C], taps [C, n] with the current token's tap last."""
    n = taps.shape[1]
    out = []
    for t in range(x.shape[0]):
        y = bias.clone()
        for j in range(n):
            s = t - (n - 1) + j
            if s >= 0:
                y = y + taps[:, j] * x[s]
        out.append(y)
    return torch.stack(out)


def block_gate(u, w, b):
    """Sigmoid of one square matrix per block of channels: u [T, C], w [blocks, n, n] as [out, in]."""
    blocks, n = w.shape[:2]
    return torch.cat([sigmoid(u[:, i * n:(i + 1) * n] @ w[i].t() + b[i]) for i in range(blocks)], -1)


def gated_linear_recurrence(u, r, i, lam):
    """S = a S + sqrt(1 - a^2) i u with log a = -8 r softplus(lam); returns every state."""
    log_a = -8.0 * r * softplus(lam)
    a, drive = torch.exp(log_a), torch.sqrt(-torch.expm1(2.0 * log_a)) * i * u
    s, out = torch.zeros_like(lam), []
    for t in range(u.shape[0]):
        s = a[t] * s + drive[t]
        out.append(s)
    return torch.stack(out)


def recurrent_block(h, w, pre):
    y = gelu_tanh(h @ w[pre + "y"].t() + w[pre + "y.b"])
    u = causal_conv(h @ w[pre + "x"].t() + w[pre + "x.b"], w[pre + "conv"], w[pre + "conv.b"])
    s = gated_linear_recurrence(u, block_gate(u, w[pre + "ra"], w[pre + "ra.b"]), block_gate(u, w[pre + "ri"], w[pre + "ri.b"]), w[pre + "lam"])
    return (s * y) @ w[pre + "o"].t()


# ------------------------------------------------------------------------------------------------- feed-forward
def silu_mlp(h, w, pre):
    g = h @ w[pre + "gate"].t()
    return (g * sigmoid(g) * (h @ w[pre + "up"].t())) @ w[pre + "down"].t()


def clamped_mlp(h, w, pre, limit):
    g = torch.clamp(h @ w[pre + "gate"].t(), max=limit)
    u = torch.clamp(h @ w[pre + "up"].t(), min=-limit, max=limit)
    return (g * sigmoid(1.702 * g) * (u + 1.0)) @ w[pre + "down"].t()


def route(h, router, w, pre):
    """(expert ids, weights) of every token: choice by corrected scores inside the best groups, weights by plain scores."""
    s = sigmoid(h @ w[pre + "router"].t())
    choice = s + w[pre + "correction"]
    E, groups = router["experts"], router.get("groups") or {"count": 1, "keep": 1}
    size = E // groups["count"]
    ids, weights = [], []
    for t in range(h.shape[0]):
        score = [sum(sorted(choice[t, g * size:(g + 1) * size].tolist(), reverse=True)[:2]) for g in range(groups["count"])]
        best = sorted(range(groups["count"]), key=lambda g: -score[g])[:groups["keep"]]
        open_ = [e for e in range(E) if e // size in best]
        pick = sorted(open_, key=lambda e: -choice[t, e].item())[:router["top"]]
        p = s[t, pick]
        ids.append(pick)
        weights.append(p / (p.sum() + 1e-20) * router["scale"])
    return ids, torch.stack(weights)


def experts(h, mlp, w, pre):
    ids, weights = route(h, mlp["router"], w, pre)
    out = []
    for t in range(h.shape[0]):
        y = sum(weights[t, j] * clamped_mlp(h[t], w, f"{pre}e{e}.", mlp["expert"]["limit"]) for j, e in enumerate(ids[t]))
        out.append(y)
    out = torch.stack(out)
    if mlp.get("shared"):
        out = out + clamped_mlp(h, w, pre + "shared.", mlp["shared"]["limit"])
    return out


# ------------------------------------------------------------------------------------------------- model
def layer_runs(cfg):
    """(layer, pass or None) in the order of execution; a pass number stands with the first layer of every pass."""
    n, loop = len(cfg["layers"]), cfg.get("loop")
    if not loop:
        return [(i, None) for i in range(n)]
    a, b = loop["start"], loop["stop"]
    runs = [(i, None) for i in range(a)]
    for t in range(loop["times"]):
        runs += [(i, t if i == a else None) for i in range(a, b)]
    return runs + [(i, None) for i in range(b, n)]


def forward(weights, cfg, tokens):
    """Logits [T, vocab] and the residual after every layer run."""
    w = {k: v.double() for k, v in weights.items()}
    eps = cfg["norm"]["eps"]
    x = w["embed"][torch.as_tensor(tokens)] * cfg["embedding"]["scale"]
    after = []
    for i, t in layer_runs(cfg):
        lc, pre = cfg["layers"][i], f"l{i}."
        if t is not None:
            x = x + w["loop.step"][t]
        h, m = rms_norm(x, w[pre + "norm1"], eps), lc["mixer"]
        if lc["type"] == "attention":
            x = x + sink_attention(h, m, w, pre + "mix.")
        elif lc["type"] == "attention_2":
            x = x + distance_attention(h, m, w, pre + "mix.", eps)
        else:
            x = x + recurrent_block(h, w, pre + "mix.")
        if lc.get("mlp"):
            h = rms_norm(x, w[pre + "norm2"], eps)
            x = x + (silu_mlp(h, w, pre + "mlp.") if lc["mlp"].get("kind", "dense") == "dense" else experts(h, lc["mlp"], w, pre + "mlp."))
        after.append(x)
    return rms_norm(x, w["final.norm"], eps) @ w["embed"].t(), after
