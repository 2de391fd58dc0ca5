"""Plain fp64 statement of the Bisudra decoder, one function per mechanism.

Everything works on one whole sequence and shares no code with the package.  ``weights`` is a flat ``name -> tensor`` dict with
the checkpoint's names, ``cfg`` the parsed ``config.json`` dictionary.
"""
import math

import torch


def sigmoid(x):
    return 1.0 / (1.0 + torch.exp(-x))


def gelu_tanh(z):
    return 0.5 * z * (1.0 + torch.tanh(math.sqrt(2.0 / math.pi) * (z + 0.044715 * z ** 3)))


def silu(z):
    return z * sigmoid(z)


def unit_rms(x, eps):
    return x / torch.sqrt((x * x).mean(-1, keepdim=True) + eps)


def layer_norm(x, w, b, eps):
    d = x - x.mean(-1, keepdim=True)
    return d / torch.sqrt((d * d).mean(-1, keepdim=True) + eps) * w + b


# ------------------------------------------------------------------------------------------------- mixer input
def causal_taps(h, w):
    """Depth-wise causal convolution of h [T, W] with w [W, taps]; zeros ahead of the sequence."""
    T, taps = h.shape[0], w.shape[1]
    out = torch.zeros_like(h)
    for t in range(T):
        for j in range(taps):
            s = t - taps + 1 + j
            if s >= 0:
                out[t] += w[:, j] * h[s]
    return out


def input_convolution(h, w):
    return h + causal_taps(h, w)


# ------------------------------------------------------------------------------------------------- attention
def rotate_pairs(x, rot, positions):
    """x [T, ..., dim]; the first ``dims`` dimensions turn in pairs (2i, 2i + 1)."""
    n = rot["dims"]
    out = x.clone()
    shape = (-1,) + (1,) * (x.dim() - 2)
    for i in range(n // 2):
        a = (positions.double() * float(rot["base"]) ** (-2.0 * i / n)).view(shape)
        c, s = torch.cos(a).to(x.dtype), torch.sin(a).to(x.dtype)
        u, v = x[..., 2 * i], x[..., 2 * i + 1]
        out[..., 2 * i], out[..., 2 * i + 1] = u * c - v * s, v * c + u * s
    return out


def window(n, size):
    """Position i sees the ``size`` tokens that end with itself (all of them without a size)."""
    i = torch.arange(n)
    d = i[:, None] - i[None, :]
    return (d >= 0) & (d < size) if size else d >= 0


def softmax_visible(scores, visible):
    s = scores.masked_fill(~visible, -math.inf)
    e = torch.exp(s - s.max(-1, keepdim=True).values)
    return e / e.sum(-1, keepdim=True)


def mix_factor(lq1, lk1, lq2, lk2, diff):
    """Weight of the second map's output."""
    return math.exp(float((lq1 * lk1).sum())) - math.exp(float((lq2 * lk2).sum())) + diff


def map_outputs(q, k, v, scale, visible):
    """q [T, H, 2, dim], k [T, G, 2, dim], v [T, G, vdim] -> both maps' outputs [T, H, 2, vdim]."""
    H, G = q.shape[1], k.shape[1]
    rows = []
    for a in range(H):
        g = a // (H // G)
        rows.append(torch.stack([softmax_visible(q[:, a, m] @ k[:, g, m].T * scale, visible) @ v[:, g] for m in range(2)], 1))
    return torch.stack(rows, 1)


def difference(o, lam, diff, eps):
    """o [T, H, 2, vdim] -> [T, H, vdim]."""
    return unit_rms(o[:, :, 0] - lam * o[:, :, 1], eps) * (1.0 - diff)


def differential_attention(h, w, pre, m, eps):
    T, H, G, D, V = h.shape[0], m["heads"], m["kv_heads"], m["dim"], m["vdim"]
    pos = torch.arange(T)
    q = (h @ w[pre + "q"].T).view(T, H, 2, D)
    k = (h @ w[pre + "k"].T).view(T, G, 2, D)
    v = (h @ w[pre + "v"].T).view(T, G, V)
    q = rotate_pairs(unit_rms(q, eps) * w[pre + "q.norm"], m["rot"], pos)
    k = rotate_pairs(unit_rms(k, eps) * w[pre + "k.norm"], m["rot"], pos)
    o = map_outputs(q, k, v, m["scale"], window(T, m["mask"]["size"] if m.get("mask") else 0))
    lam = mix_factor(*(w[pre + n] for n in ("lq1", "lk1", "lq2", "lk2")), m["diff"])
    o = difference(o, lam, m["diff"], eps).reshape(T, H * V)
    return (o * sigmoid(h @ w[pre + "g"].T)) @ w[pre + "o"].T


# ------------------------------------------------------------------------------------------------- feed-forward
def squared_relu_mlp(h, w, pre):
    u = torch.clamp(h @ w[pre + "up"].T + w[pre + "up.b"], min=0)
    return (u * u) @ w[pre + "down"].T + w[pre + "down.b"]


def route(h, w_router, bias, top):
    """Expert numbers [T, top] and their weights: the softmax over the chosen logits."""
    z = h @ w_router.T + bias
    best = torch.sort(z, dim=-1, descending=True, stable=True)
    chosen = best.values[:, :top]
    e = torch.exp(chosen - chosen[:, :1])
    return best.indices[:, :top], e / e.sum(-1, keepdim=True)


def expert(h, gate, up, down):
    return (silu(h @ gate.T) * (h @ up.T)) @ down.T


def mixture(h, w, pre, mlp):
    ids, weight = route(h, w[pre + "router"], w[pre + "router.b"], mlp["router"]["top"])
    out = torch.zeros_like(h)
    for t in range(h.shape[0]):
        for e, p in zip(ids[t].tolist(), weight[t]):
            out[t] += p * expert(h[t:t + 1], *(w[f"{pre}e{e}.{n}"] for n in ("gate", "up", "down")))[0]
    return out


def feed_forward(h, w, pre, mlp):
    return mixture(h, w, pre, mlp) if mlp.get("kind", "dense") == "moe" else squared_relu_mlp(h, w, pre)


# ------------------------------------------------------------------------------------------------- layer
def gated(y, h, w, name):
    return y * sigmoid(h @ w[name].T + w[name + ".b"])


def token_side(x, e, w, pre, eps):
    """x plus the normed projection of the layer's share e [T, dim] of the tokens' side embeddings, gated by x."""
    g = gelu_tanh(x @ w[pre + "side.gate"].T) * e
    return x + unit_rms(g @ w[pre + "side.proj"].T, eps) * w[pre + "side.norm"]


def depth_average(states, factors):
    return sum(f * s for f, s in zip(factors, states))


def layer(x, e, w, pre, lc, eps):
    """One layer ahead of the depth average."""
    y = differential_attention(input_convolution(x, w[pre + "canon1"]), w, pre + "mix.", lc["mixer"], eps)
    x = x + layer_norm(gated(y, x, w, pre + "rg1"), w[pre + "norm1"], w[pre + "norm1.b"], eps)
    if lc.get("mlp") is not None:
        y = feed_forward(x, w, pre + "mlp.", lc["mlp"])
        x = x + layer_norm(gated(y, x, w, pre + "rg2"), w[pre + "norm2"], w[pre + "norm2.b"], eps)
    return token_side(x, e, w, pre, eps)


def forward(cfg, weights, tokens, layers=None):
    """Logits [T, vocab] in fp64; ``layers`` (a list) receives the stream after every layer."""
    w = {k: v.double() for k, v in weights.items()}
    eps, n = cfg["norm"]["eps"], cfg["token_side"]["dim"]
    ids = torch.as_tensor(tokens)
    side = w["side.embed"][ids]
    x = w["embed"][ids]
    states = [x]
    for i, lc in enumerate(cfg["layers"]):
        pre = f"l{i}."
        states.append(layer(x, side[:, i * n:(i + 1) * n], w, pre, lc, eps))
        x = depth_average(states, w[pre + "dwa"])
        if layers is not None:
            layers.append(x)
    return layer_norm(x, w["final.norm"], w["final.norm.b"], eps) @ w["embed"].T
