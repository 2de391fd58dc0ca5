"""Plain fp64 statement of the Tomizen decoder, one function per mechanism.

Everything works on one whole sequence, token by token where the mechanism is a recurrence, and shares no code with the
package.  ``weights`` is a flat ``name -> tensor`` dict with the checkpoint's names, ``cfg`` the parsed ``config.json``
dictionary.
"""
import math

import torch


def unit_rms(x, eps):
    return x / torch.sqrt((x * x).mean(-1, keepdim=True) + eps)


def sigmoid(x):
    return 1.0 / (1.0 + torch.exp(-x))


def log_sigmoid(x):
    return -(torch.clamp(-x, min=0) + torch.log1p(torch.exp(-x.abs())))


def output_norm(y, w, eps):
    """Norm of a sublayer's output; the weight is stored around zero."""
    return unit_rms(y, eps) * (1.0 + w)


# ------------------------------------------------------------------------------------------------- rotation
def frequencies(rot):
    """Rotation frequencies [dims / 2] and the factor on cos / sin, blended by YaRN where ``scaling`` is given."""
    n, base = rot["dims"], float(rot["base"])
    plain = [base ** (-2.0 * i / n) for i in range(n // 2)]
    sc = rot.get("scaling")
    if not sc:
        return plain, 1.0

    def dim(turns):
        return n * math.log(sc["original"] / (2.0 * math.pi * turns)) / (2.0 * math.log(base))
    lo, hi = max(math.floor(dim(sc["fast"])), 0), min(math.ceil(dim(sc["slow"])), n - 1)
    blended = []
    for i, f in enumerate(plain):
        ramp = min(max((i - lo) / max(hi - lo, 0.001), 0.0), 1.0)
        blended.append(f / sc["factor"] * ramp + f * (1.0 - ramp))
    return blended, 0.1 * math.log(sc["factor"]) + 1.0


def rotate_pairs(x, rot, positions):
    """x [T, heads, dim]; the first ``dims`` dimensions turn in pairs (2i, 2i + 1)."""
    f, mul = frequencies(rot)
    n = rot["dims"]
    out = x.clone()
    for i, fi in enumerate(f):
        a = positions.double() * fi
        c, s = (torch.cos(a) * mul)[:, None].to(x.dtype), (torch.sin(a) * mul)[:, None].to(x.dtype)
        u, v = x[..., 2 * i], x[..., 2 * i + 1]
        out[..., 2 * i], out[..., 2 * i + 1] = u * c - v * s, v * c + u * s
    assert 2 * len(f) == n
    return out


# ------------------------------------------------------------------------------------------------- attention
def causal(n):
    i = torch.arange(n)
    return i[None, :] <= i[:, None]


def window(n, size):
    """Position i sees the ``size`` tokens that end with itself."""
    i = torch.arange(n)
    d = i[:, None] - i[None, :]
    return (d >= 0) & (d < size)


def softmax_visible(scores, visible):
    s = scores.masked_fill(~visible, -math.inf)
    e = torch.exp(s - s.max(-1, keepdim=True).values)
    return e / e.sum(-1, keepdim=True)


def soft_cap(s, cap):
    return cap * torch.tanh(s / cap)


def latent_heads(qu, qr, c, kr, w_uk, w_uv, scale, visible):
    """qu [T, H, dim], qr [T, H, rot] (turned), c [T, R], kr [T, rot] (turned) -> [T, H, vdim]."""
    T, H, D = qu.shape
    ku = (c @ w_uk.T).view(T, H, D)
    v = (c @ w_uv.T).view(T, H, -1)
    outs = []
    for a in range(H):
        s = (qu[:, a] @ ku[:, a].T + qr[:, a] @ kr.T) * scale
        outs.append(softmax_visible(s, visible) @ v[:, a])
    return torch.stack(outs, 1)


def latent_attention(h, w, pre, m, eps):
    T, H, D, R, RO = h.shape[0], m["heads"], m["dim"], m["kv_rank"], m["rot_dim"]
    pos = torch.arange(T)
    q = (h @ w[pre + "q"].T).view(T, H, D + RO)
    down = h @ w[pre + "dkv"].T
    c = unit_rms(down[:, :R], eps) * w[pre + "dkv.norm"]
    kr = rotate_pairs(down[:, None, R:], m["rot"], pos)[:, 0]
    qr = rotate_pairs(q[..., D:], m["rot"], pos)
    vis = window(T, m["mask"]["size"]) if m.get("mask") else causal(T)
    o = latent_heads(q[..., :D], qr, c, kr, w[pre + "uk"], w[pre + "uv"], m["scale"], vis)
    return o.reshape(T, -1) @ w[pre + "o"].T


def capped_heads(q, k, v, scale, cap, visible):
    """q [T, H, D], k [T, G, D], v [T, G, V] -> [T, H, V]."""
    H, G = q.shape[1], k.shape[1]
    outs = []
    for a in range(H):
        b = a // (H // G)
        s = (q[:, a] @ k[:, b].T) * scale
        outs.append(softmax_visible(soft_cap(s, cap) if cap else s, visible) @ v[:, b])
    return torch.stack(outs, 1)


def attention(h, w, pre, m, eps):
    T, H, G, D, V = h.shape[0], m["heads"], m["kv_heads"], m["dim"], m["vdim"]
    q = unit_rms((h @ w[pre + "q"].T).view(T, H, D), eps) * w[pre + "q.norm"]
    k = unit_rms((h @ w[pre + "k"].T).view(T, G, D), eps) * w[pre + "k.norm"]
    v = (h @ w[pre + "v"].T).view(T, G, V)
    o = capped_heads(q, k, v, m["scale"], m["softcap"], causal(T))
    o = o * sigmoid(h @ w[pre + "g"].T)[:, :, None]
    return o.reshape(T, H * V) @ w[pre + "o"].T


# ------------------------------------------------------------------------------------------------- mLSTM
def log_gates(i_raw, f_raw, cap):
    return soft_cap(i_raw, cap), log_sigmoid(soft_cap(f_raw, cap))


def matrix_memory(q, k, v, i, f, state=None):
    """q (scaled) / k [T, H, D], v [T, H, V], log gates i / f [T, H] -> (o [T, H, V], (S, n, m))."""
    T, H, D = q.shape
    if state is None:
        S, n, m = (torch.zeros(H, D, v.shape[-1], dtype=q.dtype), torch.zeros(H, D, dtype=q.dtype), torch.zeros(H, dtype=q.dtype))
    else:
        S, n, m = (t.clone() for t in state)
    out = torch.zeros(T, H, v.shape[-1], dtype=q.dtype)
    for t in range(T):
        new = torch.maximum(f[t] + m, i[t])
        keep, add = torch.exp(f[t] + m - new), torch.exp(i[t] - new)
        m = new
        S = keep[:, None, None] * S + add[:, None, None] * k[t][:, :, None] * v[t][:, None, :]
        n = keep[:, None] * n + add[:, None] * k[t]
        den = torch.maximum((n * q[t]).sum(-1).abs(), torch.exp(-m)) + 1e-6
        out[t] = (S * q[t][:, :, None]).sum(1) / den[:, None]
    return out, (S, n, m)


def mlstm(h, w, pre, m, eps):
    T, H, D, V = h.shape[0], m["heads"], m["dim"], m["vdim"]
    q = (h @ w[pre + "q"].T).view(T, H, D) * D ** -0.5
    k = (h @ w[pre + "k"].T).view(T, H, D)
    v = (h @ w[pre + "v"].T).view(T, H, V)
    i, f = log_gates(h @ w[pre + "i"].T + w[pre + "i.b"], h @ w[pre + "f"].T + w[pre + "f.b"], m["gate_cap"])
    o, _ = matrix_memory(q, k, v, i, f)
    y = unit_rms(o, eps).reshape(T, H * V) * w[pre + "norm"] * sigmoid(h @ w[pre + "g"].T)
    return y @ w[pre + "o"].T


# ------------------------------------------------------------------------------------------------- experts, layers
def expert(h, up, down):
    return torch.square(torch.clamp(h @ up.T, min=0)) @ down.T


def route(z, top):
    """Softmax over all experts; the ``top`` best keep their scores as they are."""
    e = torch.exp(z - z.max(-1, keepdim=True).values)
    s = e / e.sum(-1, keepdim=True)
    return torch.topk(s, top, dim=-1)


def experts(h, w, pre, mlp):
    weights, ids = route(h @ w[pre + "router"].T, mlp["router"]["top"])
    out = torch.zeros_like(h)
    for t in range(h.shape[0]):
        for wt, e in zip(weights[t], ids[t].tolist()):
            out[t] = out[t] + wt * expert(h[t], w[f"{pre}e{e}.up"], w[f"{pre}e{e}.down"])
    return out


MIXERS = {"mlstm": mlstm, "latent_attention": latent_attention, "attention": attention}


def forward(cfg, weights, tokens, layers_out=None, dtype=torch.float64):
    """Logits [T, vocab] of every position; ``layers_out`` (a list) collects the residual stream after every layer."""
    w = {n: t.to(dtype) for n, t in weights.items()}
    eps = cfg["norm"]["eps"]
    x = w["embed"][torch.tensor(tokens)]
    for i, lc in enumerate(cfg["layers"]):
        pre = f"l{i}."
        x = x + output_norm(MIXERS[lc["type"]](x, w, pre + "mix.", lc["mixer"], eps), w[pre + "norm1"], eps)
        if lc["mlp"] is not None:
            x = x + output_norm(experts(x, w, pre + "mlp.", lc["mlp"]), w[pre + "norm2"], eps)
        if layers_out is not None:
            layers_out.append(x)
    return output_norm(x, w["final.norm"], eps) @ w["head"].T
