"""Plain fp32/fp64 statement of the Papidra decoder, one function per mechanism.

Everything works on one whole sequence at a time, token by token where the mechanism is a recurrence, and shares no code
with the package.  ``weights`` is a flat ``name -> tensor`` dict with the checkpoint's names, ``cfg`` the parsed
``config.json`` dictionary.
"""
import math

import torch


def rms(x, eps):
    return x / torch.sqrt((x * x).mean(-1, keepdim=True) + eps)


def sigmoid(x):
    return 1.0 / (1.0 + torch.exp(-x))


def silu(x):
    return x * sigmoid(x)


# ------------------------------------------------------------------------------------------------- rotation
def rope_frequencies(rot):
    """Rotation frequencies [dims / 2] and the factor on cos / sin, YaRN-blended where ``scaling`` is given."""
    n, base = rot["dims"], float(rot["base"])
    f = [base ** (-2.0 * i / n) for i in range(n // 2)]
    sc = rot.get("scaling")
    if not sc:
        return f, 1.0

    def where(turns):
        return n * math.log(sc["original"] / (2 * math.pi * turns)) / (2 * math.log(base))
    lo = max(math.floor(where(sc["fast"])), 0)
    hi = min(math.ceil(where(sc["slow"])), n - 1)
    out = []
    for i, fi in enumerate(f):
        ramp = min(max((i - lo) / max(hi - lo, 0.001), 0.0), 1.0)
        out.append(fi / sc["factor"] * ramp + fi * (1.0 - ramp))
    return out, 0.1 * math.log(sc["factor"]) + 1.0


def rotate(x, rot, positions):
    """x [T, heads, dim]; the first ``dims`` dimensions turn, pairing i with i + dims / 2."""
    f, mul = rope_frequencies(rot)
    n = rot["dims"]
    ang = positions.double()[:, None] * torch.tensor(f, dtype=torch.float64)[None, :]
    c, s = (torch.cos(ang) * mul).to(x.dtype)[:, None, :], (torch.sin(ang) * mul).to(x.dtype)[:, None, :]
    u, v = x[..., :n // 2], x[..., n // 2:n]
    return torch.cat([u * c - v * s, v * c + u * s, x[..., n:]], -1)


# ------------------------------------------------------------------------------------------------- attention
def chunk_visible(n, size):
    i = torch.arange(n)
    return (i[:, None] // size == i[None, :] // size) & (i[None, :] <= i[:, None])


def sink_softmax(scores, visible, sink):
    """scores [T, T]; the sink joins the denominator only."""
    s = scores.masked_fill(~visible, -math.inf)
    m = torch.maximum(s.max(-1).values, sink.expand(s.shape[0]))
    e = torch.exp(s - m[:, None])
    return e / (e.sum(-1, keepdim=True) + torch.exp(sink - m)[:, None])


def attention(h, w, pre, mc):
    T, H, G, D, DV = h.shape[0], mc["heads"], mc["kv_heads"], mc["dim"], mc["vdim"]
    pos = torch.arange(T)
    q = rotate((h @ w[pre + "q"].T).view(T, H, D), mc["rot"], pos)
    k = rotate((h @ w[pre + "k"].T).view(T, G, D), mc["rot"], pos)
    v = (h @ w[pre + "v"].T).view(T, G, DV)
    vis = chunk_visible(T, mc["mask"]["size"])
    outs = []
    for a in range(H):
        b = a // (H // G)
        p = sink_softmax((q[:, a] @ k[:, b].T) * mc["scale"], vis, w[pre + "sink"][a])
        outs.append(p @ v[:, b])
    return torch.cat(outs, -1) @ w[pre + "o"].T


# ------------------------------------------------------------------------------------------------- Mamba-2
def short_conv(x, taps_w, bias):
    T, W = x.shape[0], taps_w.shape[1]
    pad = torch.cat([torch.zeros(W - 1, x.shape[1], dtype=x.dtype), x])
    y = bias + sum(pad[i:i + T] * taps_w[:, i] for i in range(W))
    return silu(y)


def ssd(x, dt, a_log, b, c, d):
    """x [T, H, P], dt [T, H] (positive), b / c [T, G, N]."""
    T, H, P = x.shape
    G, N = b.shape[1:]
    S = torch.zeros(H, N, P, dtype=x.dtype)
    ys = []
    for t in range(T):
        y = []
        for h in range(H):
            g = h // (H // G)
            S[h] = torch.exp(-torch.exp(a_log[h]) * dt[t, h]) * S[h] + dt[t, h] * torch.outer(b[t, g], x[t, h])
            y.append(S[h].T @ c[t, g] + d[h] * x[t, h])
        ys.append(torch.cat(y))
    return torch.stack(ys)


def softplus(x):
    return torch.where(x > 0, x + torch.log1p(torch.exp(-x.abs())), torch.log1p(torch.exp(-x.abs())))


def mamba2(h, w, pre, mc, eps):
    T, H, P, N, G = h.shape[0], mc["heads"], mc["vdim"], mc["state"], mc["groups"]
    inner = H * P
    z, xbc, dt = (h @ w[pre + "in"].T).split([inner, inner + 2 * G * N, H], -1)
    xbc = short_conv(xbc, w[pre + "conv"], w[pre + "conv.b"])
    x, b, c = xbc.split([inner, G * N, G * N], -1)
    y = ssd(x.reshape(T, H, P), softplus(dt + w[pre + "dt_bias"]), w[pre + "A_log"], b.reshape(T, G, N),
            c.reshape(T, G, N), w[pre + "D"])
    y = rms((y * silu(z)).view(T, mc["norm_groups"], -1), eps).reshape(T, inner) * w[pre + "norm"]
    return y @ w[pre + "o"].T


def parallel_mixer(h, w, pre, mc, eps):
    left = attention(h, w, pre + "left.", mc["left"])
    right = mamba2(h, w, pre + "right.", mc["right"], eps)
    return 0.5 * (rms(left, eps) * w[pre + "left.out"] + rms(right, eps) * w[pre + "right.out"])


# ------------------------------------------------------------------------------------------------- WKV
def wkv_recurrence(r, k, v, decay, u):
    """r / k / decay [T, H, D], v [T, H, D], u [H, D]; the current token enters with the bonus, before the state update."""
    T, H, D = r.shape
    S = torch.zeros(H, D, v.shape[-1], dtype=r.dtype)
    out = torch.zeros(T, H, v.shape[-1], dtype=r.dtype)
    for t in range(T):
        for h in range(H):
            kv = torch.outer(k[t, h], v[t, h])
            out[t, h] = (S[h] + u[h][:, None] * kv).T @ r[t, h]
            S[h] = decay[t, h][:, None] * S[h] + kv
    return out


def wkv(h, w, pre, mc, eps):
    T, H, D = h.shape[0], mc["heads"], mc["dim"]
    prev = torch.cat([torch.zeros_like(h[:1]), h[:-1]])
    m = {s: h + (prev - h) * w[pre + "mu." + s] for s in "rkvgw"}
    r, k, v = ((m[s] @ w[pre + s].T).view(T, H, D) for s in "rkv")
    gate = silu(m["g"] @ w[pre + "g"].T)
    raw = torch.tanh(m["w"] @ w[pre + "w1"].T) @ w[pre + "w2"].T + w[pre + "w0"]
    o = wkv_recurrence(r, k, v, torch.exp(-torch.exp(raw)).view(T, H, D), w[pre + "u"])
    return (rms(o, eps).reshape(T, H * D) * w[pre + "norm"] * gate) @ w[pre + "o"].T


# ------------------------------------------------------------------------------------------------- feed-forward, layers
def clamped_glu(gate, up, limit):
    g = torch.clamp(gate, max=limit)
    u = torch.clamp(up, min=-limit, max=limit)
    return g * sigmoid(1.702 * g) * (u + 1.0)


def feed_forward(h, w, pre, limit):
    return clamped_glu(h @ w[pre + "gate"].T, h @ w[pre + "up"].T, limit) @ w[pre + "down"].T


def hyper_step(streams, w, pre, sub):
    """streams [S, T, W]: read one mix, run ``sub``, write all streams from the old ones."""
    read, write, mix = w[pre + "in"], w[pre + "out"], w[pre + "mix"]
    y = sub(torch.einsum("s,stw->tw", read, streams))
    return torch.einsum("sq,stw->qtw", mix, streams) + write[:, None, None] * y


def forward(cfg, weights, tokens, layers_out=None, dtype=torch.float64):
    """Logits [T, vocab] of every position; ``layers_out`` (a list) collects the summed streams after every layer."""
    w = {n: t.to(dtype) for n, t in weights.items()}
    eps = cfg["norm"]["eps"]
    x = w["embed"][torch.tensor(tokens)] * cfg["embedding"]["scale"]
    streams = x.expand(cfg["streams"], *x.shape).clone()
    for i, lc in enumerate(cfg["layers"]):
        pre, mc = f"l{i}.", lc["mixer"]
        mixer = {"wkv": wkv, "parallel": parallel_mixer}[lc["type"]]
        streams = hyper_step(streams, w, pre + "hc1.", lambda u: mixer(rms(u, eps) * w[pre + "norm1"], w, pre + "mix.", mc, eps))
        if lc["mlp"] is not None:
            streams = hyper_step(streams, w, pre + "hc2.", lambda u: feed_forward(rms(u, eps) * w[pre + "norm2"], w, pre + "mlp.",
                                                                                  lc["mlp"]["limit"]))
        if layers_out is not None:
            layers_out.append(streams.sum(0))
    return (rms(streams.sum(0), eps) * w["final.norm"]) @ w["embed"].T
