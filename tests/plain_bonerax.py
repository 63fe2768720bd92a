"""A plain, slow Bonerax: one function per mechanism, written from the design's equations.

Nothing here is shared with the package's compute path: it reads a configuration dict and a dict of
tensors, works on one whole sequence at a time in float64 (or the dtype asked for), builds the attention's
mask as a dense [T, T] table and walks every recurrence token by token.  The engine's results are compared
with it.

Notation.  x[t] is the residual stream at token t.  A layer reads the stream as it is and norms what comes out of
its sublayers: x <- x + L1(mixer(x)), then (where it has a feed-forward) x <- x + L2(ff(x)), every L a layer norm
with a weight and no bias.  A mixer is a gated linear attention, a delta rule with one decay per key channel, or
the sum of two scaled mixers, windowed softmax attention and such a delta rule, on the same input.
"""
from __future__ import annotations

import math

import torch


def layer_norm(x, eps, weight):
    d = x - x.mean(-1, keepdim=True)
    return d / torch.sqrt((d * d).mean(-1, keepdim=True) + eps) * weight


def rms_norm(x, eps, weight=None):
    y = x / torch.sqrt((x * x).mean(-1, keepdim=True) + eps)
    return y if weight is None else y * weight


def silu(z):
    return z * torch.sigmoid(z)


def softplus(z):
    return torch.clamp(z, min=0) + torch.log1p(torch.exp(-z.abs()))


# ---- positions
def yarn(rot):
    """-> (frequencies, multiplier of cosines and sines).  Without a `scaling` block f_i = base^(-2i/dims) and 1.  With
    one, pair i keeps f_i where i is at most lo, gets f_i / factor where i is at least hi, and a linear mix of the two
    in between; lo and hi are the (fractional, then rounded outwards) pair numbers whose waves turn `fast` and `slow`
    times within `original` positions."""
    dims, base = int(rot["dims"]), float(rot["base"])
    f = [base ** (-2.0 * i / dims) for i in range(dims // 2)]
    sc = rot.get("scaling")
    if not sc:
        return f, 1.0
    factor, original = float(sc["factor"]), float(sc["original"])

    def pair_that_turns(times):
        return dims * math.log(original / (2 * math.pi * times)) / (2 * math.log(base))

    lo = max(math.floor(pair_that_turns(float(sc["fast"]))), 0)
    hi = min(math.ceil(pair_that_turns(float(sc["slow"]))), dims - 1)
    out = []
    for i, fi in enumerate(f):
        r = min(max((i - lo) / max(hi - lo, 0.001), 0.0), 1.0)
        out.append(fi / factor * r + fi * (1.0 - r))
    return out, 0.1 * math.log(factor) + 1.0


def rotate(u, rot):
    """u[T, heads, dim]: pairs (2i, 2i+1) of the first rot.dims dimensions turn by position * f_i; the rest pass."""
    if not rot or not int(rot.get("dims", 0)):
        return u
    T, dims = u.shape[0], int(rot["dims"])
    f, mult = yarn(rot)
    a = torch.arange(T, dtype=u.dtype)[:, None] * torch.tensor(f, dtype=u.dtype)[None, :]
    c, s = (torch.cos(a) * mult)[:, None, :], (torch.sin(a) * mult)[:, None, :]
    even, odd = u[..., 0:dims:2], u[..., 1:dims:2]
    out = u.clone()
    out[..., 0:dims:2] = even * c - odd * s
    out[..., 1:dims:2] = odd * c + even * s
    return out


# ---- mixers
def windowed_attention(h, W, m, eps):
    T = h.shape[0]
    H, G, D, Dv = int(m["heads"]), int(m["kv_heads"]), int(m["dim"]), int(m["vdim"])
    q = (h @ W["q"].T + W["q.b"]).reshape(T, H, D)
    k = (h @ W["k"].T + W["k.b"]).reshape(T, G, D)
    v = (h @ W["v"].T + W["v.b"]).reshape(T, G, Dv)
    q, k = rms_norm(q, eps, W["q.norm"]), rms_norm(k, eps, W["k.norm"])
    q, k = rotate(q, m.get("rot")), rotate(k, m.get("rot"))
    i, j = torch.arange(T)[:, None], torch.arange(T)[None, :]
    visible = i >= j
    if m.get("mask"):
        visible &= i - j < int(m["mask"]["size"])
    out = torch.zeros(T, H, Dv, dtype=h.dtype)
    for hd in range(H):
        g = hd // (H // G)
        s = (q[:, hd] @ k[:, g].T) * float(m["scale"])
        out[:, hd] = torch.softmax(s.masked_fill(~visible, float("-inf")), dim=-1) @ v[:, g]
    return out.reshape(T, H * Dv) @ W["o"].T + W["o.b"]


def short_convolution(u, taps):
    """y[t, c] = sum_j taps[c, j] u[t - (n - 1) + j, c], inputs before the start zero, then silu."""
    n = taps.shape[1]
    padded = torch.cat([torch.zeros(n - 1, u.shape[1], dtype=u.dtype), u], 0)
    return silu(sum(taps[:, j] * padded[j:j + u.shape[0]] for j in range(n)))


def unit(x):
    return x / torch.sqrt((x * x).sum(-1, keepdim=True) + 1e-6)


def channel_delta(h, W, m, eps):
    T = h.shape[0]
    H, G, D, Dv = int(m["heads"]), int(m["kv_heads"]), int(m["dim"]), int(m["vdim"])
    q = unit(short_convolution(h @ W["q"].T, W["q.conv"]).reshape(T, G, D)) * D ** -0.5
    k = unit(short_convolution(h @ W["k"].T, W["k.conv"]).reshape(T, G, D))
    v = short_convolution(h @ W["v"].T, W["v.conv"]).reshape(T, H, Dv)
    q, k = q.repeat_interleave(H // G, 1), k.repeat_interleave(H // G, 1)
    beta = torch.sigmoid(h @ W["b"].T)
    z = ((h @ W["a1"].T) @ W["a2"].T + W["dt_bias"]).reshape(T, H, D)
    g = torch.exp(-torch.exp(W["A_log"])[None, :, None] * softplus(z))
    S = torch.zeros(H, D, Dv, dtype=h.dtype)
    o = torch.zeros(T, H, Dv, dtype=h.dtype)
    for t in range(T):
        S = g[t][:, :, None] * S
        u = beta[t][:, None] * (v[t] - torch.einsum("hdv,hd->hv", S, k[t]))
        S = S + k[t][:, :, None] * u[:, None, :]
        o[t] = torch.einsum("hdv,hd->hv", S, q[t])
    gate = torch.sigmoid((h @ W["g1"].T) @ W["g2"].T).reshape(T, H, Dv)
    return (rms_norm(o, eps, W["norm"]) * gate).reshape(T, H * Dv) @ W["o"].T


def gated_linear_attention(h, W, m, eps):
    T = h.shape[0]
    H, D, Dv = int(m["heads"]), int(m["dim"]), int(m["vdim"])
    q = (h @ W["q"].T).reshape(T, H, D) * D ** -0.5
    k = (h @ W["k"].T).reshape(T, H, D)
    v = (h @ W["v"].T).reshape(T, H, Dv)
    z = (h @ W["a1"].T) @ W["a2"].T + W["a2.b"]
    alpha = (torch.sigmoid(z) ** (1.0 / float(m["tau"]))).reshape(T, H, D)
    S = torch.zeros(H, D, Dv, dtype=h.dtype)
    o = torch.zeros(T, H, Dv, dtype=h.dtype)
    for t in range(T):
        S = alpha[t][:, :, None] * S + k[t][:, :, None] * v[t][:, None, :]
        o[t] = torch.einsum("hdv,hd->hv", S, q[t])
    o = rms_norm(o, eps, W["norm"]).reshape(T, H * Dv)
    return (o * silu(h @ W["g"].T)) @ W["o"].T


def sub(tensors, prefix):
    n = len(prefix)
    return {k[n:]: v for k, v in tensors.items() if k.startswith(prefix)}


def parallel_mixer(h, W, m, eps):
    left = windowed_attention(h, sub(W, "left."), m["left"], eps)
    right = channel_delta(h, sub(W, "right."), m["right"], eps)
    return float(m["left_scale"]) * left + float(m["right_scale"]) * right


MIXERS = {"parallel": parallel_mixer, "channel_delta": channel_delta, "gla": gated_linear_attention}


# ---- feed-forwards
def gated(h, W):
    return (silu(h @ W["gate"].T) * (h @ W["up"].T)) @ W["down"].T


def routed_feed_forward(h, W, mlp, margins=None):
    """The `top` experts with the largest logits, weighed by the softmax over those logits alone.  `margins`, a list,
    receives [T]: the gap between the last logit chosen and the first one left out (infinite where all are chosen)."""
    E, top = int(mlp["router"]["experts"]), int(mlp["router"]["top"])
    z = h @ W["router"].T + W["router.b"]
    best = torch.sort(z, dim=-1, descending=True, stable=True)
    if margins is not None:
        margins.append(best.values[:, top - 1] - best.values[:, top] if top < E else torch.full_like(z[:, 0], float("inf")))
    w = torch.softmax(best.values[:, :top], dim=-1)
    out = torch.zeros_like(h)
    for t in range(h.shape[0]):
        for i in range(top):
            out[t] += w[t, i] * gated(h[t:t + 1], sub(W, f"e{int(best.indices[t, i])}."))[0]
    return out


# ---- the model
def own_layer(layers, i):
    """The layer whose tensors layer i uses: itself, or the one that `weights_of` names."""
    while layers[i].get("weights_of") is not None:
        i = int(layers[i]["weights_of"])
    return i


def output(x, W, cfg, eps):
    logits = layer_norm(x, eps, W["final.norm"]) @ W["head"].T * float(cfg.get("logit_scale", 1.0))
    cap = cfg.get("logit_softcap")
    return float(cap) * torch.tanh(logits / float(cap)) if cap else logits


def forward(cfg, tensors, ids, dtype=torch.float64, return_layers=False, margins=None):
    """Logits [T, vocab] of one whole sequence; with `return_layers` also the stream after every layer; `margins`, a
    list, receives every router's margins (see `routed_feed_forward`)."""
    W = {k: v.to(dtype) if v.is_floating_point() else v for k, v in tensors.items()}
    ids = torch.as_tensor(ids, dtype=torch.long)
    eps = float(cfg["norm"]["eps"])
    x = W["embed"][ids]
    streams = []
    for i, layer in enumerate(cfg["layers"]):
        p = f"l{own_layer(cfg['layers'], i)}."
        x = x + layer_norm(MIXERS[layer["type"]](x, sub(W, p + "mix."), layer["mixer"], eps), eps, W[p + "norm1"])
        mlp = layer.get("mlp")
        if mlp is not None:
            w = sub(W, p + "mlp.")
            y = gated(x, w) if mlp["kind"] == "dense" else routed_feed_forward(x, w, mlp, margins)
            x = x + layer_norm(y, eps, W[p + "norm2"])
        streams.append(x)
    logits = output(x, W, cfg, eps)
    return (logits, torch.stack(streams)) if return_layers else logits
