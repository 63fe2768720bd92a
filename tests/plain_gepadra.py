"""A plain, slow Gepadra: one function per mechanism, written from the design's equations.

Nothing here is shared with the package's compute path: it reads a configuration dict and a dict of
tensors, works on one whole sequence at a time in float64 (or the dtype asked for), builds the attention's
mask as a dense [T, T] table, walks the recurrence token by token and runs the chosen experts one by one.
The engine's results are compared with it.

Notation.  x[t] is the residual stream at token t.  A layer norms the stream twice and adds both sublayers to it at
once: x <- x + mixer(N1(x)) + ff(N2(x)), N(x) = x / sqrt(mean(x^2) + eps) * (1 + w).
"""
from __future__ import annotations

import math

import torch


def over_rms(x, eps):
    return x / torch.sqrt((x * x).mean(-1, keepdim=True) + eps)


def norm(x, eps, weight):
    return over_rms(x, eps) * (1 + weight)


def log_sigmoid(z):
    return torch.clamp(z, max=0) - torch.log1p(torch.exp(-z.abs()))


def gelu(z):
    return 0.5 * z * (1 + torch.erf(z / math.sqrt(2.0)))


# ---- attention
def rotate(u, rot):
    """u[T, heads, dim]: dimensions (i, i + dims/2) of the first rot.dims turn by position * base^(-2i/dims); the rest pass."""
    if not rot or not int(rot.get("dims", 0)):
        return u
    T, dims, base = u.shape[0], int(rot["dims"]), float(rot["base"])
    half = dims // 2
    f = torch.tensor([base ** (-2.0 * i / dims) for i in range(half)], dtype=u.dtype)
    a = torch.arange(T, dtype=u.dtype)[:, None] * f[None, :]
    c, s = torch.cos(a)[:, None, :], torch.sin(a)[:, None, :]
    lo, hi = u[..., :half], u[..., half:dims]
    return torch.cat([lo * c - hi * s, hi * c + lo * s, u[..., dims:]], -1)


def visible(T, mask):
    """[T, T]: does position i see j?"""
    i, j = torch.arange(T)[:, None], torch.arange(T)[None, :]
    see = j <= i
    if mask:
        see &= (i - j < int(mask["size"])) | (j < int(mask.get("keep_first", 0)))
    return see


def softmax_with_sink(s, sink):
    """Rows of scores (minus infinity: not seen); the denominator has one more term exp(sink)."""
    m = torch.clamp(s.max(-1, keepdim=True).values, min=float(sink))
    e = torch.exp(s - m)
    return e / (e.sum(-1, keepdim=True) + torch.exp(sink - m))


def attention(h, W, m, eps, first):
    """`first`: a dict that carries the values of the first layer that mixes its values (under "v")."""
    T = h.shape[0]
    H, G, D, Dv = int(m["heads"]), int(m["kv_heads"]), int(m["dim"]), int(m["vdim"])
    q = rotate((h @ W["q"].T + W["q.b"]).reshape(T, H, D), m.get("rot"))
    k = rotate((h @ W["k"].T + W["k.b"]).reshape(T, G, D), m.get("rot"))
    v = h @ W["v"].T + W["v.b"]                          # mixed as projected, all heads side by side
    if m.get("v_mix"):
        if "v" in first:
            v = (1 - W["vmix"]) * v + W["vmix"] * first["v"]
        else:
            first["v"] = v
    v = v.reshape(T, G, Dv)
    see = visible(T, m.get("mask"))
    out = torch.zeros(T, H, Dv, dtype=h.dtype)
    for hd in range(H):
        g = hd // (H // G)
        s = (q[:, hd] @ k[:, g].T) * float(m["scale"])
        out[:, hd] = softmax_with_sink(s.masked_fill(~see, float("-inf")), W["sink"][hd]) @ v[:, g]
    return out.reshape(T, H * Dv) @ W["o"].T


# ---- the matrix memory with exponential gates
def log_gates(h, W, cap):
    """-> (log input gate, log forget gate), [T, heads] each."""
    i = cap * torch.tanh((h @ W["i"].T + W["i.b"]) / cap)
    f = log_sigmoid(cap * torch.tanh((h @ W["f"].T + W["f.b"]) / cap))
    return i, f


def mlstm_walk(q, k, v, i, f):
    """q, k [T, H, D], v [T, H, Dv], log gates [T, H] -> the read-outs [T, H, Dv]."""
    T, H, D = q.shape
    S = torch.zeros(H, D, v.shape[-1], dtype=q.dtype)
    n = torch.zeros(H, D, dtype=q.dtype)
    m = torch.zeros(H, dtype=q.dtype)
    o = torch.zeros_like(v)
    for t in range(T):
        new = torch.maximum(f[t] + m, i[t])
        keep, put = torch.exp(f[t] + m - new), torch.exp(i[t] - new)
        S = keep[:, None, None] * S + put[:, None, None] * k[t][:, :, None] * v[t][:, None, :]
        n = keep[:, None] * n + put[:, None] * k[t]
        m = new
        den = torch.maximum((n * q[t]).sum(-1).abs(), torch.exp(-m)) + 1e-6
        o[t] = torch.einsum("hdv,hd->hv", S, q[t]) / den[:, None]
    return o


def mlstm(h, W, m, eps, first):
    T = h.shape[0]
    H, D, Dv = int(m["heads"]), int(m["dim"]), int(m["vdim"])
    q = (h @ W["q"].T).reshape(T, H, D) * D ** -0.5
    k = (h @ W["k"].T).reshape(T, H, D)
    v = (h @ W["v"].T).reshape(T, H, Dv)
    i, f = log_gates(h, W, float(m["gate_cap"]))
    o = over_rms(mlstm_walk(q, k, v, i, f), eps).reshape(T, H * Dv)
    return (o * W["norm"] * torch.sigmoid(h @ W["g"].T)) @ W["o"].T


MIXERS = {"attention": attention, "mlstm": mlstm}


# ---- feed-forwards
def clamped_gated(h, W, limit):
    g = torch.clamp(h @ W["gate"].T, max=limit)
    u = torch.clamp(h @ W["up"].T, -limit, limit)
    return (g * torch.sigmoid(1.702 * g) * (u + 1)) @ W["down"].T


def expert(h, W):
    return gelu(h @ W["up"].T) @ W["down"].T


def sub(tensors, prefix):
    n = len(prefix)
    return {k[n:]: v for k, v in tensors.items() if k.startswith(prefix)}


def routed(h, W, mlp, margins=None):
    """The `top` experts with the largest sigmoid scores, each fed the input times its score.  `margins`, a list, receives [T]:
    the gap between the last score chosen and the first one left out (infinite where all are chosen)."""
    E, top = int(mlp["router"]["experts"]), int(mlp["router"]["top"])
    s = torch.sigmoid(h @ W["router"].T)
    best = torch.sort(s, dim=-1, descending=True, stable=True)
    if margins is not None:
        margins.append(best.values[:, top - 1] - best.values[:, top] if top < E else torch.full_like(s[:, 0], float("inf")))
    out = torch.zeros_like(h)
    for t in range(h.shape[0]):
        for r in range(top):
            out[t] += expert(best.values[t, r] * h[t:t + 1], sub(W, f"e{int(best.indices[t, r])}."))[0]
    if mlp.get("shared"):
        out = out + torch.sigmoid(h @ W["shared.sg"].T) * expert(h, sub(W, "shared."))
    return out


# ---- the model
def forward(cfg, tensors, ids, dtype=torch.float64, return_layers=False, margins=None):
    """Logits [T, vocab] of one whole sequence; with `return_layers` also the stream after every layer; `margins`, a
    list, receives every router's margins (see `routed`)."""
    W = {k: v.to(dtype) if v.is_floating_point() else v for k, v in tensors.items()}
    ids = torch.as_tensor(ids, dtype=torch.long)
    eps = float(cfg["norm"]["eps"])
    x = W["embed"][ids]
    streams, first = [], {}
    for i, layer in enumerate(cfg["layers"]):
        p = f"l{i}."
        y = MIXERS[layer["type"]](norm(x, eps, W[p + "norm1"]), sub(W, p + "mix."), layer["mixer"], eps, first)
        mlp = layer.get("mlp")
        if mlp is not None:
            h, w = norm(x, eps, W[p + "norm2"]), sub(W, p + "mlp.")
            y = y + (clamped_gated(h, w, float(mlp["limit"])) if mlp["kind"] == "dense" else routed(h, w, mlp, margins))
        x = x + y
        streams.append(x)
    logits = norm(x, eps, W["final.norm"]) @ W["embed"].T
    return (logits, torch.stack(streams)) if return_layers else logits
