"""Plain, slow implementation of the Nivotar decoder, one function per
mechanism, for whole sequences on the CPU.  It shares no code with
``prism_b200``: weights come in as a dict of tensors keyed by the model file's
tensor names, the configuration as the raw ``config.json`` dict.  Everything
runs in the dtype of the weights handed in (float32 or float64).  ``rnd``,
where a function takes it, is applied to what a 16-bit engine may keep in 16
bits (the input of a matrix product, queries, cached keys and values, the
inner activations of a feed-forward); the default leaves everything as it is.

Notation: ``x [T, D]`` is one sequence, positions are ``0 .. T-1``; ``W`` are
stored ``[out, in]`` and applied as ``x @ W.T``.
"""

from __future__ import annotations

import math

import torch

GATE_RATE = 1.702


def _same(x):
    return x


# ---- small pieces -----------------------------------------------------------------

def rms(x, eps):
    """``x / sqrt(mean(x^2) + eps)`` over the last axis."""
    return x / torch.sqrt((x * x).mean(-1, keepdim=True) + eps)


def silu(z):
    return z * torch.sigmoid(z)


def softplus(z):
    return torch.clamp(z, min=0) + torch.log1p(torch.exp(-z.abs()))


def rotate_halves(x, dims, base):
    """``x [T, ..., d]``: entry i of the first ``dims`` turns with entry ``i + dims / 2`` by the row's position."""
    half = dims // 2
    y = x.clone()
    for p in range(x.shape[0]):
        for i in range(half):
            a = p * base ** (-2.0 * i / dims)
            u, v = x[p, ..., i], x[p, ..., i + half]
            y[p, ..., i] = u * math.cos(a) - v * math.sin(a)
            y[p, ..., i + half] = v * math.cos(a) + u * math.sin(a)
    return y


# ---- attention under a sliding window ---------------------------------------------------

def visible(T, size):
    """``[T, T]`` bool: query i sees key j."""
    i, j = torch.arange(T)[:, None], torch.arange(T)[None, :]
    return (j <= i) & ((i - j) < size) if size else j <= i


def window_attention(h, w, p, mx, eps, rnd=_same):
    T = h.shape[0]
    H, G, d = mx["heads"], mx["kv_heads"], mx["dim"]
    dv = mx.get("vdim", d)
    q = rms(h @ w[p + "q"].T, eps) * w[p + "q.norm"]
    k = rms(h @ w[p + "k"].T, eps) * w[p + "k.norm"]
    rot = mx.get("rot") or dict(dims=0, base=1.0)
    q = rnd(rotate_halves(q.view(T, H, d), rot["dims"], rot["base"]))
    k = rnd(rotate_halves(k.view(T, G, d), rot["dims"], rot["base"]))
    v = rnd((h @ w[p + "v"].T).view(T, G, dv))
    see = visible(T, (mx.get("mask") or {}).get("size"))
    out = torch.zeros(T, H, dv, dtype=h.dtype)
    for i in range(H):
        g = i // (H // G)
        s = (q[:, i] @ k[:, g].T * mx["scale"]).masked_fill(~see, -math.inf)
        out[:, i] = torch.softmax(s, -1) @ v[:, g]
    return rnd(out.reshape(T, H * dv)) @ w[p + "o"].T


# ---- linear recurrences -------------------------------------------------------------------

def decayed_sum(q, k, v, decay):
    """``S <- decay_t S + k_t v_t^T; o_t = S^T q_t`` for one head; ``decay [T, n]``: per row of S, n the key size or 1."""
    S = torch.zeros(k.shape[1], v.shape[1], dtype=q.dtype)
    o = torch.zeros(q.shape[0], v.shape[1], dtype=q.dtype)
    for t in range(q.shape[0]):
        S = decay[t][:, None] * S + k[t][:, None] * v[t][None, :]
        o[t] = S.T @ q[t]
    return o


def short_conv(x, taps, bias):
    """``y_t = bias + sum_j taps[:, K-1-j] x_(t-j)``, zeros before the start."""
    T, K = x.shape[0], taps.shape[1]
    y = torch.zeros_like(x) + bias
    for t in range(T):
        for j in range(min(K, t + 1)):
            y[t] = y[t] + taps[:, K - 1 - j] * x[t - j]
    return y


def state_space(h, w, p, mx, eps, rnd=_same):
    T = h.shape[0]
    H, dv, N, G, parts = mx["heads"], mx["vdim"], mx["state"], mx["groups"], mx["norm_groups"]
    inner = H * dv
    z, u, dt = (h @ w[p + "in"].T).split([inner, inner + 2 * G * N, H], -1)
    u = silu(short_conv(u, w[p + "conv"], w[p + "conv.b"]))
    x, B, C = u.split([inner, G * N, G * N], -1)
    x, B, C = x.reshape(T, H, dv), B.reshape(T, G, N), C.reshape(T, G, N)
    dt = softplus(dt + w[p + "dt_bias"])
    y = torch.zeros(T, H, dv, dtype=h.dtype)
    for i in range(H):
        g = i // (H // G)
        decay = torch.exp(-torch.exp(w[p + "A_log"][i]) * dt[:, i])[:, None]
        y[:, i] = decayed_sum(C[:, g], B[:, g], dt[:, i:i + 1] * x[:, i], decay) + w[p + "D"][i] * x[:, i]
    y = y.reshape(T, inner) * silu(z)
    y = rms(y.view(T, parts, inner // parts), eps).reshape(T, inner) * w[p + "norm"]
    return rnd(y) @ w[p + "o"].T


def parallel(h, w, p, mx, eps, rnd=_same):
    return (mx["left_scale"] * window_attention(h, w, p + "left.", mx["left"], eps, rnd)
            + mx["right_scale"] * state_space(h, w, p + "right.", mx["right"], eps, rnd))


def lightning(h, w, p, mx, eps, rnd=_same):
    T = h.shape[0]
    H, d, dv = mx["heads"], mx["dim"], mx.get("vdim", mx["dim"])
    q, k = silu(h @ w[p + "q"].T).view(T, H, d), silu(h @ w[p + "k"].T).view(T, H, d)
    v = silu(h @ w[p + "v"].T).view(T, H, dv)
    o = torch.stack([decayed_sum(q[:, i], k[:, i], v[:, i], torch.full((T, 1), mx["decay"][i], dtype=h.dtype))
                     for i in range(H)], 1)
    o = rms(o.reshape(T, H * dv), eps) * w[p + "norm"]
    return rnd(o * torch.sigmoid(h @ w[p + "g"].T)) @ w[p + "o"].T


def gated_linear(h, w, p, mx, eps, rnd=_same):
    T = h.shape[0]
    H, d, dv = mx["heads"], mx["dim"], mx.get("vdim", mx["dim"])
    q = (h @ w[p + "q"].T).view(T, H, d) * d ** -0.5
    k, v = (h @ w[p + "k"].T).view(T, H, d), (h @ w[p + "v"].T).view(T, H, dv)
    z = (h @ w[p + "a1"].T) @ w[p + "a2"].T + w[p + "a2.b"]
    alpha = torch.exp(-softplus(-z) / mx["tau"]).view(T, H, d)
    o = torch.stack([decayed_sum(q[:, i], k[:, i], v[:, i], alpha[:, i]) for i in range(H)], 1)
    o = (rms(o, eps) * w[p + "norm"]).reshape(T, H * dv)
    return rnd(o * silu(h @ w[p + "g"].T)) @ w[p + "o"].T


# ---- feed-forward ---------------------------------------------------------------------

def dense_ff(h, w, p, rnd=_same):
    a = silu(h @ w[p + "gate"].T + w[p + "gate.b"]) * (h @ w[p + "up"].T + w[p + "up.b"])
    return rnd(a) @ w[p + "down"].T + w[p + "down.b"]


def clamped_expert(h, w, p, limit, rnd=_same):
    g = torch.clamp(h @ w[p + "gate"].T, max=limit)
    u = torch.clamp(h @ w[p + "up"].T, -limit, limit)
    return rnd(g * torch.sigmoid(GATE_RATE * g) * (u + 1.0)) @ w[p + "down"].T


def route(z, correction, top):
    """For one token's router logits: the chosen experts and their weights."""
    s = torch.softmax(z, -1)
    c = s + correction
    chosen = sorted(range(z.shape[0]), key=lambda e: (-float(c[e]), e))[:top]
    return chosen, s[chosen]


def moe_ff(h, w, p, mlp, rnd=_same, own=None):
    """``own``: the layer's input as the identity experts return it (default: ``h``)."""
    own = h if own is None else own
    E, idle = mlp["router"]["experts"], mlp["router"].get("identity", 0)
    z = h @ w[p + "router"].T
    picks = [route(row, w[p + "correction"], mlp["router"]["top"]) for row in z]
    out = torch.zeros_like(h)
    for e in range(E + idle):
        rows = [(t, float(wt[ch.index(e)])) for t, (ch, wt) in enumerate(picks) if e in ch]
        if rows:
            idx = torch.tensor([t for t, _ in rows])
            y = clamped_expert(h[idx], w, f"{p}e{e}.", mlp["expert"]["limit"], rnd) if e < E else own[idx]
            out[idx] += torch.tensor([x for _, x in rows], dtype=h.dtype)[:, None] * y
    return out


# ---- the model ------------------------------------------------------------------------

MIXERS = {"parallel": parallel, "lightning": lightning, "gla": gated_linear}


def layer(x, w, p, lr, eps, rnd=_same):
    x = x + rms(MIXERS[lr["type"]](rnd(x), w, p + "mix.", lr["mixer"], eps, rnd), eps) * w[p + "norm1"]
    mlp = lr.get("mlp")
    if mlp is not None:
        y = dense_ff(rnd(x), w, p + "mlp.", rnd) if mlp["kind"] == "dense" else moe_ff(rnd(x), w, p + "mlp.", mlp, rnd, x)
        x = x + rms(y, eps) * w[p + "norm2"]
    return x


def forward(cfg, w, tokens, rnd=_same, streams=None):
    """Logits ``[T, vocab]`` for one sequence.  ``streams``: a list that receives the residual rows after every layer."""
    eps = cfg["norm"]["eps"]
    x = w["embed"][torch.as_tensor(tokens, dtype=torch.long)]
    for i, lr in enumerate(cfg["layers"]):
        x = layer(x, w, f"l{i}.", lr, eps, rnd)
        if streams is not None:
            streams.append(x.clone())
    return rnd(rms(x, eps) * w["final.norm"]) @ w["embed"].T
