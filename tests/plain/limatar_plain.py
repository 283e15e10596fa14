"""Plain, slow implementation of the Limatar decoder, one function per
mechanism, for whole sequences on the CPU.  It shares no code with
``prism_b200``: weights come in as a dict of tensors keyed by the model file's
tensor names, the configuration as the raw ``config.json`` dict.  Everything
runs in the dtype of the weights handed in (float32 or float64).  ``rnd``,
where a function takes it, is applied to what a 16-bit engine may keep in 16
bits (the input of a matrix product, cached latents and rotated keys, queries,
the inner activations of a feed-forward); the default leaves everything as it is.

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


def centred_norm(x, w, eps):
    """RMS norm with a weight stored around zero."""
    return rms(x, eps) * (1.0 + w)


def silu(z):
    return z * torch.sigmoid(z)


def frequencies(rot):
    """The ``dims / 2`` rotation frequencies and the factor on cosine and sine."""
    n, base = rot["dims"], rot["base"]
    f = [base ** (-2.0 * i / n) for i in range(n // 2)]
    sc = rot.get("scaling")
    if not sc:
        return f, 1.0

    def turns(t):
        return n * math.log(sc["original"] / (2.0 * math.pi * t)) / (2.0 * math.log(base))
    lo = max(math.floor(turns(sc["fast"])), 0)
    hi = min(math.ceil(turns(sc["slow"])), n - 1)
    out = []
    for i, fi in enumerate(f):
        ramp = min(max((i - lo) / max(hi - lo, 0.001), 0.0), 1.0)
        out.append(fi / sc["factor"] * ramp + fi * (1.0 - ramp))
    return out, 0.1 * math.log(sc["factor"]) + 1.0


def rotate(x, rot, interleaved):
    """``x [T, ..., d]``: the first ``rot.dims`` entries turned by the row's position, the others as they are."""
    f, amp = frequencies(rot)
    half = len(f)
    y = x.clone()
    for p in range(x.shape[0]):
        for i in range(half):
            a, b = (2 * i, 2 * i + 1) if interleaved else (i, i + half)
            c, s = amp * math.cos(p * f[i]), amp * math.sin(p * f[i])
            u, v = x[p, ..., a], x[p, ..., b]
            y[p, ..., a] = u * c - v * s
            y[p, ..., b] = v * c + u * s
    return y


# ---- latent attention ---------------------------------------------------------------

def sink_softmax(scores, sink):
    """Rows of ``scores`` over their visible entries (the others are -inf), with ``exp(sink)`` in the denominator."""
    m = torch.maximum(scores.max(-1, keepdim=True).values, sink)
    e = torch.exp(scores - m)
    return e / (e.sum(-1, keepdim=True) + torch.exp(sink - m))


def latent_attention(h, w, p, mx, eps, rnd=_same):
    T = h.shape[0]
    H, d, r, dv, R = mx["heads"], mx["dim"], mx["rot_dim"], mx["vdim"], mx["kv_rank"]
    cq = rnd(rms(h @ w[p + "dq"].T, eps) * w[p + "dq.norm"])
    q = (cq @ w[p + "uq"].T).view(T, H, d + r)
    down = h @ w[p + "dkv"].T
    c = rnd(rms(down[:, :R], eps) * w[p + "dkv.norm"])
    kr = rnd(rotate(down[:, R:], mx["rot"], True))
    qn, qr = rnd(q[..., :d]), rnd(rotate(q[..., d:], mx["rot"], True))
    k = (c @ w[p + "uk"].T).view(T, H, d)
    v = (c @ w[p + "uv"].T).view(T, H, dv)
    hidden = torch.ones(T, T, dtype=torch.bool).triu(1)
    out = torch.zeros(T, H, dv, dtype=h.dtype)
    for hh in range(H):
        s = (qn[:, hh] @ k[:, hh].T + qr[:, hh] @ kr.T) * mx["scale"]
        out[:, hh] = sink_softmax(s.masked_fill(hidden, -math.inf), w[p + "sink"][hh]) @ v[:, hh]
    out = out.reshape(T, H * dv) * torch.sigmoid(h @ w[p + "g"].T)
    return rnd(out) @ w[p + "o"].T


# ---- retention -----------------------------------------------------------------------

def retain(q, k, v, decay):
    """``S <- decay S + k v^T; o = S^T q`` for one head, token after token."""
    S = torch.zeros(k.shape[1], v.shape[1], dtype=q.dtype)
    o = torch.zeros(q.shape[0], v.shape[1], dtype=q.dtype)
    for t in range(q.shape[0]):
        S = decay * S + k[t][:, None] * v[t][None, :]
        o[t] = S.T @ q[t]
    return o


def retention(h, w, p, mx, eps, rnd=_same):
    T = h.shape[0]
    H, d, dv = mx["heads"], mx["dim"], mx["vdim"]
    q = rotate((h @ w[p + "q"].T).view(T, H, d), mx["rot"], False)
    k = rotate((h @ w[p + "k"].T).view(T, H, d), mx["rot"], False) * d ** -0.5
    v = (h @ w[p + "v"].T).view(T, H, dv)
    o = torch.stack([rms(retain(q[:, i], k[:, i], v[:, i], mx["decay"][i]), eps) for i in range(H)], 1)
    return rnd(o.reshape(T, H * dv) * silu(h @ w[p + "g"].T)) @ w[p + "o"].T


# ---- feed-forward ---------------------------------------------------------------------

def dense_ff(h, w, p, limit, rnd=_same):
    g = torch.clamp(h @ w[p + "gate"].T, max=limit)
    u = torch.clamp(h @ w[p + "up"].T, -limit, limit)
    return rnd(g * torch.sigmoid(GATE_RATE * g) * (u + 1.0)) @ w[p + "down"].T


def expert(h, w, p, rnd=_same):
    return rnd(silu(h @ w[p + "gate"].T) * (h @ w[p + "up"].T)) @ w[p + "down"].T


def route(z, top):
    """For one token's router logits: the chosen experts and their weights."""
    chosen = sorted(range(z.shape[0]), key=lambda e: (-float(z[e]), e))[:top]
    return chosen, torch.softmax(z[chosen], -1)


def moe_ff(h, w, p, mlp, rnd=_same):
    z = h @ w[p + "router"].T + w[p + "router.b"]
    picks = [route(row, mlp["router"]["top"]) for row in z]
    out = torch.zeros_like(h)
    for e in range(mlp["router"]["experts"]):
        rows = [(t, float(wt[ch.index(e)])) for t, (ch, wt) in enumerate(picks) if e in ch]
        if rows:
            idx = torch.tensor([t for t, _ in rows])
            out[idx] += torch.tensor([x for _, x in rows], dtype=h.dtype)[:, None] * expert(h[idx], w, f"{p}e{e}.", rnd)
    if mlp.get("shared"):
        out = out + expert(h, w, p + "shared.", rnd)
    return out


# ---- the model ------------------------------------------------------------------------

def run_order(cfg):
    """Indices of the layers in the order they run."""
    n, loop = len(cfg["layers"]), cfg.get("loop")
    if not loop:
        return list(range(n))
    a, b = loop["start"], loop["stop"]
    return list(range(a)) + list(range(a, b)) * loop["times"] + list(range(b, n))


def layer(x, w, p, lr, eps, rnd=_same):
    h = rnd(centred_norm(x, w[p + "norm1"], eps))
    mix = {"latent_attention": latent_attention, "retention": retention}[lr["type"]]
    x = x + centred_norm(mix(h, w, p + "mix.", lr["mixer"], eps, rnd), w[p + "norm1b"], eps)
    mlp = lr.get("mlp")
    if mlp is not None:
        h = rnd(centred_norm(x, w[p + "norm2"], eps))
        y = dense_ff(h, w, p + "mlp.", mlp["limit"], rnd) if mlp["kind"] == "dense" else moe_ff(h, w, p + "mlp.", mlp, rnd)
        x = x + centred_norm(y, w[p + "norm2b"], eps)
    return x


def forward(cfg, w, tokens, rnd=_same, streams=None):
    """Logits ``[T, vocab]`` for one sequence.  ``streams``: a list that receives the residual rows after every layer run."""
    eps = cfg["norm"]["eps"]
    x = centred_norm(w["embed"][torch.as_tensor(tokens, dtype=torch.long)], w["embed.norm"], eps)
    for i in run_order(cfg):
        x = layer(x, w, f"l{i}.", cfg["layers"][i], eps, rnd)
        if streams is not None:
            streams.append(x.clone())
    return rnd(centred_norm(x, w["final.norm"], eps)) @ w["embed"].T
