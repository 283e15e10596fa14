"""Shared pieces of the Limatar tests: small configurations that differ from one another in every size and option,
model folders with weights drawn here (larger than the framework's random-weights recipe, so that attention is far
from uniform, the sink matters, gates and limits cut in, the router's scores are spread, and a wrong key, a lost
state or a missing sink shows), and the comparison with the plain implementation."""

from __future__ import annotations

import json
import math
import os
import sys
import tempfile

import torch

HERE = os.path.dirname(os.path.abspath(__file__))
if HERE not in sys.path:
    sys.path.insert(0, HERE)

from plain import limatar_plain as LP  # noqa: E402
from zuvulorn_helpers import errors, judge, row_error, to_bf16_and_back  # noqa: E402,F401  (generic: rows against a reference)


def yarn(factor=4.0, original=40, fast=8.0, slow=1.0):
    return dict(factor=factor, original=original, fast=fast, slow=slow)


def latent(heads, dim, rot_dim, vdim, q_rank, kv_rank, scale=0.3, base=500.0, scaling=None):
    rot = dict(base=base, dims=rot_dim)
    if scaling:
        rot["scaling"] = scaling
    return dict(heads=heads, dim=dim, rot_dim=rot_dim, vdim=vdim, q_rank=q_rank, kv_rank=kv_rank, scale=scale, rot=rot)


def retain(heads, dim, vdim, decay, rot_dims=None, base=200.0):
    return dict(heads=heads, dim=dim, vdim=vdim, decay=list(decay), rot=dict(base=base, dims=dim if rot_dims is None else rot_dims))


def dense(ff, limit):
    return dict(kind="dense", ff=ff, limit=limit)


def moe(ff, experts, top, shared=None):
    m = dict(kind="moe", expert=dict(ff=ff), router=dict(experts=experts, top=top))
    if shared is not None:
        m["shared"] = dict(ff=shared)
    return m


def layer(kind, mixer, mlp):
    return dict(type={"latent": "latent_attention"}.get(kind, kind), mixer=mixer, mlp=mlp)


def model(vocab, width, layers, loop=None, eps=1e-5):
    raw = dict(architecture="Limatar", vocab=vocab, width=width, norm=dict(eps=eps), layers=layers)
    if loop is not None:
        raw["loop"] = dict(start=loop[0], stop=loop[1], times=loop[2])
    return raw


# A: sizes that are multiples of nothing, so every kernel is the shape-generic one; a layer without feed-forward inside the
# loop; a rotated part larger than the plain one; a retention that turns part of its heads
CONFIG_A = model(211, 74, loop=(1, 3, 2), layers=[
    layer("latent", latent(5, 7, 10, 9, 11, 13, scale=0.4, scaling=yarn()), moe(13, 5, 3, shared=9)),
    layer("retention", retain(3, 10, 7, (0.9, 0.5, 0.99), rot_dims=6), None),
    layer("latent", latent(2, 12, 4, 5, 6, 20, scale=0.25), dense(37, 0.8)),
    layer("retention", retain(2, 6, 11, (0.97, 0.8)), dense(50, 3.0)),
])
# B: sizes the tensor-core kernels take, pages of 64; the loop runs both kinds three times; values of another size than keys,
# key and value channels of a state of different sizes
CONFIG_B = model(300, 128, loop=(0, 2, 3), layers=[
    layer("latent", latent(4, 32, 16, 24, 40, 48, scale=0.2, scaling=yarn(2.0, 64, 16.0, 2.0)), dense(256, 0.7)),
    layer("retention", retain(2, 64, 32, (0.98, 0.9), rot_dims=32), moe(64, 8, 2, shared=96)),
    layer("latent", latent(6, 16, 32, 40, 64, 96, scale=0.15, base=10000.0, scaling=yarn(8.0, 128, 32.0, 1.0)), moe(32, 4, 2)),
])
# C: everything 1 that can be: one head, one expert and one chosen, a loop of one pass, the smallest rotation, a limit of one
CONFIG_C = model(64, 32, loop=(0, 3, 1), layers=[
    layer("latent", latent(1, 1, 2, 1, 3, 3, scale=1.0), moe(16, 1, 1)),
    layer("retention", retain(1, 2, 3, (1.0,)), dense(16, 1.0)),
    layer("latent", latent(2, 4, 2, 3, 5, 4, scaling=yarn(1.0, 16, 4.0, 4.0)), None),
])
# D: recurrent layers only (no paged cache group at all), the whole model twice; decays of zero and of one, no rotation
CONFIG_D = model(90, 48, loop=(0, 3, 2), layers=[
    layer("retention", retain(6, 8, 8, (0.0, 1.0, 0.5, 0.9, 0.99, 0.999)), moe(32, 4, 1, shared=32)),
    layer("retention", retain(3, 16, 24, (0.7, 0.96, 0.9961), rot_dims=0), None),
    layer("retention", retain(1, 40, 16, (0.95,), rot_dims=16, base=1e6), dense(24, 0.5)),
])
# E: a few hundred wide; more than sixteen heads on one latent, a latent of 160 entries; states of 128 x 64 and 256 x 96; a
# shared expert as wide as the others; inner widths that are no multiple of a k-block; no loop
CONFIG_E = model(500, 384, layers=[
    layer("latent", latent(20, 64, 32, 48, 96, 160, scale=0.1, scaling=yarn(16.0, 256, 32.0, 1.0)), moe(72, 12, 4, shared=72)),
    layer("retention", retain(3, 128, 64, (0.97, 0.99, 0.998)), dense(200, 2.0)),
    layer("retention", retain(2, 256, 96, (0.9, 0.995), rot_dims=128), moe(40, 3, 3, shared=24)),
    layer("latent", latent(3, 96, 64, 128, 56, 192, scale=0.08, base=10000.0), dense(136, 0.9)),
])
CONFIGS = {"A": (CONFIG_A, 11, 8), "B": (CONFIG_B, 12, 64), "C": (CONFIG_C, 13, 16), "D": (CONFIG_D, 14, 16), "E": (CONFIG_E, 15, 64)}
LENGTHS = {"A": (61, 9, 2, 34, 1, 27), "B": (150, 31, 77, 64, 3), "C": (40, 1, 17, 5), "D": (75, 3, 22, 1, 30), "E": (130, 40, 66, 7)}


def every_expert(raw: dict) -> dict:
    """The same model with every expert chosen for every token.  In bfloat16 two experts' logits lie within rounding of
    each other for a token now and then, the choice falls the other way, and through the states every later row of the
    request moves: no rounding bound holds then.  The bfloat16 runs of whole models use these variants; the choice itself
    is covered in float32 and, in bfloat16, on given logits."""
    out = json.loads(json.dumps(raw))
    for l in out["layers"]:
        if l.get("mlp") is not None and l["mlp"]["kind"] == "moe":
            l["mlp"]["router"]["top"] = l["mlp"]["router"]["experts"]
    return out


for _name in list(CONFIGS):
    CONFIGS[_name + "x"] = (every_expert(CONFIGS[_name][0]),) + CONFIGS[_name][1:]


def draw_weights(raw: dict, seed: int) -> dict:
    """bf16 tensors keyed by the model file's names."""
    g = torch.Generator().manual_seed(seed)
    W = raw["width"]

    def mat(o, i, gain=1.0):
        return torch.randn(o, i, generator=g) * (gain / math.sqrt(i))

    def vec(n, std, mean=0.0):
        return torch.randn(n, generator=g) * std + mean

    def gated(p, F):
        t[p + "gate"], t[p + "up"], t[p + "down"] = mat(F, W, 1.5), mat(F, W, 1.2), mat(W, F, 0.8)

    t = {"embed": torch.randn(raw["vocab"], W, generator=g) * 0.7, "embed.norm": vec(W, 0.2), "final.norm": vec(W, 0.2)}
    for i, lr in enumerate(raw["layers"]):
        p, m, q = f"l{i}.", lr["mixer"], f"l{i}.mix."
        t[p + "norm1"], t[p + "norm1b"] = vec(W, 0.2), vec(W, 0.2, -0.3)
        H = m["heads"]
        if lr["type"] == "latent_attention":
            t[q + "dq"], t[q + "dq.norm"] = mat(m["q_rank"], W), vec(m["q_rank"], 0.1, 1.0)
            t[q + "uq"] = mat(H * (m["dim"] + m["rot_dim"]), m["q_rank"], 2.0)
            t[q + "dkv"], t[q + "dkv.norm"] = mat(m["kv_rank"] + m["rot_dim"], W, 1.5), vec(m["kv_rank"], 0.1, 1.0)
            t[q + "uk"], t[q + "uv"] = mat(H * m["dim"], m["kv_rank"], 2.0), mat(H * m["vdim"], m["kv_rank"], 1.5)
            t[q + "sink"], t[q + "g"], t[q + "o"] = vec(H, 1.0), mat(H * m["vdim"], W, 1.5), mat(W, H * m["vdim"])
        else:
            t[q + "q"], t[q + "k"] = mat(H * m["dim"], W, 1.5), mat(H * m["dim"], W, 1.5)
            t[q + "v"], t[q + "g"], t[q + "o"] = mat(H * m["vdim"], W, 1.5), mat(H * m["vdim"], W, 1.5), mat(W, H * m["vdim"])
        mlp = lr.get("mlp")
        if mlp is None:
            continue
        t[p + "norm2"], t[p + "norm2b"] = vec(W, 0.2), vec(W, 0.2, -0.3)
        if mlp["kind"] == "dense":
            gated(p + "mlp.", mlp["ff"])
        else:
            E = mlp["router"]["experts"]
            t[p + "mlp.router"], t[p + "mlp.router.b"] = mat(E, W, 2.0), vec(E, 1.0)
            for e in range(E):
                gated(f"{p}mlp.e{e}.", mlp["expert"]["ff"])
            if mlp.get("shared"):
                gated(p + "mlp.shared.", mlp["shared"]["ff"])
    return {k: v.to(torch.bfloat16).contiguous() for k, v in t.items()}


_folders = {}


def write_folder(raw: dict, weights: dict, d: str = None) -> str:
    from safetensors.torch import save_file
    d = d or tempfile.mkdtemp(prefix="prism_limatar_")
    with open(os.path.join(d, "config.json"), "w") as f:
        json.dump(raw, f)
    save_file(weights, os.path.join(d, "model.safetensors"))
    return d


def model_folder(name: str) -> str:
    if name not in _folders:
        raw, seed, _ = CONFIGS[name]
        _folders[name] = write_folder(raw, draw_weights(raw, seed))
    return _folders[name]


_plain, _logits, _rounding = {}, {}, {}


def plain_weights(name: str, dtype=torch.float64):
    if (name, dtype) not in _plain:
        raw, seed, _ = CONFIGS[name]
        _plain[(name, dtype)] = {k: v.to(dtype) for k, v in draw_weights(raw, seed).items()}
    return _plain[(name, dtype)]


def plain_logits(name: str, seq) -> torch.Tensor:
    """The plain model in float64 on the whole sequence."""
    key = (name, tuple(seq))
    if key not in _logits:
        _logits[key] = LP.forward(CONFIGS[name][0], plain_weights(name), list(seq))
    return _logits[key]


def plain_rounding(name: str, seq, dtype: str = "float32") -> list:
    """Per position: how far rounding alone moves the plain model from itself in float64.  For float32 it is the
    plain model run in float32; for bfloat16 the plain model in float64 with what a 16-bit engine may keep in 16 bits
    rounded to bfloat16."""
    key = (name, tuple(seq), dtype)
    if key not in _rounding:
        ref = plain_logits(name, seq)
        if dtype == "float32":
            low = LP.forward(CONFIGS[name][0], plain_weights(name, torch.float32), list(seq))
        else:
            low = LP.forward(CONFIGS[name][0], plain_weights(name), list(seq), rnd=to_bf16_and_back)
        scale = float((ref - ref.mean(-1, keepdim=True)).pow(2).mean().sqrt())
        _rounding[key] = [row_error(low[p], ref[p], scale) for p in range(len(seq))]
    return _rounding[key]


def compare(name: str, seqs: dict, got: dict, limit: float, ill: float = 0.0, dtype: str = "float32"):
    """Every row the trace produced against the plain model on the whole sequence."""
    errs = []
    for rid, seq in seqs.items():
        errs += errors(plain_logits(name, seq), got, rid, plain_rounding(name, seq, dtype))
    return judge(errs, limit, ill)
