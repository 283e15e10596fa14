"""Shared pieces of the Nivotar tests: small configurations that differ from one another in every size and option,
model folders with weights drawn here (larger than the framework's random-weights recipe, so that attention is far
from uniform, decays range from fast to slow, gates and limits cut in, the router's scores are spread, and a wrong key
or a lost state shows), and the comparison with the plain implementation."""

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

from plain import nivotar_plain as NP  # noqa: E402
from zuvulorn_helpers import errors, judge, row_error, to_bf16_and_back  # noqa: E402,F401  (generic: rows against a reference)


def left(heads, kv_heads, dim, vdim, size, scale=0.3, rot_dims=None, base=500.0):
    m = dict(heads=heads, kv_heads=kv_heads, dim=dim, vdim=vdim, scale=scale, rot=dict(base=base, dims=dim if rot_dims is None else rot_dims))
    if size:
        m["mask"] = dict(size=size)
    return m


def right(heads, vdim, state, groups, conv, norm_groups):
    return dict(heads=heads, vdim=vdim, state=state, groups=groups, conv=conv, norm_groups=norm_groups)


def parallel(lft, rgt, left_scale=0.7, right_scale=0.6):
    return dict(left=lft, right=rgt, left_scale=left_scale, right_scale=right_scale)


def lightning(heads, dim, vdim, decay):
    return dict(heads=heads, dim=dim, vdim=vdim, decay=list(decay))


def gla(heads, dim, vdim, tau, rank):
    return dict(heads=heads, dim=dim, vdim=vdim, tau=tau, decay_rank=rank)


def dense(ff):
    return dict(kind="dense", ff=ff)


def moe(ff, experts, top, identity=0, limit=1.2):
    r = dict(experts=experts, top=top)
    if identity:
        r["identity"] = identity
    return dict(kind="moe", expert=dict(ff=ff, limit=limit), router=r)


def layer(kind, mixer, mlp):
    return dict(type=kind, mixer=mixer, mlp=mlp)


def model(vocab, width, layers, eps=1e-5):
    return dict(architecture="Nivotar", vocab=vocab, width=width, norm=dict(eps=eps), layers=layers)


# A: sizes that are multiples of nothing, so every kernel is the shape-generic one; a window shorter than a page; a head that
# turns in part; a convolution of two taps; a layer without feed-forward; identity experts beside few real ones
CONFIG_A = model(211, 74, [
    layer("parallel", parallel(left(5, 1, 10, 9, 6, scale=0.4, rot_dims=6), right(6, 5, 7, 3, 2, 2)), moe(13, 5, 3, 2, limit=0.9)),
    layer("gla", gla(3, 10, 7, 5.0, 3), None),
    layer("lightning", lightning(2, 6, 11, (0.9, 0.5)), dense(37)),
    layer("parallel", parallel(left(4, 2, 7, 12, 33, scale=0.35, rot_dims=2, base=50.0), right(3, 9, 5, 1, 5, 3), 1.3, -0.4), moe(9, 3, 2, 1)),
    layer("gla", gla(5, 6, 13, 16.0, 5), moe(17, 4, 1, limit=3.0)),
])
# B: sizes the tensor-core kernels take, pages of 64; one window with a page's length and one across several; states with
# more keys than values and the reverse
CONFIG_B = model(300, 128, [
    layer("gla", gla(2, 64, 32, 8.0, 16), dense(256)),
    layer("parallel", parallel(left(4, 2, 32, 48, 64, scale=0.2), right(4, 32, 64, 2, 4, 1)), moe(64, 8, 2, 3, limit=1.0)),
    layer("lightning", lightning(4, 16, 64, (0.6, 0.9, 0.99, 0.999)), moe(32, 4, 2, 1)),
    layer("parallel", parallel(left(8, 8, 16, 16, 150, scale=0.3, rot_dims=8, base=10000.0), right(8, 16, 32, 1, 3, 4), 0.4, 1.1), dense(72)),
])
# C: everything 1 that can be: heads, groups, taps, ranks, a window of one token, one expert; tau of one; no rotation.  (A norm
# over one channel leaves a sign: its weights are drawn so that no read-out of the tests' prompts lies next to zero.)
CONFIG_C = model(64, 32, [
    layer("parallel", parallel(left(1, 1, 1, 1, 1, scale=1.0, rot_dims=0), right(1, 1, 1, 1, 1, 1), 1.0, 1.0), moe(16, 1, 1)),
    layer("gla", gla(1, 1, 1, 1.0, 1), dense(16)),
    layer("lightning", lightning(1, 2, 3, (1.0,)), moe(8, 1, 1, 1)),
    layer("parallel", parallel(left(2, 1, 4, 3, 2, rot_dims=2), right(2, 3, 2, 1, 2, 6)), None),
])
# D: recurrent layers only (no paged cache group at all); decays of zero and of one; fast decays per channel
CONFIG_D = model(90, 48, [
    layer("lightning", lightning(6, 8, 8, (0.0, 1.0, 0.5, 0.9, 0.99, 0.999)), moe(32, 4, 1, 2)),
    layer("gla", gla(3, 16, 24, 0.5, 4), None),
    layer("gla", gla(1, 40, 16, 30.0, 8), dense(24)),
    layer("lightning", lightning(3, 16, 24, (0.7, 0.96, 0.9961)), moe(24, 2, 2, 1, limit=0.5)),
])
# E: a few hundred wide; sixteen query heads on two key heads, values wider than keys, attention without a window, and keys and
# values of 64 (portions of prompts on tcgen05); states of
# 128 x 64 and 96 x 128; more groups than one on the right; inner widths that are no multiple of a k-block
CONFIG_E = model(500, 384, [
    layer("parallel", parallel(left(16, 2, 64, 96, None, scale=0.12, rot_dims=32, base=10000.0), right(6, 64, 128, 3, 4, 2), 0.9, 0.3),
          moe(72, 12, 4, 4, limit=1.5)),
    layer("gla", gla(4, 96, 128, 16.0, 24), dense(200)),
    layer("lightning", lightning(3, 128, 64, (0.97, 0.99, 0.998)), moe(40, 6, 3, 2)),
    layer("parallel", parallel(left(6, 3, 64, 64, 100, scale=0.15), right(4, 48, 32, 4, 2, 1), 0.5, 0.8), dense(136)),
])
CONFIGS = {"A": (CONFIG_A, 11, 8), "B": (CONFIG_B, 12, 64), "C": (CONFIG_C, 23, 16), "D": (CONFIG_D, 14, 16), "E": (CONFIG_E, 15, 64)}
LENGTHS = {"A": (61, 9, 2, 34, 1, 27), "B": (150, 31, 77, 64, 3), "C": (40, 1, 17, 5), "D": (75, 3, 22, 1, 30), "E": (130, 40, 66, 7)}


def every_expert(raw: dict) -> dict:
    """The same model with every expert chosen for every token.  In bfloat16 two experts' scores lie within rounding of
    each other for a token now and then, the choice falls the other way, and through the states every later row of the
    request moves: no rounding bound holds then.  The bfloat16 runs of whole models use these variants; the choice itself
    is covered in float32 and, in bfloat16, on given logits."""
    out = json.loads(json.dumps(raw))
    for l in out["layers"]:
        if l.get("mlp") is not None and l["mlp"]["kind"] == "moe":
            r = l["mlp"]["router"]
            r["top"] = r["experts"] + r.get("identity", 0)
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

    t = {"embed": torch.randn(raw["vocab"], W, generator=g) * 0.7, "final.norm": vec(W, 0.2, 1.0)}
    for i, lr in enumerate(raw["layers"]):
        p, m, q = f"l{i}.", lr["mixer"], f"l{i}.mix."
        t[p + "norm1"] = vec(W, 0.2, 0.7)
        if lr["type"] == "parallel":
            a, s = m["left"], m["right"]
            L, R = q + "left.", q + "right."
            t[L + "q"], t[L + "k"] = mat(a["heads"] * a["dim"], W, 1.5), mat(a["kv_heads"] * a["dim"], W, 1.5)
            t[L + "v"], t[L + "o"] = mat(a["kv_heads"] * a["vdim"], W, 1.5), mat(W, a["heads"] * a["vdim"])
            t[L + "q.norm"], t[L + "k.norm"] = vec(a["heads"] * a["dim"], 0.3, 1.5), vec(a["kv_heads"] * a["dim"], 0.3, 1.5)
            inner, C = s["heads"] * s["vdim"], s["heads"] * s["vdim"] + 2 * s["groups"] * s["state"]
            t[R + "in"] = mat(inner + C + s["heads"], W, 1.5)
            t[R + "conv"], t[R + "conv.b"] = mat(C, s["conv"], 1.2), vec(C, 0.3)
            t[R + "dt_bias"], t[R + "A_log"], t[R + "D"] = vec(s["heads"], 1.0, -2.0), vec(s["heads"], 0.8), vec(s["heads"], 0.5, 1.0)
            t[R + "norm"], t[R + "o"] = vec(inner, 0.2, 1.0), mat(W, inner)
        else:
            H, A, B = m["heads"], m["heads"] * m["dim"], m["heads"] * m["vdim"]
            t[q + "q"], t[q + "k"], t[q + "v"] = mat(A, W, 1.5), mat(A, W, 1.5), mat(B, W, 1.5)
            t[q + "g"], t[q + "o"] = mat(B, W, 1.5), mat(W, B)
            t[q + "norm"] = vec(B if lr["type"] == "lightning" else m["vdim"], 0.2, 1.0)
            if lr["type"] == "gla":
                t[q + "a1"], t[q + "a2"], t[q + "a2.b"] = mat(m["decay_rank"], W), mat(A, m["decay_rank"], 1.5), vec(A, 1.5, 1.0)
        mlp = lr.get("mlp")
        if mlp is None:
            continue
        t[p + "norm2"] = vec(W, 0.2, 0.7)
        p += "mlp."
        if mlp["kind"] == "dense":
            F = mlp["ff"]
            t[p + "gate"], t[p + "up"], t[p + "down"] = mat(F, W, 1.5), mat(F, W, 1.2), mat(W, F, 0.8)
            t[p + "gate.b"], t[p + "up.b"], t[p + "down.b"] = vec(F, 0.5), vec(F, 0.5), vec(W, 0.3)
        else:
            n = mlp["router"]["experts"] + mlp["router"].get("identity", 0)
            t[p + "router"], t[p + "correction"] = mat(n, W, 1.5), vec(n, 0.2)
            F = mlp["expert"]["ff"]
            for e in range(mlp["router"]["experts"]):
                t[f"{p}e{e}.gate"], t[f"{p}e{e}.up"], t[f"{p}e{e}.down"] = mat(F, W, 1.5), mat(F, W, 1.2), mat(W, F, 0.8)
    return {k: v.to(torch.bfloat16).contiguous() for k, v in t.items()}


_folders = {}


def write_folder(raw: dict, weights: dict, d: str = None) -> str:
    """The folder's config.json has no decay ranks: a model file's tensors give them."""
    from safetensors.torch import save_file
    d = d or tempfile.mkdtemp(prefix="prism_nivotar_")
    out = json.loads(json.dumps(raw))
    for l in out["layers"]:
        l["mixer"].pop("decay_rank", None)
    with open(os.path.join(d, "config.json"), "w") as f:
        json.dump(out, f)
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
        _logits[key] = NP.forward(CONFIGS[name][0], plain_weights(name), list(seq))
    return _logits[key]


def plain_rounding(name: str, seq, dtype: str = "float32") -> list:
    """Per position: how far rounding alone moves the plain model from itself in float64.  For float32 it is the
    plain model run in float32; for bfloat16 the plain model in float64 with what a 16-bit engine may keep in 16 bits
    rounded to bfloat16."""
    key = (name, tuple(seq), dtype)
    if key not in _rounding:
        ref = plain_logits(name, seq)
        if dtype == "float32":
            low = NP.forward(CONFIGS[name][0], plain_weights(name, torch.float32), list(seq))
        else:
            low = NP.forward(CONFIGS[name][0], plain_weights(name), list(seq), rnd=to_bf16_and_back)
        scale = float((ref - ref.mean(-1, keepdim=True)).pow(2).mean().sqrt())
        _rounding[key] = [row_error(low[p], ref[p], scale) for p in range(len(seq))]
    return _rounding[key]


def compare(name: str, seqs: dict, got: dict, limit: float, ill: float = 0.0, dtype: str = "float32"):
    """Every row the trace produced against the plain model on the whole sequence."""
    errs = []
    for rid, seq in seqs.items():
        errs += errors(plain_logits(name, seq), got, rid, plain_rounding(name, seq, dtype))
    return judge(errs, limit, ill)
