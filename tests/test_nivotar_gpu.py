"""Nivotar on the GPU against the plain implementation (tests/plain/nivotar_plain.py): each kernel alone, each
mixer and feed-forward alone, whole prompts against token-by-token decoding, portions down to two tokens, mixed batches
with pages and state slots that are used again, keys at a window's edges, the first tokens of a sequence, long
decoding, and greedy generation through the engine's scheduler."""

import math
import types

import pytest
import torch

from nivotar_helpers import (CONFIGS, LENGTHS, NP, compare, dense, draw_weights, errors, every_expert, gla, judge, layer, left, lightning, model,
                             model_folder, moe, parallel, right, row_error, to_bf16_and_back, write_folder)
from helpers import random_tokens, run_trace, trace_budget, trace_mixed, trace_portions, trace_tail, trace_whole

pytestmark = pytest.mark.gpu
DEV = "cuda:0"
LIMIT = {"float32": 2e-5, "bfloat16": 2.5e-2}
ILL = {"float32": 0.0, "bfloat16": 0.05}
DTYPES = {"float32": torch.float32, "bfloat16": torch.bfloat16}


def alloc(shape, dtype):
    return torch.empty(shape, dtype=dtype, device=DEV)


def step_ctx(qlens, slots, dtype=torch.float32):
    """What a kernel sees of a step: segments of ``qlens`` tokens in ``slots``."""
    i32 = lambda x: torch.as_tensor(x, dtype=torch.int32).to(DEV)
    return types.SimpleNamespace(
        seg_start=i32([0] + torch.tensor(qlens).cumsum(0).tolist()), S=len(qlens), max_q_len=max(qlens), decode_only=max(qlens) == 1,
        tok_seg=i32(torch.cat([torch.full((n,), s) for s, n in enumerate(qlens)])), state_slots=i32(slots), scratch={}, alloc=alloc,
        positions=i32(torch.cat([torch.arange(n) for n in qlens])), dtype=dtype)


def pieces(lens, sizes):
    """Steps that feed every sequence in portions of changing size: lists of (sequence, first token, tokens)."""
    at, j = [0] * len(lens), 0
    while any(a < n for a, n in zip(at, lens)):
        live = [(s, at[s], min(sizes[(j + s) % len(sizes)], n - at[s])) for s, n in enumerate(lens) if at[s] < n]
        for s, _, n in live:
            at[s] += n
        j += 1
        yield live


# ---------------------------------------------------------------------------------------------------------
# kernels alone
# ---------------------------------------------------------------------------------------------------------

@pytest.mark.parametrize("T, W, nsplit", [(1, 8, 1), (5, 74, 3), (9, 384, 1), (3, 2048, 4), (2, 10000, 2), (2, 33, 1)])
@pytest.mark.parametrize("delta_dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("copy_dtype", [torch.float32, torch.bfloat16, None])
def test_norm_of_a_result_and_sum(T, W, nsplit, delta_dtype, copy_dtype):
    from prism_b200.parts.base import NormedDelta
    g = torch.Generator().manual_seed(T + W)
    x, d = torch.randn(T, W, generator=g), (torch.randn(nsplit, T, W, generator=g) * 3).to(delta_dtype)
    w = torch.randn(W, generator=g)
    ref = x.double() + NP.rms(d.double().sum(0), 1e-2) * w.double()
    xd = x.to(DEV)
    copy = None if copy_dtype is None else torch.empty(T, W, dtype=copy_dtype, device=DEV)
    NormedDelta(d.to(DEV) if nsplit > 1 else d[0].to(DEV), w.to(DEV), 1e-2).carry_out(xd, copy)
    assert float((xd.cpu().double() - ref).abs().max()) <= 1e-5 * float(ref.abs().max())
    if copy is not None:
        assert torch.equal(copy, xd.to(copy_dtype))


@pytest.mark.parametrize("T, W, F", [(1, 64, 40), (7, 256, 96), (16, 1024, 384), (33, 128, 72), (64, 520, 136), (130, 64, 48), (3, 30, 17)])
@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_gated_feed_forward_with_biases(T, W, F, dtype):
    """On every path: float32, the weight-streaming product with and without shares of K, the library's product."""
    from prism_b200 import ops
    g = torch.Generator().manual_seed(T + F)
    dt = DTYPES[dtype]
    w = {"gate": torch.randn(F, W, generator=g) / math.sqrt(W), "up": torch.randn(F, W, generator=g) / math.sqrt(W),
         "down": torch.randn(W, F, generator=g) / math.sqrt(F), "gate.b": torch.randn(F, generator=g), "up.b": torch.randn(F, generator=g) * 2,
         "down.b": torch.randn(W, generator=g)}
    w = {k: v.to(torch.bfloat16) for k, v in w.items()}
    x = torch.randn(T, W, generator=g).to(dt)
    wd = {k: v.double() for k, v in w.items()}
    ref = NP.dense_ff(x.double(), wd, "")
    dev = lambda *ns: torch.cat([w[n] for n in ns]).to(DEV) if ns[0].endswith(".b") else torch.cat([w[n] for n in ns]).to(dt).to(DEV)
    ctx = types.SimpleNamespace(alloc=alloc)
    gu, gb = dev("gate", "up"), dev("gate.b", "up.b")
    got = ops.feed_forward_glu(ctx, x.to(DEV), gu, dev("down"), "silu", 0.0, gb, dev("down.b"))
    got = (got if got.dim() == 2 else got.sum(0)).cpu().double()
    tol = 2e-5 if dtype == "float32" else 2.5e-2
    assert float((got - ref).abs().max()) <= tol * max(1.0, float(ref.abs().max()))
    if dtype == "bfloat16" and T <= 16 and W % 8 == 0:
        z = x.double() @ torch.cat([wd["gate"], wd["up"]]).T + torch.cat([wd["gate.b"], wd["up.b"]])
        for ks in (1, 2, 3):
            act = torch.empty(T, F, dtype=dt, device=DEV)
            for epi, ref_h in ((ops.EPI_SWIGLU, NP.silu(z[:, :F]) * z[:, F:]),
                               (ops.EPI_CLAMPED, z[:, :F].clamp(max=0.8) * torch.sigmoid(1.702 * z[:, :F].clamp(max=0.8)) * (z[:, F:].clamp(-0.8, 0.8) + 1))):
                ops.gemm_tc(x.to(DEV), gu, gb, act, epi, ksplit=ks, limit=0.8)
                assert float((act.cpu().double() - ref_h).abs().max()) <= tol * max(1.0, float(ref_h.abs().max())), (ks, epi)
        ops.check_tc_errors()


@pytest.mark.parametrize("C, K", [(64, 4), (130, 3), (7, 2), (512, 1), (96, 9)])
def test_convolution_with_bias_and_silu_in_pieces(C, K):
    from prism_b200 import ops
    g = torch.Generator().manual_seed(C + K)
    lens = (70, 23, 1)
    xs = [torch.randn(n, C + 6, generator=g) for n in lens]           # the product has more columns on both sides
    taps, bias = torch.randn(C, K, generator=g), torch.randn(C, generator=g)
    refs = [NP.silu(NP.short_conv(x[:, 4:4 + C].double(), taps.double(), bias.double())) for x in xs]
    for taps_t in (None, taps.t().contiguous().to(DEV)):
        tail = torch.zeros(4, K - 1, C, device=DEV)
        for live in pieces(lens, (20, 1, 1, 33, 2, 1)):
            ctx = step_ctx([n for _, _, n in live], [(3, 1, 2)[s] for s, _, _ in live])
            x = torch.cat([xs[s][a:a + n] for s, a, n in live]).to(DEV)
            out = torch.empty(x.shape[0], C, device=DEV)
            ops.causal_conv(x[:, 4:4 + C], taps.to(DEV), bias.to(DEV), tail, ctx, out, move_tail=ctx.decode_only, taps_t=taps_t, silu=True)
            if not ctx.decode_only:
                ops.state_tail(x[:, 4:4 + C], tail, ctx)
            o = 0
            for s, a, n in live:
                assert float((out[o:o + n].cpu().double() - refs[s][a:a + n]).abs().max()) <= 2e-5 * max(1.0, float(refs[s].abs().max())), (s, a)
                o += n


@pytest.mark.parametrize("T, parts, w", [(3, 1, 37), (5, 4, 64), (2, 3, 1030), (1, 1, 4096), (4, 2, 1)])
@pytest.mark.parametrize("first", [True, False])
@pytest.mark.parametrize("act", ["silu", "sigmoid"])
@pytest.mark.parametrize("out_dtype", [torch.float32, torch.bfloat16])
def test_norm_in_parts_with_a_gate_on_either_side(T, parts, w, first, act, out_dtype):
    from prism_b200 import ops
    g = torch.Generator().manual_seed(w)
    D = parts * w
    x, z, wt = torch.randn(T, D, generator=g) * 2, torch.randn(T, D + 5, generator=g), torch.randn(D, generator=g)
    f = NP.silu if act == "silu" else torch.sigmoid
    xd, zd = x.double(), f(z[:, :D].double())
    ref = NP.rms((xd * zd if first else xd).view(T, parts, w), 1e-3).reshape(T, D) * wt.double() * (1.0 if first else zd) * 0.6
    wide = torch.zeros(T, D + 8, dtype=out_dtype, device=DEV)
    ops.part_norm_gate(x.to(DEV), z.to(DEV)[:, :D], wt.to(DEV), 1e-3, parts, wide[:, 4:4 + D], act, first, 0.6)
    tol = 1e-5 if out_dtype == torch.float32 else 1e-2
    assert float((wide[:, 4:4 + D].cpu().double() - ref).abs().max()) <= tol * float(ref.abs().max())
    assert float(wide[:, :4].abs().max()) == float(wide[:, 4 + D:].abs().max()) == 0.0


def test_step_sizes_and_decays():
    from prism_b200 import ops
    z = torch.tensor([[-200.0, -3.0, 0.5, 30.0, 300.0]] * 3)
    bias, a_log = torch.tensor([0.0, 1.0, -1.0, 0.5, 0.0]), torch.tensor([0.0, -2.0, 2.0, -5.0, -9.0])
    bg = torch.empty(3, 10, device=DEV)
    ops.step_sizes(z.to(DEV), bias.to(DEV), a_log.to(DEV), bg)
    d = NP.softplus((z + bias).double())
    assert torch.allclose(bg[:, :5].cpu().double(), d, rtol=1e-5, atol=1e-7)
    assert torch.allclose(bg[:, 5:].cpu().double(), torch.exp(-torch.exp(a_log.double()) * d), rtol=1e-4, atol=1e-7)
    low, a2, b = torch.randn(20, 3), torch.randn(11, 3) * 3, torch.randn(11)
    zz = low.double() @ a2.double().T + b.double()
    out = torch.empty(20, 11, device=DEV)
    ops.lowrank_decay(low.to(DEV), a2.t().contiguous().to(DEV), b.to(DEV), out, inner_tanh=False, epilogue=ops.LR_SIGPOW, rate=1.0 / 16.0)
    assert torch.allclose(out.cpu().double(), torch.exp(-NP.softplus(-zz) / 16.0), rtol=1e-5, atol=1e-6)


def decayed_case(kind, H, rep, dk, dv, lens, g, strength=1.0, R=5):
    """Float32 rows of a product and the plain result per request: a dict of what the op gets beside them."""
    A, B = (H // rep) * dk, H * dv
    xs = [torch.randn(n, 2 * A + B, generator=g) for n in lens]
    args, decays = {}, []
    if kind == "head":
        args["decay"] = torch.tensor([0.9 ** strength] + [1.0 - 2.0 ** (-4 - 3 * i) for i in range(H - 1)])
        decays = [[args["decay"][i].double().expand(n, 1) for i in range(H)] for n in lens]
    elif kind == "token":
        args.update(dt_bias=torch.randn(H, generator=g), a_log=torch.randn(H, generator=g) + math.log(strength), skip=torch.randn(H, generator=g))
        args["dt"] = [torch.randn(n, H, generator=g) - 2.0 for n in lens]
        steps = [NP.softplus((d + args["dt_bias"]).double()) for d in args["dt"]]
        decays = [[torch.exp(-torch.exp(args["a_log"][i].double()) * s[:, i:i + 1]) for i in range(H)] for s in steps]
    else:
        args.update(a2t=torch.randn(R, H * dk, generator=g) * (5.0 / R) ** 0.5, a2_bias=torch.randn(H * dk, generator=g) * 2, rate=strength / 8.0)
        args["low"] = [torch.randn(n, R, generator=g) * 1.5 for n in lens]
        w = [torch.exp(-NP.softplus(-(l.double() @ args["a2t"].double() + args["a2_bias"].double())) * args["rate"]) for l in args["low"]]
        decays = [[x[:, i * dk:(i + 1) * dk] for i in range(H)] for x in w]
    refs = []
    for s, x in enumerate(xs):
        n, x = x.shape[0], x.double()
        f = NP.silu if kind == "head" else (lambda y: y)
        q, k, v = f(x[:, :A]).view(n, -1, dk), f(x[:, A:2 * A]).view(n, -1, dk), f(x[:, 2 * A:]).view(n, H, dv)
        o = torch.zeros(n, H, dv, dtype=torch.float64)
        for i in range(H):
            vv = v[:, i] * (steps[s][:, i:i + 1] if kind == "token" else 1.0)
            o[:, i] = NP.decayed_sum(q[:, i // rep], k[:, i // rep], vv, decays[s][i]) + (args["skip"][i].double() * v[:, i] if kind == "token" else 0.0)
        refs.append(o.reshape(n, B))
    return xs, args, refs


def decayed_sum(kind, ctx, rows, args, live, H, rep, dk, dv, state, out, path, gate=None, weight=None):
    from prism_b200 import ops
    A, B = (H // rep) * dk, H * dv
    at = lambda t: torch.cat([t[s][a:a + n] for s, a, n in live]).to(DEV)
    kw = {k: (at(v) if isinstance(v, list) else v.to(DEV) if torch.is_tensor(v) else v) for k, v in args.items()}
    if kind == "head":
        kw.update(powers=ops.decay_powers(kw["decay"]), silu=True)
    code = {"head": ops.DECAY_HEAD, "token": ops.DECAY_TOKEN, "channel": ops.DECAY_CHANNEL}[kind]
    ops.DecayedSum(code, rows[:, :A], rows[:, A:2 * A], rows[:, 2 * A:], H, rep, dk, dv, state, out, gate=gate, weight=weight, eps=1e-6,
                   **kw).run(ctx, path)


SHAPES = [(2, 1, 64, 32), (4, 2, 32, 64), (3, 3, 128, 64), (1, 1, 8, 8), (2, 1, 16, 136), (2, 1, 256, 24), (2, 2, 96, 256), (3, 1, 7, 5), (2, 1, 4, 3),
          (1, 1, 1, 1)]


@pytest.mark.parametrize("H, rep, dk, dv", SHAPES)
@pytest.mark.parametrize("sizes", [(64, 65, 63, 1, 16), (1,), (200,), (17, 2, 1, 1, 100)])
@pytest.mark.parametrize("kind", ["head", "token", "channel"])
def test_decayed_sums_in_pieces_on_every_path(kind, H, rep, dk, dv, sizes):
    """Three requests in slots 2, 0 and 3 (slot 1 is a neighbour's and must stay), cut into pieces of several sizes - ends
    on, one past and one short of a chunk's last token - against the plain recurrence in float64, the read-out itself and
    the one that is normed and gated per head."""
    from prism_b200 import ops
    if kind != "token":
        rep = 1
    g = torch.Generator().manual_seed(H * 1000 + dk)
    lens = (210, 75, 1) if sizes != (1,) else (19, 5, 1)
    B = H * dv
    xs, args, refs = decayed_case(kind, H, rep, dk, dv, lens, g)
    gates = [torch.randn(n, B, generator=g) for n in lens]
    weight = torch.randn(dv, generator=g)
    chunks = bool(ops.lib().prism_decay_chunks_supported(dk, dv, 0, 0))
    for path, dt in (("scan", torch.float32), (None, torch.float32), (None, torch.bfloat16)) + ((("chunks", torch.bfloat16),) if chunks else ()):
        for normed in (False, True) if kind != "token" else (False,):
            state = torch.zeros(4, H, dv, dk, device=DEV)
            state[1] = 5.0
            got = [torch.zeros(n, B) for n in lens]
            for live in pieces(lens, sizes):
                ctx = step_ctx([n for _, _, n in live], [(2, 0, 3)[s] for s, _, _ in live], dt)
                x = torch.cat([xs[s][a:a + n] for s, a, n in live]).to(DEV)
                z = torch.cat([gates[s][a:a + n] for s, a, n in live]).to(DEV) if normed else None
                out = torch.empty(x.shape[0], B, dtype=dt if normed else torch.float32, device=DEV)
                decayed_sum(kind, ctx, x, args, live, H, rep, dk, dv, state, out, path, z, weight.to(DEV) if normed else None)
                o = 0
                for s, a, n in live:
                    got[s][a:a + n] = out[o:o + n].float().cpu()
                    o += n
            for s in range(3):
                ref = refs[s]
                if normed:
                    ref = (NP.rms(ref.view(-1, H, dv), 1e-6) * weight.double()).reshape(-1, B) * NP.silu(gates[s].double())
                # per token, over the size of what is added up: a read-out may cancel to almost nothing
                scale = ref.pow(2).sum(1).sqrt()
                scale = torch.maximum(scale, scale.median()) if not normed else scale
                err = (got[s].double() - ref).pow(2).sum(1).sqrt() / scale
                tol = 2e-4 if dt == torch.float32 else (8e-3 if normed else 1e-3)
                if normed and dv < 8:           # a head of a few channels whose read-out cancels is normed up from its rounding
                    tol *= 20
                assert float(err.max()) <= tol, (path, dt, normed, s, int(err.argmax()), float(err.max()))
            assert float((state[1] - 5.0).abs().max()) == 0.0


@pytest.mark.parametrize("strength", [1e-4, 1.0, 40.0, 300.0])
@pytest.mark.parametrize("kind", ["token", "channel"])
def test_weak_and_strong_decays_in_chunks(kind, strength):
    """From decays that hardly act over a whole prompt to ones that leave nothing of a token after the next: sums of log
    decays up to thousands across a chunk, where factors of one sign only may be formed (a decay per channel beyond its
    limit across sixteen tokens goes term by term)."""
    g = torch.Generator().manual_seed(7)
    H, dk, dv, lens = 2, 48, 32, (150, 40)
    xs, args, refs = decayed_case(kind, H, 1, dk, dv, lens, g, strength)
    for path in ("chunks", "scan"):
        state, got = torch.zeros(2, H, dv, dk, device=DEV), []
        for live in pieces(lens, (100, 7)):
            ctx = step_ctx([n for _, _, n in live], [s for s, _, _ in live], torch.bfloat16)
            out = torch.empty(sum(n for _, _, n in live), H * dv, device=DEV)
            decayed_sum(kind, ctx, torch.cat([xs[s][a:a + n] for s, a, n in live]).to(DEV), args, live, H, 1, dk, dv, state, out, path)
            got.append((live, out.cpu().double()))
        assert bool(torch.isfinite(state).all())
        for live, out in got:
            o = 0
            for s, a, n in live:
                ref = refs[s][a:a + n]
                assert float((out[o:o + n] - ref).abs().max()) <= 1e-3 * float(refs[s].abs().max()), (path, s, a)
                o += n


@pytest.mark.parametrize("R", [1, 15, 16, 17, 40, 41, 130])
def test_ranks_of_the_decays_low_rank_product(R):
    """Below, at and above what the kernels keep in registers, and above what their tile of shared memory holds."""
    g = torch.Generator().manual_seed(R)
    H, dk, dv, lens = 2, 40, 8, (90, 1)
    xs, args, refs = decayed_case("channel", H, 1, dk, dv, lens, g, R=R)
    for path, sizes in (("chunks", (70, 20)), ("scan", (70, 20)), (None, (89, 1))):
        state = torch.zeros(2, H, dv, dk, device=DEV)
        for live in pieces(lens, sizes):
            ctx = step_ctx([n for _, _, n in live], [s for s, _, _ in live], torch.bfloat16)
            out = torch.empty(sum(n for _, _, n in live), H * dv, device=DEV)
            decayed_sum("channel", ctx, torch.cat([xs[s][a:a + n] for s, a, n in live]).to(DEV), args, live, H, 1, dk, dv, state, out, path)
            o = 0
            for s, a, n in live:
                assert float((out[o:o + n].cpu().double() - refs[s][a:a + n]).abs().max()) <= 1e-3 * float(refs[s].abs().max()), (path, s, a)
                o += n


@pytest.mark.parametrize("kind", ["head", "token", "channel"])
def test_an_old_token_comes_back_through_the_state_of_many_chunks(kind):
    """Keys and queries are orthogonal but for token 3: with decays close to one, what the last tokens read is token 3's
    value from five chunks earlier, and nothing else."""
    H, d, n = 1, 64, 330
    x = torch.zeros(n, 3 * d)
    x[:, 0] = 1.0                                            # every query looks along entry 0
    x[:, d + 1] = 1.0                                        # every key lies along entry 1
    x[:, 2 * d:] = torch.randn(n, d, generator=torch.Generator().manual_seed(1))
    x[3, d:2 * d] = 0.0
    x[3, d] = 1.0
    v = x[3, 2 * d:].double()
    silu1 = float(NP.silu(torch.tensor(1.0)))
    if kind == "head":
        args, rate, ref = dict(decay=torch.tensor([0.999])), 0.999, NP.silu(v) * silu1 * silu1
    elif kind == "token":
        dt = NP.softplus(torch.tensor(0.3).double())
        args = dict(dt=[torch.full((n, 1), 0.3)], dt_bias=torch.zeros(1), a_log=torch.tensor([math.log(0.001)]), skip=torch.zeros(1))
        rate, ref = float(torch.exp(-0.001 * dt)), v * dt
    else:
        args = dict(low=[torch.full((n, 1), 2.0)], a2t=torch.ones(1, d), a2_bias=torch.zeros(d), rate=0.01)
        rate, ref = float(torch.sigmoid(torch.tensor(2.0).double()) ** 0.01), v
    for path, dt in (("scan", torch.float32), ("chunks", torch.bfloat16)):
        state, out = torch.zeros(1, H, d, d, device=DEV), torch.empty(n, d, device=DEV)
        decayed_sum(kind, step_ctx([n], [0], dt), x.to(DEV), args, [(0, 0, n)], H, 1, d, d, state, out, path)
        for t in (3, 63, 64, 200, 329):
            want = ref * rate ** (t - 3)
            assert float((out[t].cpu().double() - want).abs().max()) <= 2e-4 * float(ref.abs().max()), (path, t)
        assert float(out[2].abs().max()) == 0.0              # nothing to read before token 3


@pytest.mark.parametrize("T, W, F, E, idle, top", [(1, 32, 16, 1, 1, 2), (7, 72, 24, 6, 2, 3), (8, 1024, 64, 4, 4, 2), (16, 640, 136, 12, 1, 4),
                                                   (33, 64, 40, 8, 8, 2), (64, 128, 64, 8, 3, 4), (130, 128, 64, 8, 2, 2), (9, 37, 11, 5, 3, 2),
                                                   (40, 64, 32, 2, 0, 1), (200, 96, 48, 3, 5, 8)])
@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_limited_experts_with_identity_experts(T, W, F, E, idle, top, dtype):
    """On given logits: the softmax over all of them, a correction on the choice only, the scores as they are, and identity
    experts at the end that return rows given in 32-bit."""
    from prism_b200 import ops
    g = torch.Generator().manual_seed(T * 7 + E)
    dt = DTYPES[dtype]
    mk = lambda *s: (torch.randn(*s, generator=g) * (1.5 / math.sqrt(s[-1]))).to(dt)
    own = torch.randn(T, W, generator=g)
    x, z = own.to(dt), torch.randn(T, E + idle, generator=g) * 2
    corr = (torch.randn(E + idle, generator=g) * 0.2).to(torch.bfloat16)
    gu, dn, limit = mk(E, 2 * F, W), mk(E, W, F), 0.7
    w = {f"e{e}.{n}": t.double() for e in range(E) for n, t in (("gate", gu[e, :F]), ("up", gu[e, F:]), ("down", dn[e]))}
    ref = torch.zeros(T, W, dtype=torch.float64)
    used = set()
    for t in range(T):
        for e, wt in zip(*NP.route(z[t].double(), corr.double(), top)):
            used.add(e >= E)
            ref[t] += wt * (NP.clamped_expert(x[t:t + 1].double(), w, f"e{e}.", limit)[0] if e < E else own[t].double())
    assert T < 7 or used == ({False, True} if idle else {False})
    ctx = types.SimpleNamespace(alloc=alloc)
    tol = 2e-5 if dtype == "float32" else 2.5e-2
    keep = ops.moe_tensor_cores
    for tc in (True, False):
        ops.moe_tensor_cores = tc
        try:
            y = ops.moe_feed_forward(ctx, x.to(DEV), z.to(DEV), gu.to(DEV), dn.to(DEV), top, True, False, False, act="clamped", limit=limit,
                                     choice=ops.MoeChoice(corr.to(DEV)), own=own.to(DEV))
        finally:
            ops.moe_tensor_cores = keep
        assert y.shape == (top, T, W)
        assert float((y.sum(0).cpu().double() - ref).abs().max()) <= tol * max(1.0, float(ref.abs().max())), tc
    ops.check_tc_errors()


@pytest.mark.parametrize("hd, nh, nkv", [(64, 4, 2), (128, 6, 1), (64, 3, 3)])
@pytest.mark.parametrize("window", [None, 1, 30, 64, 65, 100, 500])
def test_windowed_attention_of_portions_with_weights_as_two_terms(hd, nh, nkv, window):
    """Portions that start and end around pages, tiles and windows, single tokens among them, NaN in the slots nothing was
    stored in, and one key that stands out just inside and just outside the last query's window: on tcgen05 and on the
    masked mma.sync kernel."""
    from prism_b200 import ops
    g = torch.Generator().manual_seed(hd + nh)
    mask, P = ops.KeyMask.window(window), 64
    segs = [(0, 3), (200, 70), (63, 2), (0, 130), (330, 128), (447, 1)]
    per = [-(-(c + n) // P) for c, n in segs]
    order = torch.randperm(sum(per), generator=g).tolist()
    bt = torch.full((len(segs), max(per)), sum(per), dtype=torch.int32)
    k, v = torch.randn(sum(per) + 1, P, nkv, hd, generator=g), torch.randn(sum(per) + 1, P, nkv, hd, generator=g)
    T = sum(n for _, n in segs)
    q, ids, o = torch.randn(T, nh, hd, generator=g), [], 0
    for s, (c, n) in enumerate(segs):
        ids.append(order[o:o + per[s]])
        bt[s, :per[s]] = torch.tensor(ids[s], dtype=torch.int32)
        o += per[s]
        if (c + n) % P:
            k[ids[s][-1], (c + n) % P:] = math.nan
            v[ids[s][-1], (c + n) % P:] = math.nan
    edge = 330 + 127 - (window or 10 ** 6) + 1                # the first key the fifth request's last query sees
    for key in (edge - 1, edge):
        if 0 <= key <= 457:
            k[ids[4][key // P], key % P] = 0.0
            k[ids[4][key // P], key % P, :, :8] = 8.0
            v[ids[4][key // P], key % P] = 50.0 if key == edge else -300.0
    last = sum(n for _, n in segs[:5]) - 1
    q[last] = 0.0
    q[last, :, :8] = 8.0
    q, k, v = q.to(torch.bfloat16), k.to(torch.bfloat16), v.to(torch.bfloat16)
    refs, t = [], 0
    for s, (c, n) in enumerate(segs):
        kk, vv = (x[ids[s]].reshape(-1, nkv, hd)[:c + n].double() for x in (k, v))
        see = NP.visible(c + n, window)[c:]
        row = torch.zeros(n, nh, hd, dtype=torch.float64)
        for h in range(nh):
            sc = (q[t:t + n, h].double() @ kk[:, h // (nh // nkv)].T * 0.1).masked_fill(~see, -math.inf)
            row[:, h] = torch.softmax(sc, -1) @ vv[:, h // (nh // nkv)]
        refs.append(row.reshape(n, nh * hd))
        t += n
    ref = torch.cat(refs)
    i32 = lambda x: torch.as_tensor(x, dtype=torch.int32).to(DEV)
    ctx = types.SimpleNamespace(S=len(segs), max_q_len=130, max_kv_len=458, decode_only=False, err=torch.zeros(1, dtype=torch.int32, device=DEV),
                                seg_start=i32([0] + torch.tensor([n for _, n in segs]).cumsum(0).tolist()), cached_len=i32([c for c, _ in segs]))
    qd, kd, vd, btd = q.to(DEV), k.to(DEV), v.to(DEV), bt.to(DEV)
    keep = ops.ATTENTION_TC
    for tc in (True, False):
        ops.ATTENTION_TC = tc
        try:
            out = torch.zeros(T, nh * hd + 8, dtype=torch.bfloat16, device=DEV)[:, :nh * hd]
            assert ops.masked_prefill_tc_ok(ctx, qd, out, kd, vd, mask, 0.1) == tc
            ops.masked_attention(ctx, qd, out, kd, vd, btd, sum(per), mask, 0.1)
        finally:
            ops.ATTENTION_TC = keep
        assert int(ctx.err.item()) == 0
        err = (out.float().cpu().double() - ref).abs()
        # the result is rounded to bfloat16 once; the weights are not
        assert bool((err <= 2.0 ** -8 * ref.abs() + 2e-3).all()), (tc, float(err.max()))
    ops.check_tc_errors()


# ---------------------------------------------------------------------------------------------------------
# whole models
# ---------------------------------------------------------------------------------------------------------

def runner_for(folder, dtype, max_tokens, page_size, max_live=4):
    from prism_b200.engine.replay import build_runner
    return build_runner(folder, dtype, max_tokens, page_size, max_live)[3]


def sequences(name):
    vocab = CONFIGS[name][0]["vocab"]
    return {f"r{i}": random_tokens(vocab, n, 300 + i) for i, n in enumerate(LENGTHS[name[0]])}


def served(name, dtype):
    """The configuration a dtype is tested on: in bfloat16 the variant in which every expert is chosen."""
    return name + "x" if dtype == "bfloat16" else name


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("name", ["A", "B", "C", "D", "E"])
@pytest.mark.parametrize("mode", ["whole", "tail", "portions", "small_portions", "mixed"])
def test_cutting(name, dtype, mode):
    """Whole prompts, a decoded tail, portions (one schedule of twos and threes only), and mixed batches of up to four
    live requests in a pool that holds no more than the schedule needs, so that pages and state slots come back and
    are used again."""
    name = served(name, dtype)
    seqs = sequences(name)
    steps = {"whole": trace_whole, "tail": lambda s: trace_tail(s, 48), "portions": trace_portions,
             "small_portions": lambda s: trace_portions(s, (2, 3, 2, 2, 5, 2)),
             "mixed": lambda s: trace_mixed(s, seed=3)}[mode](seqs)
    ps = CONFIGS[name][2]
    runner = runner_for(model_folder(name), dtype, trace_budget(steps, max(ps, 64)), ps)
    got = run_trace(runner, steps)
    assert len(got) == sum(len(s) for s in seqs.values())
    compare(name, seqs, got, LIMIT[dtype], ILL[dtype], dtype)
    assert runner.cache.pages_in_use() == 0 and len(runner.cache.requests) == 0


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_the_stream_after_every_layer(dtype):
    """The residual rows after each layer, whole prompt, against the plain model's: a fault shows in the layer that has it."""
    from prism_b200.engine.batch import Segment
    for name in (served("A", dtype), served("B", dtype)):
        raw, seed, ps = CONFIGS[name]
        seq = random_tokens(raw["vocab"], 45, 7)
        wd = {k: v.double() for k, v in draw_weights(raw, seed).items()}
        after, rounded = [], []
        NP.forward(raw, wd, seq, streams=after)
        if dtype == "bfloat16":
            NP.forward(raw, wd, seq, rnd=to_bf16_and_back, streams=rounded)
        else:
            rounded = after
        runner = runner_for(model_folder(name), dtype, 64, ps)
        kept = []

        def watch(block):
            inner = block.forward

            def forward(ctx, residual, delta, cache):
                x, d = inner(ctx, residual, delta, cache)
                y = d.delta.float() if d.delta.dim() == 2 else d.delta.float().sum(0)
                kept.append((x + NP.rms(y, d.eps) * d.weight.float()).cpu())
                return x, d
            block.forward = forward
        for block in runner.model.layers:
            watch(block)
        runner.begin_request("a")
        runner.step([Segment("a", seq, [44])])
        runner.check_errors()
        assert len(kept) == len(after)
        for i, x in enumerate(kept):
            scale = float(after[i].pow(2).mean().sqrt())
            err = float((x - after[i]).pow(2).mean().sqrt()) / scale
            own = float((rounded[i] - after[i]).pow(2).mean().sqrt()) / scale          # what rounding alone does here
            assert err <= (2e-5 if dtype == "float32" else max(1e-2, 3 * own)), (name, i, err, own)


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_long_decoding_across_pages(dtype):
    name = served("B", dtype)
    seq = random_tokens(CONFIGS[name][0]["vocab"], 420, 9)
    runner = runner_for(model_folder(name), dtype, 448, 64)
    got = run_trace(runner, trace_tail({"a": seq}, 300))
    compare(name, {"a": seq}, got, LIMIT[dtype], ILL[dtype], dtype)


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("name", ["A", "E"])
def test_batches_of_unequal_requests_against_each_alone(name, dtype):
    name = served(name, dtype)
    seqs = sequences(name)
    ps = CONFIGS[name][2]
    alone = run_trace(runner_for(model_folder(name), dtype, 4096, ps), trace_portions(seqs, (5, 2, 40, 9)))
    together = run_trace(runner_for(model_folder(name), dtype, 4096, ps, max_live=5), trace_mixed(seqs, seed=11, max_live=5))
    tol = 2e-5 if dtype == "float32" else 8e-2
    for key, row in alone.items():
        assert float((row - together[key]).abs().max()) <= tol * max(1.0, float(row.abs().max())), key


def test_a_state_slot_that_is_used_again_starts_from_zero():
    """One slot only: the second request gets the slot the first one left, and must not inherit its states."""
    for letter, ps in (("D", 16), ("B", 64)):
        vocab = CONFIGS[letter][0]["vocab"]
        seqs = {"a": random_tokens(vocab, 40, 1), "b": random_tokens(vocab, 25, 2), "c": random_tokens(vocab, 2, 3)}
        for dtype, sizes in (("float32", (7, 1, 3)), ("bfloat16", (20, 1, 1, 17))):
            name = served(letter, dtype)
            runner = runner_for(model_folder(name), dtype, 64, ps, max_live=1)
            got = run_trace(runner, trace_portions(seqs, sizes))
            compare(name, seqs, got, LIMIT[dtype], ILL[dtype], dtype)


TINY = layer("lightning", lightning(1, 4, 4, (0.9,)), None)
ONE_LAYER = {
    "parallel": [layer("parallel", parallel(left(4, 2, 16, 24, 20), right(4, 8, 16, 2, 4, 2)), None)],
    "parallel_all_equal": [layer("parallel", parallel(left(4, 4, 16, 16, 16, rot_dims=16), right(4, 16, 16, 4, 4, 4), 1.0, 1.0), None)],
    "parallel_left_only": [layer("parallel", parallel(left(6, 3, 8, 16, 12, rot_dims=4), right(2, 8, 8, 1, 2, 1), 0.8, 0.0), None)],
    "parallel_right_only": [layer("parallel", parallel(left(2, 1, 8, 8, 4), right(6, 8, 24, 3, 3, 2), 0.0, 1.5), None)],
    "lightning": [layer("lightning", lightning(4, 24, 16, (0.5, 0.9, 0.97, 0.99)), None)],
    "gla": [layer("gla", gla(4, 24, 16, 16.0, 8), None)],
    "gla_fast": [layer("gla", gla(2, 32, 64, 0.2, 3), None)],
    "dense": [dict(TINY, mlp=dense(40))],
    "experts": [dict(TINY, mlp=moe(24, 6, 2, 2, limit=0.5))],
    "experts_only": [dict(TINY, mlp=moe(20, 5, 2))],
    "mostly_identity": [dict(TINY, mlp=moe(16, 1, 3, 6))],
    "odd_sizes": [layer("parallel", parallel(left(3, 1, 5, 7, 9, rot_dims=4), right(3, 3, 5, 3, 3, 1)), moe(9, 3, 2, 1)),
                  layer("gla", gla(3, 6, 5, 3.0, 2), dense(13)), layer("lightning", lightning(2, 3, 7, (0.9, 0.5)), None)],
}


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("which", sorted(ONE_LAYER))
def test_each_mixer_and_feed_forward_alone(which, dtype):
    odd = which == "odd_sizes"
    raw = model(51 if odd else 97, 37 if odd else 48, ONE_LAYER[which])
    if dtype == "bfloat16":
        raw = every_expert(raw)
    w = draw_weights(raw, 21)
    folder = write_folder(raw, w)
    seq = random_tokens(raw["vocab"], 95, 4)
    wd = {k: v.double() for k, v in w.items()}
    ref = NP.forward(raw, wd, seq)
    low = NP.forward(raw, wd, seq, rnd=to_bf16_and_back) if dtype == "bfloat16" else NP.forward(raw, {k: v.float() for k, v in w.items()}, seq)
    scale = float((ref - ref.mean(-1, keepdim=True)).pow(2).mean().sqrt())
    runner = runner_for(folder, dtype, 128, 16)
    got = run_trace(runner, trace_portions({"a": seq}, (20, 1, 1, 30, 2, 1)))
    judge(errors(ref, got, "a", [row_error(low[p], ref[p], scale) for p in range(95)]), LIMIT[dtype], ILL[dtype])


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("size, page", [(1, 16), (7, 4), (64, 64), (65, 64), (100, 16)])
def test_a_windows_edges(size, page, dtype):
    """Two prompts that differ in one token, a layer of which only the attention counts: the last position that sees the
    token differs by a lot, the next one not at all - in prompts, in decoding, in portions that are cut at the edge - and
    each agrees with the plain model."""
    raw = model(60, 64, [layer("parallel", parallel(left(4, 2, 16, 32, size, scale=0.5, rot_dims=0), right(2, 8, 8, 1, 2, 1), 1.0, 0.0), None)])
    w = draw_weights(raw, 5)
    folder = write_folder(raw, w)
    wd = {k: v.double() for k, v in w.items()}
    base = [t if t not in (2, 4) else 7 for t in random_tokens(60, 3 * size + 30, 6)]
    at = 9
    seqs = {"a": base[:at] + [2] + base[at + 1:], "b": base[:at] + [4] + base[at + 1:]}
    refs = {k: NP.forward(raw, wd, s).float() for k, s in seqs.items()}
    inside, outside = at + size - 1, at + size
    scale = float(refs["a"].std())
    assert float((refs["a"][outside] - refs["b"][outside]).abs().max()) == 0.0
    shown = float((refs["a"][inside] - refs["b"][inside]).abs().max())
    tol = 2e-5 if dtype == "float32" else 3e-2
    assert shown > (5 * tol * scale if size <= 7 or dtype == "float32" else 0.0)
    n = len(base)
    cut = {"whole": trace_whole(seqs), "decoded": trace_tail(seqs, n - at - 1), "at_the_edge": trace_portions(seqs, (inside, 1, 2, n)),
           "behind_it": trace_portions(seqs, (outside, 2, n)), "portions": trace_portions(seqs)}
    for how, steps in cut.items():
        got = run_trace(runner_for(folder, dtype, 4 * (n // 64 + 2) * 64, page), steps)
        for rid in seqs:
            for pos in (0, 1, at, inside - 1, inside, outside, outside + 1, n - 1):
                assert float((got[(rid, pos)] - refs[rid][pos]).abs().max()) <= tol * max(1.0, float(refs[rid].abs().max())), (how, rid, pos)
        same = float((got[("a", outside)] - got[("b", outside)]).abs().max())
        assert same == 0.0, (how, same)
        if dtype == "float32":
            assert float((got[("a", inside)] - got[("b", inside)]).abs().max()) > 0.5 * shown, how


@pytest.mark.parametrize("kind", ["lightning", "gla", "state_space"])
def test_a_first_token_decides_through_the_mixer_alone(kind):
    """A model of one layer whose first token differs between two prompts that are otherwise equal and several hundred
    tokens long: the logits at the end differ, in a whole prompt and when the end is decoded token by token, and each
    agrees with the plain model."""
    mixer = {"lightning": lightning(2, 16, 16, (0.999, 0.9999)), "gla": gla(2, 16, 16, 500.0, 4),
             "state_space": parallel(left(1, 1, 4, 4, 2), right(2, 16, 16, 1, 2, 1), 0.0, 1.0)}[kind]
    raw = model(60, 64, [layer("parallel" if kind == "state_space" else kind, mixer, None)])
    w = draw_weights(raw, 5)
    if kind == "state_space":
        w["l0.mix.right.A_log"] = torch.full((2,), -8.0).to(torch.bfloat16)
        w["l0.mix.right.dt_bias"] = torch.zeros(2).to(torch.bfloat16)
    folder = write_folder(raw, w)
    base = [t if t != 2 else 7 for t in random_tokens(60, 390, 6)]
    seqs = {"a": [2] + base, "b": [4] + base}
    wd = {k: v.double() for k, v in w.items()}
    refs = {k: NP.forward(raw, wd, s).float() for k, s in seqs.items()}
    tol = 2e-5 * float(refs["a"].abs().max())
    assert float((refs["a"][-1] - refs["b"][-1]).abs().max()) > 5 * tol
    for steps in (trace_whole(seqs), trace_tail(seqs, 70)):
        got = run_trace(runner_for(folder, "float32", 1024, 64), steps)
        for rid in seqs:
            for pos in (0, 1, 49, 63, 64, 320, 389, 390):
                assert float((got[(rid, pos)] - refs[rid][pos]).abs().max()) <= tol, (rid, pos)


def test_greedy_generation_through_the_scheduler():
    """Engine.generate (scheduler, batching, sampling, CUDA graphs for the decode steps) picks the plain model's greedy
    tokens; more prompts than request slots, so that state slots are used again."""
    from prism_b200.config.engine_config import EngineConfig, SchedulerConfig
    from prism_b200.engine.llm import Engine
    from prism_b200.sampling.sampler import SamplingParams
    raw, seed, ps = CONFIGS["A"]
    w = {k: v.double() for k, v in draw_weights(raw, seed).items()}
    prompts = [random_tokens(raw["vocab"], n, 40 + n) for n in (3, 17, 30, 8, 1, 12)]
    n_new = 24
    folder = model_folder("A")
    for graphs in (False, True):
        eng = Engine(folder, EngineConfig(kv_page_size=ps, num_pages=40, max_seq_len=128, use_cuda_graph=graphs,
                                          graph_batch_sizes=(1, 2, 4, 8),
                                          scheduler=SchedulerConfig(max_batch_tokens=48, max_num_seqs=4, prefill_chunk=16)),
                     dtype="float32")
        assert eng.runner.use_cuda_graph == graphs
        res = eng.generate(prompts, SamplingParams(max_new_tokens=n_new, ignore_eos=True))
        for p, r in zip(prompts, res):
            logits = NP.forward(raw, w, list(p) + r.token_ids)
            for i, tok in enumerate(r.token_ids):
                row = logits[len(p) - 1 + i]
                top = torch.topk(row, 2).values
                if float(top[0] - top[1]) > 1e-3:          # a near tie may fall either way
                    assert tok == int(row.argmax()), (graphs, len(p), i)
            assert len(r.token_ids) == n_new
        assert eng.cache.pages_in_use() == 0


def test_decode_graphs_give_what_eager_steps_give():
    """bfloat16, the fused decode kernels throughout: the same tokens through captured graphs and step by step."""
    from prism_b200.config.engine_config import EngineConfig, SchedulerConfig
    from prism_b200.engine.llm import Engine
    from prism_b200.sampling.sampler import SamplingParams
    prompts = [random_tokens(500, n, 60 + n) for n in (70, 5, 33)]
    out = []
    for graphs in (False, True):
        eng = Engine(model_folder("E"), EngineConfig(kv_page_size=64, num_pages=12, max_seq_len=256, use_cuda_graph=graphs,
                                                     graph_batch_sizes=(1, 2, 4), scheduler=SchedulerConfig(max_num_seqs=4)), dtype="bfloat16")
        out.append([r.token_ids for r in eng.generate(prompts, SamplingParams(max_new_tokens=20, ignore_eos=True))])
    assert out[0] == out[1]


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_the_replay_program_serves_the_design(tmp_path, dtype):
    """bin/trace_run as a user runs it, on a Nivotar folder: the model class is found by config.json, the pool holds what
    --max-tokens says and there are four slots."""
    import json
    import os
    import subprocess
    import sys
    import numpy as np
    root = os.path.dirname(os.path.dirname(os.path.abspath(__file__)))
    name = served("B", dtype)
    raw = CONFIGS[name][0]
    folder = model_folder(name)
    vocab = raw["vocab"]
    seqs = {f"q{i}": random_tokens(vocab, n, 500 + i) for i, n in enumerate([70, 33, 90, 12, 64, 5])}
    steps = trace_mixed(seqs, seed=17)
    out = tmp_path / "out"
    proc = subprocess.run([sys.executable, os.path.join(root, "bin", "trace_run"), "--model", folder, "--dtype", dtype,
                           "--out", str(out), "--max-tokens", str(trace_budget(steps, 64))],
                          input="\n".join(json.dumps(s) for s in steps) + "\n", capture_output=True, text=True, timeout=600)
    assert proc.returncode == 0, proc.stderr[-2000:]
    assert [l for l in proc.stdout.split("\n") if l.startswith("done")] == [f"done {s['step']}" for s in steps]
    got, fed = {}, {}
    for s in steps:
        n_want = sum(len(e["want"]) for e in s["entries"])
        data = np.fromfile(out / f"{s['step']}.f32", dtype="<f4").reshape(n_want, vocab)
        r = 0
        for e in s["entries"]:
            for w in e["want"]:
                got[(e["id"], fed.get(e["id"], 0) + w)] = torch.from_numpy(data[r].copy())
                r += 1
            fed[e["id"]] = fed.get(e["id"], 0) + len(e["tokens"])
    assert len(got) == sum(len(s) for s in seqs.values())
    compare(name, seqs, got, LIMIT[dtype], ILL[dtype], dtype)
