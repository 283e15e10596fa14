"""Limatar on the GPU against the plain implementation (tests/plain/limatar_plain.py): each kernel alone, each
mixer alone, whole prompts against token-by-token decoding, portions down to two tokens, mixed batches with pages
and state slots that are used again, keys far back and at page borders, the first tokens of a sequence, long
decoding, and greedy generation through the engine's scheduler."""

import math
import types

import pytest
import torch

from limatar_helpers import (CONFIGS, LENGTHS, LP, compare, dense, draw_weights, errors, every_expert, judge, latent, layer, model, model_folder,
                             moe, retain, row_error, to_bf16_and_back, write_folder, yarn)
from helpers import random_tokens, run_trace, trace_budget, trace_mixed, trace_portions, trace_tail, trace_whole

pytestmark = pytest.mark.gpu
DEV = "cuda:0"
LIMIT = {"float32": 2e-5, "bfloat16": 2.5e-2}
ILL = {"float32": 0.0, "bfloat16": 0.05}
DTYPES = {"float32": torch.float32, "bfloat16": torch.bfloat16}


def alloc(shape, dtype):
    return torch.empty(shape, dtype=dtype, device=DEV)


def step_ctx(qlens, slots, first=None):
    """What a kernel sees of a step: segments of ``qlens`` tokens in ``slots``, starting at positions ``first``."""
    first = first or [0] * len(qlens)
    i32 = lambda x: torch.as_tensor(x, dtype=torch.int32).to(DEV)
    return types.SimpleNamespace(
        seg_start=i32([0] + torch.tensor(qlens).cumsum(0).tolist()), S=len(qlens), max_q_len=max(qlens), decode_only=max(qlens) == 1,
        tok_seg=i32(torch.cat([torch.full((n,), s) for s, n in enumerate(qlens)])), state_slots=i32(slots), scratch={}, alloc=alloc,
        positions=i32(torch.cat([torch.arange(p, p + n) for p, n in zip(first, qlens)])))


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
@pytest.mark.parametrize("out_dtype", [torch.float32, torch.bfloat16])
def test_norm_sum_and_norm_in_one_launch(T, W, nsplit, delta_dtype, out_dtype):
    from prism_b200 import ops
    g = torch.Generator().manual_seed(T + W)
    x, d = torch.randn(T, W, generator=g), (torch.randn(nsplit, T, W, generator=g) * 3).to(delta_dtype)
    wd, w = torch.randn(W, generator=g), torch.randn(W, generator=g)
    eps_d, eps = 1e-2, 1e-3
    ref_x = x.double() + LP.rms(d.double().sum(0), eps_d) * wd.double()
    ref_h = LP.rms(ref_x, eps) * w.double()
    tol = 1e-5 if out_dtype == torch.float32 else 2e-2
    for rows in (None, [T - 1, 0]):
        xd, out = x.to(DEV), torch.empty(T if rows is None else 2, W, dtype=out_dtype, device=DEV)
        ops.add_normed_rmsnorm(xd, d.to(DEV) if nsplit > 1 else d[0].to(DEV), wd.to(DEV), eps_d, w.to(DEV), eps, out,
                               None if rows is None else torch.tensor(rows, dtype=torch.int32, device=DEV))
        assert float((out.cpu().double() - (ref_h if rows is None else ref_h[rows])).abs().max()) <= tol * float(ref_h.abs().max())
        want = ref_x if rows is None else x.double()          # a norm of some rows leaves the stream alone
        assert float((xd.cpu().double() - want).abs().max()) <= 1e-5 * float(want.abs().max())


@pytest.mark.parametrize("T, W, F", [(1, 64, 40), (7, 256, 96), (16, 1024, 384), (33, 128, 72), (64, 520, 136), (130, 64, 48), (3, 30, 17)])
@pytest.mark.parametrize("limit", [0.4, 7.0])
@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_clamped_hidden_layer(T, W, F, limit, dtype):
    """The product and its epilogue, on every path (float32, the weight-streaming product with and without shares of K, the
    library's product and the elementwise kernel)."""
    from prism_b200 import ops
    g = torch.Generator().manual_seed(T + F)
    dt = DTYPES[dtype]
    x, gu = torch.randn(T, W, generator=g).to(dt), (torch.randn(2 * F, W, generator=g) * 2 / math.sqrt(W)).to(dt)
    h = x.double() @ gu.double().T
    gg, uu = h[:, :F].clamp(max=limit), h[:, F:].clamp(-limit, limit)
    ref = gg * torch.sigmoid(1.702 * gg) * (uu + 1.0)
    ctx = types.SimpleNamespace(alloc=alloc)
    tol = 2e-5 if dtype == "float32" else 2.5e-2
    got = ops.glu_hidden(ctx, x.to(DEV), gu.to(DEV), "clamped", limit).cpu().double()
    assert float((got - ref).abs().max()) <= tol * max(1.0, float(ref.abs().max()))
    if dtype == "bfloat16" and T <= 16 and W % 8 == 0:
        for ks in (1, 2, 3):
            act = torch.empty(T, F, dtype=dt, device=DEV)
            for kind, epi in (("clamped", ops.EPI_CLAMPED), ("silu", ops.EPI_SWIGLU), ("gelu_tanh", ops.EPI_GEGLU)):
                ops.gemm_tc(x.to(DEV), gu.to(DEV), None, act, epi, ksplit=ks, limit=limit)
                if kind == "clamped":
                    assert float((act.cpu().double() - ref).abs().max()) <= tol * max(1.0, float(ref.abs().max())), ks
                elif ks == 1:
                    first = {} if kind == "silu" else first
                    first[kind] = act.clone()
                else:
                    assert float((act.float() - first[kind].float()).abs().max()) <= 2e-2 * max(1.0, float(first[kind].abs().max()))
        ops.check_tc_errors()


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("R, r, q_rank, dims", [(13, 10, 11, 10), (96, 32, 64, 32), (1400, 8, 1100, 4), (3, 2, 3, 2)])
@pytest.mark.parametrize("interleaved", [True, False])
def test_cache_row_and_rotation_with_an_amplitude(dtype, R, r, q_rank, dims, interleaved):
    from prism_b200 import ops
    g = torch.Generator().manual_seed(R)
    dt, T, P = DTYPES[dtype], 6, 8
    x = torch.randn(T, q_rank + R + r + 5, generator=g)                       # the product has more columns behind
    w, wq = torch.randn(R, generator=g), torch.randn(q_rank, generator=g)
    pos = torch.tensor([0, 7, 8, 63, 1000, 4097], dtype=torch.int32)
    bt = torch.arange(600, dtype=torch.int32).flip(0).view(1, 600).to(DEV)
    plane = torch.zeros(600, P, 1, R + r, dtype=dt, device=DEV)
    freq = (50.0 ** (-torch.arange(dims // 2).double() * 2 / dims)).float()
    err = torch.zeros(1, dtype=torch.int32, device=DEV)
    cq = torch.empty(T, q_rank, dtype=dt, device=DEV)
    xd, seg = x.to(DEV), torch.zeros(T, dtype=torch.int32, device=DEV)
    ops.latent_kv_store(xd[:, q_rank:q_rank + R + r], w.to(DEV), 1e-5, R, dims, freq.to(DEV), plane, bt, pos.to(DEV), seg, 600, 1 << 20, err,
                        xq=xd[:, :q_rank], q_weight=wq.to(DEV), q_out=cq, interleaved=interleaved, amplitude=1.3)
    assert int(err.item()) == 0
    ref_k = torch.zeros(T, R + r, dtype=torch.float64)
    turned = torch.zeros(T, r, dtype=torch.float64)
    for t, p in enumerate(pos.tolist()):
        kr = x[t, q_rank + R:q_rank + R + r].double()
        y = kr.clone()
        for i in range(dims // 2):
            a, b = (2 * i, 2 * i + 1) if interleaved else (i, i + dims // 2)
            ang = float(torch.tensor(float(p)) * freq[i])                     # a float32 angle
            c, s = 1.3 * math.cos(ang), 1.3 * math.sin(ang)
            y[a], y[b] = kr[a] * c - kr[b] * s, kr[b] * c + kr[a] * s
        turned[t] = y
        ref_k[t] = torch.cat([LP.rms(x[t, q_rank:q_rank + R].double(), 1e-5) * w.double(), y])
    tol = 1e-5 if dtype == "float32" else 1e-2
    got = torch.stack([plane[599 - p // P, p % P, 0] for p in pos.tolist()]).cpu().double()
    assert float((got - ref_k).abs().max()) <= tol * float(ref_k.abs().max())
    assert int((plane.float().abs().sum(-1) > 0).sum()) == T                  # and nothing else was written
    ref_q = LP.rms(x[:, :q_rank].double(), 1e-5) * wq.double()
    assert float((cq.cpu().double() - ref_q).abs().max()) <= tol * float(ref_q.abs().max())
    src = x[:, q_rank + R:q_rank + R + r].contiguous().to(dt).to(DEV).view(T, 1, r)
    ops.rotate_slice(src, src, dims, freq.to(DEV), pos.to(DEV), interleaved, 1.3, 0.5)      # in place, all entries halved
    assert float((src.cpu().double().view(T, r) - 0.5 * turned).abs().max()) <= tol * float(turned.abs().max())
    ops.latent_kv_store(xd[:1, q_rank:q_rank + R + r], w.to(DEV), 1e-5, R, dims, freq.to(DEV), plane, bt, torch.tensor([1 << 20], dtype=torch.int32, device=DEV),
                        seg[:1], 600, 1 << 20, err)
    assert int(err.item()) == 3                                               # a position beyond the limit is reported, not followed


@pytest.mark.parametrize("T", [1, 5, 16, 17, 64])
@pytest.mark.parametrize("H, N, K, r, dims, pairs", [(4, 48, 32, 16, 16, True), (3, 20, 8, 0, 0, True), (20, 160, 64, 32, 32, True),
                                                     (2, 24, 96, 8, 4, False), (1, 128, 192, 0, 0, False), (5, 9, 256, 6, 2, True)])
def test_per_head_products_of_a_few_tokens(T, H, N, K, r, dims, pairs):
    from prism_b200 import ops
    from prism_b200.parts.base import RotaryParams
    g = torch.Generator().manual_seed(T + N)
    wide = (K + r + 7) // 8 * 8
    x = torch.randn(T, H, wide, generator=g).to(torch.bfloat16)
    w = (torch.randn(H, N, K, generator=g) / math.sqrt(K)).to(torch.bfloat16)
    gate = torch.randn(T, H * N + 3, generator=g) * 2
    ref = torch.einsum("thk,hnk->thn", x[..., :K].double(), w.double())
    xd = x.to(DEV)[..., :K + r]
    assert ops.head_product_ok(xd, w.to(DEV))
    out = torch.empty(T, H, N, dtype=torch.bfloat16, device=DEV)
    ops.head_product(xd[..., :K], w.to(DEV), out, gate.to(DEV)[:, :H * N])
    gated = ref * torch.sigmoid(gate[:, :H * N].double()).view(T, H, N)
    assert float((out.cpu().double() - gated).abs().max()) <= 1e-2 * max(1.0, float(gated.abs().max()))
    if r:
        pos = torch.arange(T) * 37 + 3
        rot = RotaryParams((30.0 ** (-torch.arange(dims // 2).double() * 2 / max(dims, 1))).float().to(DEV), dims, pairs, 1.2)
        out = torch.full((T, H, N + r), 7.0, dtype=torch.bfloat16, device=DEV)
        ops.head_product(xd, w.to(DEV), out, rot=rot, positions=pos.to(torch.int32).to(DEV))
        full = torch.zeros(int(pos[-1]) + 1, H, r, dtype=torch.float64)
        full[pos] = x[..., K:K + r].double()
        turned = LP.rotate(full, dict(dims=dims, base=30.0), pairs)[pos]
        turned[..., :dims] *= 1.2
        assert float((out[..., :N].cpu().double() - ref).abs().max()) <= 1e-2 * max(1.0, float(ref.abs().max()))
        assert float((out[..., N:].cpu().double() - turned).abs().max()) <= 1.5e-2 * float(turned.abs().max())


@pytest.mark.parametrize("H, dk, dv, rot, pairs", [(3, 64, 64, 64, False), (2, 128, 128, 64, False), (1, 8, 8, 8, False), (2, 40, 24, 16, False),
                                                   (2, 256, 96, 128, False), (2, 72, 256, 0, False), (3, 16, 48, 12, True), (2, 5, 3, 4, False),
                                                   (1, 2, 1030, 2, True), (1, 300, 20, 100, False)])
@pytest.mark.parametrize("sizes", [(210,), (100, 30, 64, 6), (17, 3, 1, 1, 64, 65, 40, 9), (1,)])
def test_retention_in_pieces_on_every_path(H, dk, dv, rot, pairs, sizes):
    """Three requests in slots 2, 0 and 3 (slot 1 is a neighbour's and must stay), cut into pieces of several sizes - ends
    on, one past and one short of a chunk's last token - against the plain recurrence in float64; one decay far below one
    and, with more heads, others close to it."""
    from prism_b200 import ops
    from prism_b200.parts.base import RotaryParams
    g = torch.Generator().manual_seed(H * 1000 + dk)
    lens = (210, 75, 1) if sizes != (1,) else (19, 5, 1)
    A, B = H * dk, H * dv
    xs = [torch.randn(n, 2 * A + 2 * B, generator=g) for n in lens]
    decay = [0.9] + [1.0 - 2.0 ** (-4 - 3 * i) for i in range(H - 1)]
    rp = RotaryParams((100.0 ** (-torch.arange(rot // 2).double() * 2 / max(rot, 1))).float().to(DEV), rot, pairs, 1.0)
    refs = []
    for x in xs:
        n, x = x.shape[0], x.double()
        turn = lambda y: LP.rotate(y, dict(dims=rot, base=100.0), pairs) if rot else y
        q, k, v = turn(x[:, :A].view(n, H, dk)), turn(x[:, A:2 * A].view(n, H, dk)) * dk ** -0.5, x[:, 2 * A:2 * A + B].view(n, H, dv)
        o = torch.stack([LP.rms(LP.retain(q[:, i], k[:, i], v[:, i], decay[i]), 1e-6) for i in range(H)], 1)
        refs.append(o.reshape(n, B) * LP.silu(x[:, 2 * A + B:]))
    dd = torch.tensor(decay, device=DEV)
    powers = ops.decay_powers(dd)
    chunks = bool(ops.lib().prism_decay_chunks_supported(dk, dv, rot, 1 if pairs else 0))
    for path, dt in (("scan", torch.float32), ("scan", torch.bfloat16), (None, torch.float32), (None, torch.bfloat16)) + \
            ((("chunks", torch.bfloat16),) if chunks else ()):
        state = torch.zeros(4, H, dv, dk, device=DEV)
        state[1] = 5.0
        got = [torch.zeros(n, B) for n in lens]
        for live in pieces(lens, sizes):
            ctx = step_ctx([n for _, _, n in live], [(2, 0, 3)[s] for s, _, _ in live], [a for _, a, _ in live])
            x = torch.cat([xs[s][a:a + n] for s, a, n in live]).to(DEV)
            out = torch.empty(x.shape[0], B, dtype=dt, device=DEV)
            ops.retention(ctx, x, H, dk, dv, rp, dd, powers, state, 1e-6, out, path=path)
            o = 0
            for s, a, n in live:
                got[s][a:a + n] = out[o:o + n].float().cpu()
                o += n
        for s in range(3):
            err = ((got[s].double() - refs[s]).pow(2).sum(1) / refs[s].pow(2).sum(1)).sqrt()
            assert float(err.max()) <= (1e-4 if dt == torch.float32 else 6e-3), (path, dt, s, int(err.argmax()), float(err.max()))
        assert float((state[1] - 5.0).abs().max()) == 0.0


def test_an_old_token_comes_back_through_the_state_of_many_chunks():
    """Keys and queries are orthogonal but for token 3 and the last one, and the decay is close to one: what the last token
    reads is token 3's value from five chunks earlier, and nothing else."""
    from prism_b200 import ops
    H, d, n = 1, 64, 330
    x = torch.zeros(n, 4 * d)
    x[:, 0] = 1.0                                            # every query looks along entry 0
    x[:, d + 1] = 1.0                                        # every key lies along entry 1
    x[:, 2 * d:3 * d] = torch.randn(n, d, generator=torch.Generator().manual_seed(1))
    x[:, 3 * d:] = 1.0
    x[3, d:2 * d] = 0.0
    x[3, d] = 1.0
    v = x[3, 2 * d:3 * d].double()
    ref = v / v.pow(2).mean().sqrt() * float(LP.silu(torch.tensor(1.0)))
    decay = torch.tensor([0.999], device=DEV)
    for path, dt in (("scan", torch.float32), ("chunks", torch.bfloat16)):
        state = torch.zeros(1, H, d, d, device=DEV)
        out = torch.empty(n, d, dtype=dt, device=DEV)
        ops.retention(step_ctx([n], [0]), x.to(DEV), H, d, d, None, decay, ops.decay_powers(decay), state, 1e-12, out, path=path)
        for t in (3, 63, 64, 200, 329):
            assert float((out[t].cpu().double() - ref).abs().max()) <= 1e-2, (path, t)
        assert float(out[2].abs().max()) == 0.0              # nothing to read before token 3
        s = state[0, 0].cpu()                                # [value channel, key channel]
        assert float((s[:, 0].double() / d ** -0.5 - 0.999 ** (n - 4) * v).abs().max()) <= 1e-4


@pytest.mark.parametrize("T, W, F, E, top, Fs", [(1, 32, 16, 1, 1, 16), (7, 72, 24, 6, 3, 40), (8, 1024, 64, 4, 2, 192), (16, 640, 136, 12, 4, 72),
                                                 (33, 64, 40, 8, 2, 24), (64, 128, 64, 8, 4, 96), (130, 128, 64, 8, 2, 64), (9, 37, 11, 5, 2, 13)])
@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_experts_with_a_shared_one_in_their_launches(T, W, F, E, top, Fs, dtype):
    """Gated experts on given logits, weights the softmax over the chosen, beside an expert of another width that every
    token goes through: in the experts' own launches (with and without shares of K) and on its own."""
    from prism_b200 import ops
    g = torch.Generator().manual_seed(T * 7 + E)
    dt = DTYPES[dtype]
    mk = lambda *s: (torch.randn(*s, generator=g) / math.sqrt(s[-1])).to(dt)
    x, z = torch.randn(T, W, generator=g).to(dt), torch.randn(T, E, generator=g) * 2
    gu, dn, sgu, sdn = mk(E, 2 * F, W), mk(E, W, F), mk(2 * Fs, W), mk(W, Fs)
    ff = lambda h, gw, dw, n: (LP.silu(h @ gw[:n].T) * (h @ gw[n:].T)) @ dw.T
    ref = ff(x.double(), sgu.double(), sdn.double(), Fs)
    for t in range(T):
        for e, wt in zip(*LP.route(z[t].double(), top)):
            ref[t] += wt * ff(x[t].double(), gu[e].double(), dn[e].double(), F)
    ctx = types.SimpleNamespace(alloc=alloc)
    tol = 2e-5 if dtype == "float32" else 2.5e-2
    keep = ops.MOE_SHARED_TOKENS
    for riding in (0, 64):
        ops.MOE_SHARED_TOKENS = riding
        try:
            y = ops.moe_feed_forward(ctx, x.to(DEV), z.to(DEV), gu.to(DEV), dn.to(DEV), top, True, True, False,
                                     shared=(sgu.to(DEV), sdn.to(DEV)))
        finally:
            ops.MOE_SHARED_TOKENS = keep
        assert y.shape == (top + 1, T, W)
        got = y.sum(0).cpu().double()
        assert float((got - ref).abs().max()) <= tol * max(1.0, float(ref.abs().max())), riding
    ops.check_tc_errors()


def latent_case(segs, nh, R, rd, page_size, dtype, seed, boost=None, mask=None):
    """One key row per position (all heads share it), its first R entries the value; pages in a scrambled order."""
    g = torch.Generator().manual_seed(seed)
    per = [-(-(c + n) // page_size) for c, n in segs]
    order = torch.randperm(sum(per) + 3, generator=g).tolist()
    bt = torch.full((len(segs), max(per)), sum(per) + 3, dtype=torch.int32)
    rows = torch.randn(sum(per) + 4, page_size, 1, R + rd, generator=g)
    T = sum(n for _, n in segs)
    q = torch.randn(T, nh, R + rd, generator=g)
    sink = torch.randn(nh, generator=g)
    ids, o = [], 0
    for s in range(len(segs)):
        ids.append(order[o:o + per[s]])
        bt[s, :per[s]] = torch.tensor(ids[s], dtype=torch.int32)
        o += per[s]
    if boost is not None:
        boost(q, rows, ids)
    i32 = lambda x: torch.as_tensor(x, dtype=torch.int32).to(DEV)
    ctx = types.SimpleNamespace(
        positions=i32(torch.cat([torch.arange(c, c + n) for c, n in segs])), S=len(segs), max_q_len=max(n for _, n in segs),
        tok_seg=i32(torch.cat([torch.full((n,), s) for s, (_, n) in enumerate(segs)])), max_kv_len=max(c + n for c, n in segs),
        seg_start=i32([0] + torch.tensor([n for _, n in segs]).cumsum(0).tolist()), cached_len=i32([c for c, _ in segs]),
        decode_only=all(n == 1 for _, n in segs), err=torch.zeros(1, dtype=torch.int32, device=DEV))
    q, rows = q.to(dtype), rows.to(dtype)
    outs, t = [], 0
    for s, (c, n) in enumerate(segs):
        k = rows[ids[s]].reshape(-1, R + rd)[:c + n].double()
        for i in range(n):
            first = mask.first_key(c + i) if mask is not None else 0
            sc = (q[t].double() @ k[first:c + i + 1].T) * 0.2
            outs.append(LP.sink_softmax(sc, sink.double()[:, None]) @ k[first:c + i + 1, :R])
            t += 1
    return ctx, q.to(DEV), rows.to(DEV), bt.to(DEV), sink, torch.stack(outs).reshape(T, nh * R)


KERNELS = ["generic_f32", "generic_bf16", "tc_portions", "tc_decode", "tc_decode:3", "tc_decode:7", "tcgen05", "tcgen05:3"]


def latent_attention(kernel, segs, nh, R, rd, page_size, seed, boost=None, mask=None):
    from prism_b200 import ops
    dtype = torch.float32 if kernel == "generic_f32" else torch.bfloat16
    ctx, q, rows, bt, sink, ref = latent_case(segs, nh, R, rd, page_size, dtype, seed, boost, mask)
    out = torch.empty(q.shape[0], nh * R, dtype=dtype, device=DEV)
    mask, n = mask or ops.KeyMask.causal(), rows.shape[0]
    if kernel.startswith("tcgen05"):
        if not ops.attention_latent_tc_ok(q, out, rows, rows[..., :R], mask):
            assert page_size % 64
            pytest.skip("key tiles do not lie in one page")
        ops.attention_latent_tc(q, out, rows, R, bt, ctx.seg_start, ctx.cached_len, ctx.S, ctx.max_q_len, n, mask, 0.2, sink.to(DEV), ctx.err,
                                nsplit=int(kernel.split(":")[1]) if ":" in kernel else 1)
        ops.check_tc_errors()
    elif kernel.startswith("generic"):
        ops.attention_masked_generic(q, out, rows, rows[..., :R], bt, ctx.positions, ctx.tok_seg, n, mask, 0.2, sink.to(DEV), ctx.err)
    else:
        few = kernel.startswith("tc_decode")
        ops.attention_masked_bf16(q, out, rows, rows[..., :R], bt, ctx.seg_start, ctx.cached_len, ctx.S, ctx.max_q_len, n, mask, 0.2,
                                  sink.to(DEV), few, ctx.err, nsplit=int(kernel.split(":")[1]) if ":" in kernel else 1)
    assert int(ctx.err.item()) == 0
    return out.float().cpu(), ref.float()


@pytest.mark.parametrize("shape", [(4, 48, 16), (20, 160, 32), (3, 192, 64), (1, 8, 8), (17, 64, 0), (2, 256, 32)], ids=lambda s: "h%d_R%d_r%d" % s)
@pytest.mark.parametrize("page_size", [64, 16, 24])
@pytest.mark.parametrize("kernel", KERNELS)
def test_latent_attention_with_a_sink(shape, page_size, kernel):
    """Portions that start and end around pages and key tiles (whole tiles in one page take the loader's short way), single
    tokens just before, on and behind a page border, and contexts whose first tiles are asked for before the wait."""
    single, portions = [(0, 1), (63, 1), (64, 1), (300, 1), (129, 1), (447, 1)], [(0, 3), (200, 40), (63, 2), (0, 130)]
    for segs in ((single,) if kernel.startswith("tc_decode") else (portions, single) if kernel.startswith("tcgen05") else (portions,)):
        got, ref = latent_attention(kernel, segs, *shape, page_size, 5)
        assert float((got - ref).abs().max()) <= (2e-5 if kernel == "generic_f32" else 2e-2) * max(1.0, float(ref.abs().max()))


@pytest.mark.parametrize("window", [1, 30, 64, 65, 100, 500])
@pytest.mark.parametrize("kernel", ["generic_f32", "tc_portions", "tcgen05", "tcgen05:2"])
def test_latent_attention_under_a_window(window, kernel):
    from prism_b200 import ops
    got, ref = latent_attention(kernel, [(0, 3), (200, 40), (63, 2), (0, 130), (330, 70)], 6, 80, 16, 64, 7, mask=ops.KeyMask.window(window))
    assert float((got - ref).abs().max()) <= (2e-5 if kernel == "generic_f32" else 2e-2) * max(1.0, float(ref.abs().max()))


def test_unwritten_rows_of_a_page_do_not_reach_the_result():
    """The slots behind the last key of a page hold NaN (a pool that nothing was stored in yet): no kernel may let them in."""
    from prism_b200 import ops
    for segs in ([(0, 70), (64, 30)], [(69, 1), (3, 1)]):
        few = segs[0][1] == 1

        def boost(q, rows, ids):
            for (c, n), pages in zip(segs, ids):
                last = c + n
                if last % 64:
                    rows[pages[(last - 1) // 64], last % 64:] = math.nan
        for kernel in (("generic_f32", "tc_decode", "tc_decode:3") if few else ("generic_f32", "tc_portions", "tcgen05", "tcgen05:2")):
            got, ref = latent_attention(kernel, segs, 4, 96, 32, 64, 3, boost)
            assert bool(torch.isfinite(got).all()), kernel
            assert float((got - ref).abs().max()) <= 2e-2 * max(1.0, float(ref.abs().max())), kernel


@pytest.mark.parametrize("kernel", KERNELS)
@pytest.mark.parametrize("key", [0, 1, 63, 64, 191, 383, 384, 398, 399])
def test_one_key_that_stands_out(kernel, key):
    """Among 400 keys one has a score far above the rest and a value of hundreds: it is the whole output of the last query,
    wherever it lies - first, at a page's border, the query's own."""
    for segs in ([(399, 1)], [(380, 20)]):
        if kernel == "tc_portions" and segs[0][1] == 1 or kernel.startswith("tc_decode") and segs[0][1] > 1:
            continue
        one_key(kernel, segs, key)


def one_key(kernel, segs, key):
    def boost(q, rows, ids):
        q[-1] = 0.0
        q[-1, :, 48:] = 6.0                                   # the last query looks at the rotated part only
        rows[:, :, :, 48:] *= 0.1
        row = rows[ids[0][key // 64], key % 64, 0]
        row[48:] = 6.0
        row[:48] = 300.0
    got, ref = latent_attention(kernel, segs, 4, 48, 16, 64, 9, boost)
    assert float(ref[-1].min()) > 290.0
    assert float((got - ref).abs().max()) <= (2e-5 if kernel == "generic_f32" else 2e-2) * float(ref.abs().max())


@pytest.mark.parametrize("kernel", KERNELS)
def test_a_large_sink_takes_the_weight(kernel):
    """All scores are equal and the sink's number is ln(keys): half of the weight has no value."""
    from prism_b200 import ops
    n = 256
    segs = [(n - 1, 1)]
    dtype = torch.float32 if kernel == "generic_f32" else torch.bfloat16
    ctx, q, rows, bt, _, _ = latent_case(segs, 2, 16, 8, 64, dtype, 3)
    rows[..., :16], q[...] = 1.0, 0.0
    out = torch.empty(1, 32, dtype=dtype, device=DEV)
    for value, share in ((math.log(n), 0.5), (-40.0, 1.0), (math.log(3.0 * n), 0.25)):
        sink = torch.full((2,), value, device=DEV)
        if kernel.startswith("tcgen05"):
            ops.attention_latent_tc(q, out, rows, 16, bt, ctx.seg_start, ctx.cached_len, 1, 1, rows.shape[0], ops.KeyMask.causal(), 0.2, sink,
                                    ctx.err, nsplit=int(kernel.split(":")[1]) if ":" in kernel else 1)
        elif kernel.startswith("generic"):
            ops.attention_masked_generic(q, out, rows, rows[..., :16], bt, ctx.positions, ctx.tok_seg, rows.shape[0], ops.KeyMask.causal(), 0.2,
                                         sink, ctx.err)
        else:
            few = kernel.startswith("tc_decode")
            ops.attention_masked_bf16(q, out, rows, rows[..., :16], bt, ctx.seg_start, ctx.cached_len, 1, 1, rows.shape[0], ops.KeyMask.causal(),
                                      0.2, sink, few, ctx.err, nsplit=int(kernel.split(":")[1]) if ":" in kernel else 1)
        assert float((out.float() - share).abs().max()) <= 5e-3, value


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("T", [1, 40])
def test_the_routers_bias_joins_the_logits(T, dtype):
    from prism_b200 import ops
    g = torch.Generator().manual_seed(T)
    dt = DTYPES[dtype]
    x, w, b = torch.randn(T, 64, generator=g).to(dt), torch.randn(5, 64, generator=g).to(dt), torch.randn(5, generator=g).to(torch.bfloat16)
    got = ops.linear(x.to(DEV), w.to(DEV), b.to(DEV), out_dtype=torch.float32)
    ref = x.double() @ w.double().T + b.double()
    assert got.dtype == torch.float32 and float((got.cpu().double() - ref).abs().max()) <= 1e-4


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
def test_the_stream_after_every_layer_run(dtype):
    """The residual rows after each run of a layer (every pass of the loop), whole prompt, against the plain model's: a
    fault shows in the run that has it."""
    from prism_b200.engine.batch import Segment
    for name in (served("A", dtype), served("B", dtype)):
        raw, seed, ps = CONFIGS[name]
        seq = random_tokens(raw["vocab"], 45, 7)
        wd = {k: v.double() for k, v in draw_weights(raw, seed).items()}
        after, rounded = [], []
        LP.forward(raw, wd, seq, streams=after)
        if dtype == "bfloat16":
            LP.forward(raw, wd, seq, rnd=to_bf16_and_back, streams=rounded)
        else:
            rounded = after
        runner = runner_for(model_folder(name), dtype, 64, ps)
        kept = []

        def watch(block):
            inner = block.forward

            def forward(ctx, residual, delta, cache):
                x, d = inner(ctx, residual, delta, cache)
                y = d.delta.float() if d.delta.dim() == 2 else d.delta.float().sum(0)
                kept.append((x + LP.rms(y, d.eps) * d.weight.float()).cpu())
                return x, d
            block.forward = forward
        for block in runner.model.layers:
            watch(block)
        runner.begin_request("a")
        runner.step([Segment("a", seq, [44])])
        runner.check_errors()
        assert len(kept) == len(LP.run_order(raw)) == len(after)
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
    seqs = {"a": random_tokens(90, 40, 1), "b": random_tokens(90, 25, 2), "c": random_tokens(90, 2, 3)}
    for dtype, sizes in (("float32", (7, 1, 3)), ("bfloat16", (20, 1, 1, 17))):
        name = served("D", dtype)
        runner = runner_for(model_folder(name), dtype, 64, 16, max_live=1)
        got = run_trace(runner, trace_portions(seqs, sizes))
        compare(name, seqs, got, LIMIT[dtype], ILL[dtype], dtype)


ONE_LAYER = {
    "latent": [layer("latent", latent(4, 16, 8, 24, 16, 40, scaling=yarn()), None)],
    "latent_without_scaling": [layer("latent", latent(2, 24, 16, 8, 32, 32, scale=0.2), None)],
    "latent_all_equal": [layer("latent", latent(4, 16, 16, 16, 16, 16, scaling=yarn(2.0, 30, 6.0, 1.5)), None)],
    "retention": [layer("retention", retain(4, 24, 16, (0.5, 0.9, 0.97, 0.99)), None)],
    "retention_partly_turned": [layer("retention", retain(2, 32, 32, (0.8, 0.95), rot_dims=8), None)],
    "clamped": [layer("retention", retain(1, 4, 4, (0.9,)), dense(40, 0.5))],
    "experts": [layer("retention", retain(1, 4, 4, (0.9,)), moe(24, 6, 2, shared=16))],
    "experts_without_shared": [layer("retention", retain(1, 4, 4, (0.9,)), moe(20, 5, 2))],
    "looped": [layer("latent", latent(2, 8, 8, 8, 16, 16), dense(24, 1.5)), layer("retention", retain(2, 8, 16, (0.9, 0.6)), None)],
    "odd_sizes": [layer("latent", latent(3, 5, 6, 7, 9, 11, scaling=yarn(3.0, 20, 4.0, 1.0)), moe(9, 3, 2, shared=5)),
                  layer("retention", retain(3, 6, 5, (0.9, 0.5, 0.98), rot_dims=2), dense(13, 1.0))],
}


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("which", sorted(ONE_LAYER))
def test_each_mixer_alone(which, dtype):
    odd = which == "odd_sizes"
    raw = model(51 if odd else 97, 37 if odd else 48, ONE_LAYER[which], loop=(0, 2, 4) if which == "looped" else None)
    if dtype == "bfloat16":
        raw = every_expert(raw)
    w = draw_weights(raw, 21)
    folder = write_folder(raw, w)
    seq = random_tokens(raw["vocab"], 95, 4)
    wd = {k: v.double() for k, v in w.items()}
    ref = LP.forward(raw, wd, seq)
    low = LP.forward(raw, wd, seq, rnd=to_bf16_and_back) if dtype == "bfloat16" else LP.forward(raw, {k: v.float() for k, v in w.items()}, seq)
    scale = float((ref - ref.mean(-1, keepdim=True)).pow(2).mean().sqrt())
    runner = runner_for(folder, dtype, 128, 16)
    got = run_trace(runner, trace_portions({"a": seq}, (20, 1, 1, 30, 2, 1)))
    judge(errors(ref, got, "a", [row_error(low[p], ref[p], scale) for p in range(95)]), LIMIT[dtype], ILL[dtype])


@pytest.mark.parametrize("kind", ["latent", "retention"])
def test_a_first_token_decides_through_the_mixer_alone(kind):
    """A model of one layer whose first token differs between two prompts that are otherwise equal and several hundred
    tokens long: the logits at the end differ, in a whole prompt and when the end is decoded token by token, and each
    agrees with the plain model.  (Attention: the positions' part is taken out of the weights and the last token is one
    that looks at the first prompt's first token and at no other.)"""
    mixer = latent(4, 16, 8, 16, 24, 32, scale=1.0) if kind == "latent" else retain(2, 16, 16, (0.999, 0.9999))
    raw = model(60, 64, [layer(kind, mixer, None)])
    w = draw_weights(raw, 5)
    if kind == "latent":
        w["l0.mix.dkv"][32:] = 0.0
    folder = write_folder(raw, w)
    base = [t if t != 2 else 7 for t in random_tokens(60, 389, 6)] + [20]
    seqs = {"a": [2] + base, "b": [4] + base}
    wf = {k: v.double() for k, v in w.items()}
    refs = {k: LP.forward(raw, wf, s).float() for k, s in seqs.items()}
    tol = 2e-5 * float(refs["a"].abs().max())
    assert float((refs["a"][-1] - refs["b"][-1]).abs().max()) > 50 * tol
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
            logits = LP.forward(raw, w, list(p) + r.token_ids)
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
    """bin/trace_run as a user runs it, on a Limatar folder: the model class is found by config.json, the pool holds what
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
