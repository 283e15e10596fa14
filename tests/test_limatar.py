"""Limatar without a GPU: configuration and refusals, tensor names against a drawn model file, the order of runs, what
each run keeps between steps and how the cache manager groups it, the rotation's frequencies, and properties of the
plain mechanisms that the GPU tests lean on."""

import copy
import math

import pytest
import torch

from limatar_helpers import CONFIGS, LP, dense, draw_weights, latent, layer, model, moe, retain, yarn


def build(raw):
    from prism_b200.model_registry import build_model
    return build_model(copy.deepcopy(raw))


def test_the_registry_finds_the_design_and_every_tensor_has_a_taker():
    from prism_b200.model_registry import registered_architectures
    assert "Limatar" in registered_architectures()
    for name, (raw, seed, _) in CONFIGS.items():
        w = draw_weights(raw, seed)
        _, mdl = build(raw)
        asked = {s.name: tuple(s.shape) for _, spec in mdl.named_params() for s in spec.sources if not spec.optional}
        assert asked == {k: tuple(v.shape) for k, v in w.items()}, name


@pytest.mark.parametrize("edit, text", [
    (lambda r: r.pop("norm"), "norm"),
    (lambda r: r.pop("vocab"), "vocab"),
    (lambda r: r["layers"][0].update(type="attention"), "latent_attention"),
    (lambda r: r["layers"][0]["mixer"].pop("scale"), "scale"),
    (lambda r: r["layers"][0]["mixer"].pop("kv_rank"), "kv_rank"),
    (lambda r: r["layers"][0]["mixer"]["rot"].update(dims=11), "dims"),
    (lambda r: r["layers"][0]["mixer"]["rot"].update(dims=12), "rot_dim"),
    (lambda r: r["layers"][0]["mixer"]["rot"]["scaling"].pop("slow"), "slow"),
    (lambda r: r["layers"][0]["mixer"]["rot"]["scaling"].update(factor=0), "factor"),
    (lambda r: r["layers"][1]["mixer"].update(decay=[0.5]), "decay"),
    (lambda r: r["layers"][1]["mixer"].pop("dim"), "dim"),
    (lambda r: r["layers"][2]["mlp"].pop("limit"), "limit"),
    (lambda r: r["layers"][2]["mlp"].update(limit=-1.0), "limit"),
    (lambda r: r["layers"][2]["mlp"].update(kind="glu"), "dense"),
    (lambda r: r["layers"][0]["mlp"]["router"].update(top=6), "top"),
    (lambda r: r["loop"].update(stop=9), "loop"),
    (lambda r: r["loop"].update(times=0), "loop"),
    (lambda r: r["loop"].pop("start"), "start"),
])
def test_refusals_name_the_key(edit, text):
    from prism_b200.config.model_config import ConfigError
    raw = copy.deepcopy(CONFIGS["A"][0])
    edit(raw)
    with pytest.raises(ConfigError, match=text):
        build(raw)


def test_the_loop_runs_its_layers_in_a_row_each_pass_with_a_cache_of_its_own():
    from prism_b200.cache.manager import plan_groups
    cfg, mdl = build(CONFIGS["A"][0])
    assert cfg.run_order() == LP.run_order(CONFIGS["A"][0]) == [0, 1, 2, 1, 2, 3]
    groups, where = plan_groups(mdl.cache_needs(), [e.reads_cache_of for e in mdl.schedule])
    assert all(owns for _, _, owns in where) and len({w[:2] for w in where}) == 6         # six planes, none shared
    assert [groups[w[0]].kind for w in where] == ["paged", "state", "paged", "state", "paged", "state"]
    assert where[1][0] == where[3][0] and where[2][0] == where[4][0]                      # passes of a layer: one group
    assert len(mdl.layers) == 4                                                          # the weights are there once
    assert build(CONFIGS["E"][0])[0].run_order() == [0, 1, 2, 3]                          # no loop
    raw = model(40, 16, CONFIGS["C"][0]["layers"], loop=(1, 1, 5))
    assert build(raw)[0].run_order() == LP.run_order(raw) == [0, 1, 2]                   # a loop around nothing


def test_what_the_layers_keep_between_steps():
    _, mdl = build(CONFIGS["B"][0])
    needs = mdl.cache_needs()
    assert (needs[0].kind, needs[0].num_kv_heads, needs[0].head_dim, needs[0].value_dim, needs[0].window) == ("paged", 1, 64, 0, None)
    assert needs[1].kind == "state" and needs[1].state_shape == (2, 32, 64) and needs[1].state_dtype == "float32"
    _, mdl = build(CONFIGS["D"][0])
    assert all(n.kind == "state" for n in mdl.cache_needs()) and len(mdl.cache_needs()) == 6


def test_a_layer_without_feed_forward_and_files_that_leave_things_out():
    raw = model(40, 16, [layer("retention", retain(2, 4, 3, (0.5, 0.9)), None)])
    _, mdl = build(raw)
    names = {s.name for _, spec in mdl.named_params() for s in spec.sources if not spec.optional}
    assert not [n for n in names if "mlp" in n or "norm2" in n] and "l0.norm1b" in names
    raw["layers"][0]["mixer"].pop("rot")                       # no rotation
    assert build(raw)[0].layers[0].mixer.rot.dims == 0
    raw = model(40, 16, [layer("latent", latent(2, 4, 6, 3, 5, 7), moe(8, 4, 2))])
    names = {s.name for _, spec in build(raw)[1].named_params() for s in spec.sources}
    assert "l0.mlp.router.b" in names and "l0.mix.sink" in names and not [n for n in names if "shared" in n]


@pytest.mark.parametrize("dims, base, scaling", [(64, 10000.0, yarn(4.0, 4096, 32.0, 1.0)), (32, 500.0, yarn(2.0, 64, 8.0, 2.0)),
                                                 (2, 100.0, yarn(3.0, 50, 4.0, 1.0)), (16, 1e6, None), (24, 10000.0, yarn(1.0, 100, 9.0, 9.0)),
                                                 (16, 10000.0, yarn(4.0, 1e9, 1.0, 1e-6)), (16, 10000.0, yarn(4.0, 2, 32.0, 8.0))])
def test_rotation_frequencies(dims, base, scaling):
    from prism_b200.parts.positions import YarnRotaryEmbedding
    part = YarnRotaryEmbedding(dims, base, scaling)
    ref, amp = LP.frequencies(dict(dims=dims, base=base, scaling=scaling))
    got = part.frequencies()
    assert got.dtype == torch.float32 and torch.allclose(got.double(), torch.tensor(ref, dtype=torch.float64), rtol=1e-6, atol=0)
    assert abs(part.amplitude() - amp) < 1e-12
    if scaling is None:
        assert amp == 1.0
    else:
        plain, _ = LP.frequencies(dict(dims=dims, base=base))
        for f, p in zip(ref, plain):                       # between the frequency and a factor-th of it
            assert p / scaling["factor"] * (1 - 1e-12) <= f <= p * (1 + 1e-12)


def test_frequency_scaling_leaves_fast_turns_and_stretches_slow_ones():
    f, amp = LP.frequencies(dict(dims=64, base=10000.0, scaling=yarn(4.0, 4096, 32.0, 1.0)))
    g, _ = LP.frequencies(dict(dims=64, base=10000.0))
    assert f[0] == g[0] and abs(f[-1] - g[-1] / 4.0) < 1e-15 and abs(amp - (0.1 * math.log(4.0) + 1.0)) < 1e-15


def test_plain_prefix_property():
    """The plain model is causal: the logits of a prefix are those of the whole sequence (what lets the GPU tests
    compare any cutting of a prompt with one plain pass)."""
    raw, seed, _ = CONFIGS["A"]
    w = {k: v.double() for k, v in draw_weights(raw, seed).items()}
    seq = torch.randint(0, raw["vocab"], (30,), generator=torch.Generator().manual_seed(1)).tolist()
    full = LP.forward(raw, w, seq)
    assert torch.allclose(LP.forward(raw, w, seq[:17]), full[:17], atol=1e-9)


def test_plain_rotation_pairs():
    x = torch.tensor([[[1.0, 2.0, 3.0, 4.0, 9.0]]] * 3, dtype=torch.float64)
    rot = dict(dims=4, base=100.0)
    y = LP.rotate(x, rot, True)[2, 0]
    c, s = math.cos(2.0), math.sin(2.0)
    assert abs(float(y[0]) - (c - 2 * s)) < 1e-12 and abs(float(y[1]) - (2 * c + s)) < 1e-12
    z = LP.rotate(x, rot, False)[2, 0]
    assert abs(float(z[0]) - (c - 3 * s)) < 1e-12 and abs(float(z[2]) - (3 * c + s)) < 1e-12
    assert float(y[4]) == float(z[4]) == 9.0


def test_plain_retention_against_its_closed_form():
    g = torch.Generator().manual_seed(3)
    q, k, v = (torch.randn(9, n, generator=g).double() for n in (4, 4, 3))
    o = LP.retain(q, k, v, 0.8)
    ref = torch.stack([sum(0.8 ** (i - j) * (q[i] @ k[j]) * v[j] for j in range(i + 1)) for i in range(9)])
    assert torch.allclose(o, ref, atol=1e-12)
    assert torch.allclose(LP.retain(q, k, v, 0.0), (q * k).sum(1, keepdim=True) * v, atol=1e-12)


def test_plain_sink_takes_its_share_once():
    s = torch.tensor([[0.3, -1.0, -math.inf]], dtype=torch.float64)
    p = LP.sink_softmax(s, torch.tensor(0.7, dtype=torch.float64))
    den = math.exp(0.3) + math.exp(-1.0) + math.exp(0.7)
    assert abs(float(p[0, 0]) - math.exp(0.3) / den) < 1e-12 and abs(float(p.sum()) - (1 - math.exp(0.7) / den)) < 1e-12
    assert float(p[0, 2]) == 0.0


def test_plain_clamped_feed_forward_and_routing():
    eye = torch.eye(3, dtype=torch.float64)
    w = {"gate": eye, "up": eye, "down": eye}
    y = LP.dense_ff(torch.tensor([[5.0, -5.0, 0.5]], dtype=torch.float64), w, "", 2.0)[0]
    sg = lambda z: 1.0 / (1.0 + math.exp(-z))
    assert abs(float(y[0]) - 2.0 * sg(1.702 * 2.0) * 3.0) < 1e-12            # both limited from above
    assert abs(float(y[1]) - (-5.0) * sg(-1.702 * 5.0) * (-1.0)) < 1e-12     # the gate not from below, the other one is
    assert abs(float(y[2]) - 0.5 * sg(1.702 * 0.5) * 1.5) < 1e-12
    chosen, weights = LP.route(torch.tensor([1.0, 3.0, 2.0, 3.0]).double(), 3)
    assert chosen == [1, 3, 2] and abs(float(weights.sum()) - 1.0) < 1e-12
    assert abs(float(weights[2]) - math.exp(-1.0) / (2.0 + math.exp(-1.0))) < 1e-12


def test_random_weights_mode_writes_every_tensor(tmp_path):
    from prism_b200.weights.loader import read_safetensors_header
    from prism_b200.weights.random_init import write_model_folder
    from safetensors.torch import load_file
    write_model_folder(copy.deepcopy(CONFIGS["A"][0]), 3, str(tmp_path))
    header = read_safetensors_header(str(tmp_path / "model.safetensors"))
    w = draw_weights(CONFIGS["A"][0], 1)
    assert {k: v[0] for k, v in header.items()} == {k: tuple(v.shape) for k, v in w.items()}
    t = load_file(str(tmp_path / "model.safetensors"))
    assert abs(float(t["l0.norm1"].float().mean())) < 0.1                     # stored around zero
    assert abs(float(t["l0.mix.dq.norm"].float().mean()) - 1.0) < 0.1         # stored around one


def test_k_shares_of_paired_products_and_experts():
    from prism_b200 import ops
    assert ops.tc_ksplit_paired(5376, 2048, sms=148, M=8) == 3                # 42 tiles: three CTAs each
    assert ops.tc_ksplit_paired(18944, 3584, sms=148, M=8) == 1               # 148 tiles fill the GPU
    assert ops.tc_ksplit_paired(64, 128, sms=148, M=8) == 1                   # two blocks of k are not shared
    assert ops.tc_ksplit_paired(5376, 2048, sms=148, M=17) == 1
    for N in (1, 128, 300, 5000):
        for K in (8, 512, 4096):
            assert 1 <= ops.tc_ksplit_paired(N, K, sms=148, M=1) * -(-N // 128) <= max(148, -(-N // 128))


def test_powers_of_a_decay():
    from prism_b200 import ops
    p = ops.decay_powers(torch.tensor([0.0, 0.5, 1.0, 0.99951171875]))
    assert p.shape == (4, ops.DECAY_CHUNK + 1) and p.dtype == torch.float32
    assert p[0].tolist() == [1.0] + [0.0] * ops.DECAY_CHUNK and float(p[1, 3]) == 0.125 and float(p[2].min()) == 1.0
    assert abs(float(p[3, 64]) - 0.99951171875 ** 64) < 1e-7
