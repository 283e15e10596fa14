"""Nivotar without a GPU: configuration and refusals, tensor names against a drawn model file, what each layer keeps
between steps, sizes that only the model file gives, and properties of the plain mechanisms that the GPU tests lean on."""

import copy
import math

import pytest
import torch

from nivotar_helpers import CONFIGS, NP, dense, draw_weights, gla, layer, left, lightning, model, moe, parallel, right


def build(raw, shapes=None):
    from prism_b200.model_registry import build_model
    return build_model(copy.deepcopy(raw), shapes)


def names_of(mdl, optional=False):
    return {s.name: tuple(s.shape) for _, spec in mdl.named_params() for s in spec.sources if optional or not spec.optional}


def test_the_registry_finds_the_design_and_every_tensor_has_a_taker():
    from prism_b200.model_registry import registered_architectures
    assert "Nivotar" in registered_architectures()
    for name, (raw, seed, _) in CONFIGS.items():
        w = draw_weights(raw, seed)
        assert names_of(build(raw)[1]) == {k: tuple(v.shape) for k, v in w.items()}, name


@pytest.mark.parametrize("edit, text", [
    (lambda r: r.pop("norm"), "norm"),
    (lambda r: r.pop("width"), "width"),
    (lambda r: r.update(layers=[]), "layers"),
    (lambda r: r["layers"][0].update(type="attention"), "parallel"),
    (lambda r: r["layers"][0]["mixer"].pop("right_scale"), "right_scale"),
    (lambda r: r["layers"][0]["mixer"].pop("left"), "left"),
    (lambda r: r["layers"][0]["mixer"]["left"].pop("scale"), "scale"),
    (lambda r: r["layers"][0]["mixer"]["left"].update(kv_heads=2), "kv_heads"),
    (lambda r: r["layers"][0]["mixer"]["left"]["rot"].update(dims=5), "dims"),
    (lambda r: r["layers"][0]["mixer"]["left"]["rot"].update(dims=12), "dims"),
    (lambda r: r["layers"][0]["mixer"]["left"]["rot"].pop("base"), "base"),
    (lambda r: r["layers"][0]["mixer"]["left"]["mask"].update(size=0), "size"),
    (lambda r: r["layers"][0]["mixer"]["right"].update(groups=4), "groups"),
    (lambda r: r["layers"][0]["mixer"]["right"].update(norm_groups=7), "norm_groups"),
    (lambda r: r["layers"][0]["mixer"]["right"].pop("conv"), "conv"),
    (lambda r: r["layers"][1]["mixer"].pop("tau"), "tau"),
    (lambda r: r["layers"][1]["mixer"].update(tau=0.0), "tau"),
    (lambda r: r["layers"][1]["mixer"].pop("decay_rank"), "decay_rank"),
    (lambda r: r["layers"][2]["mixer"].update(decay=[0.5]), "decay"),
    (lambda r: r["layers"][2]["mlp"].pop("ff"), "ff"),
    (lambda r: r["layers"][2]["mlp"].update(kind="glu"), "dense"),
    (lambda r: r["layers"][0]["mlp"]["router"].update(top=8), "top"),
    (lambda r: r["layers"][0]["mlp"]["router"].update(identity=-1), "identity"),
    (lambda r: r["layers"][0]["mlp"]["expert"].pop("limit"), "limit"),
    (lambda r: r["layers"][0]["mlp"]["expert"].update(limit=0.0), "limit"),
])
def test_refusals_name_the_key(edit, text):
    from prism_b200.config.model_config import ConfigError
    raw = copy.deepcopy(CONFIGS["A"][0])
    edit(raw)
    with pytest.raises(ConfigError, match=text):
        build(raw)


def test_the_decays_rank_is_the_model_files():
    from prism_b200.config.model_config import ConfigError
    raw = copy.deepcopy(CONFIGS["A"][0])
    shapes = {k: tuple(v.shape) for k, v in draw_weights(raw, 1).items()}
    raw["layers"][1]["mixer"].pop("decay_rank")
    raw["layers"][4]["mixer"]["decay_rank"] = 9                    # the file's shape wins
    cfg, mdl = build(raw, shapes)
    assert [cfg.layers[i].mixer.decay_rank for i in (1, 4)] == [3, 5]
    assert names_of(mdl) == shapes
    shapes.pop("l4.mix.a1")
    with pytest.raises(ConfigError, match="l4.mix.a1"):
        build(raw, shapes)


def test_what_the_layers_keep_between_steps():
    from prism_b200.cache.manager import plan_groups
    _, mdl = build(CONFIGS["B"][0])
    needs = mdl.cache_needs()
    assert needs[0].kind == "state" and needs[0].state_shape == (2, 32, 64) and needs[0].state_dtype == "float32"
    att, state, tail = needs[1]
    assert (att.kind, att.num_kv_heads, att.head_dim, att.value_dim, att.window) == ("paged", 2, 32, 48, 64)
    assert state.state_shape == (4, 32, 64) and tail.state_shape == (3, 4 * 32 + 2 * 2 * 64)
    assert needs[3][0].window == 150
    groups, where = plan_groups(needs, [None] * len(needs))
    assert sorted(g.kind for g in groups) == ["paged", "paged"] + ["state"] * 6 and len(where) == 4
    assert all(n.kind == "state" for n in build(CONFIGS["D"][0])[1].cache_needs())


def test_files_that_leave_things_out():
    mx = parallel(left(2, 2, 4, 4, 8), right(2, 3, 4, 1, 2, 1))
    raw = model(40, 16, [layer("parallel", mx, None), layer("lightning", lightning(2, 4, 3, (0.5, 0.9)), moe(8, 4, 2))])
    for k in ("mask", "rot", "kv_heads", "vdim"):                   # every key, no rotation, a key head per head, values as keys
        mx["left"].pop(k)
    cfg, mdl = build(raw)
    a = cfg.layers[0].mixer.left
    assert (a.window, a.rot_dims, a.kv_heads, a.vdim) == (None, 0, 2, 4)
    names = names_of(mdl)
    assert not [n for n in names if n.startswith("l0.mlp") or n == "l0.norm2"] and names["l1.mlp.router"] == (4, 16)
    assert "l0.norm2" in names_of(mdl, optional=True)               # may be in the file; nothing reads it
    assert "head" not in names and "head" in names_of(mdl, optional=True)
    assert cfg.layers[1].mlp.identity == 0


def test_plain_prefix_property():
    """The plain model is causal: the logits of a prefix are those of the whole sequence (what lets the GPU tests
    compare any cutting of a prompt with one plain pass)."""
    raw, seed, _ = CONFIGS["A"]
    w = {k: v.double() for k, v in draw_weights(raw, seed).items()}
    seq = torch.randint(0, raw["vocab"], (40,), generator=torch.Generator().manual_seed(1)).tolist()
    full = NP.forward(raw, w, seq)
    assert torch.allclose(NP.forward(raw, w, seq[:17]), full[:17], atol=1e-9)


def test_plain_window_and_rotation():
    see = NP.visible(6, 3)
    assert [see[5, j].item() for j in range(6)] == [False, False, False, True, True, True] and see[0].tolist() == [True] + [False] * 5
    assert NP.visible(4, 1).equal(torch.eye(4, dtype=torch.bool)) and int(NP.visible(4, None).sum()) == 10
    x = torch.tensor([[[1.0, 2.0, 3.0, 4.0, 9.0]]] * 3, dtype=torch.float64)
    y = NP.rotate_halves(x, 4, 100.0)[2, 0]
    assert abs(float(y[0]) - (math.cos(2.0) - 3 * math.sin(2.0))) < 1e-12 and abs(float(y[2]) - (3 * math.cos(2.0) + math.sin(2.0))) < 1e-12
    assert abs(float(y[1]) - (2 * math.cos(0.2) - 4 * math.sin(0.2))) < 1e-12 and float(y[4]) == 9.0


def test_plain_decayed_sum_against_its_closed_form():
    g = torch.Generator().manual_seed(3)
    q, k, v = (torch.randn(9, n, generator=g).double() for n in (4, 4, 3))
    for d in (torch.rand(9, 4, generator=g).double(), torch.rand(9, 1, generator=g).double(), torch.zeros(9, 1).double()):
        o = NP.decayed_sum(q, k, v, d)
        full = d.expand(9, 4)
        ref = torch.stack([sum((q[i] * full[j + 1:i + 1].prod(0) * k[j]).sum() * v[j] for j in range(i + 1)) for i in range(9)])
        assert torch.allclose(o, ref, atol=1e-12)


def test_plain_convolution_and_softplus():
    x = torch.arange(8, dtype=torch.float64).view(4, 2)
    taps, bias = torch.tensor([[1.0, 10.0], [100.0, 0.5]], dtype=torch.float64), torch.tensor([0.25, 0.0], dtype=torch.float64)
    y = NP.short_conv(x, taps, bias)
    assert y[:, 0].tolist() == [0.25, 20.25, 42.25, 64.25] and y[:, 1].tolist() == [0.5, 101.5, 302.5, 503.5]
    z = torch.tensor([-800.0, -3.0, 0.0, 4.0, 800.0], dtype=torch.float64)
    ref = [0.0, math.log1p(math.exp(-3.0)), math.log(2.0), math.log1p(math.exp(4.0)), 800.0]
    assert torch.allclose(NP.softplus(z), torch.tensor(ref, dtype=torch.float64), atol=1e-12)


def test_plain_routing_and_feed_forwards():
    z = torch.tensor([1.0, 3.0, 2.0, 3.0]).double()
    s = torch.softmax(z, -1)
    assert NP.route(z, torch.zeros(4), 3)[0] == [1, 3, 2]
    chosen, weights = NP.route(z, torch.tensor([0.9, 0.0, 0.0, -0.5]), 2)       # the correction moves the choice, not the weights
    assert chosen == [0, 1] and torch.allclose(weights, s[[0, 1]])
    eye = torch.eye(3, dtype=torch.float64)
    w = {"e0.gate": eye, "e0.up": eye, "e0.down": eye, "router": torch.zeros(2, 3).double(), "correction": torch.tensor([0.0, 1.0]).double()}
    h = torch.tensor([[5.0, -5.0, 0.5]], dtype=torch.float64)
    sg = lambda v: 1.0 / (1.0 + math.exp(-v))
    y = NP.clamped_expert(h, w, "e0.", 2.0)[0]
    assert abs(float(y[0]) - 2.0 * sg(3.404) * 3.0) < 1e-12 and abs(float(y[1]) - 5.0 * sg(-1.702 * 5.0)) < 1e-12
    mlp = moe(3, 1, 1, 1, limit=2.0)
    assert torch.allclose(NP.moe_ff(h, w, "", mlp), 0.5 * h)                     # the identity expert, with half the weight
    mlp["router"]["top"] = 2
    assert torch.allclose(NP.moe_ff(h, w, "", mlp), 0.5 * h + 0.5 * y)
    w = {"gate": eye, "up": eye, "down": eye, "gate.b": h[0], "up.b": h[0] * 0 + 1, "down.b": h[0]}
    y = NP.dense_ff(h, w, "")[0]
    assert abs(float(y[0]) - (10.0 * sg(10.0) * 6.0 + 5.0)) < 1e-9


def test_random_weights_mode_writes_every_tensor(tmp_path):
    from prism_b200.weights.loader import read_safetensors_header
    from prism_b200.weights.random_init import write_model_folder
    write_model_folder(copy.deepcopy(CONFIGS["A"][0]), 3, str(tmp_path))
    header = read_safetensors_header(str(tmp_path / "model.safetensors"))
    assert {k: v[0] for k, v in header.items()} == {k: tuple(v.shape) for k, v in draw_weights(CONFIGS["A"][0], 1).items()}


def test_constants_of_the_mixers_are_parameters():
    from prism_b200.config.model_config import ConfigError
    from prism_b200.parts.base import PartSpec, build_part
    with pytest.raises(ConfigError):
        build_part("mixer", PartSpec("state_space", dict(hidden_size=8, num_heads=4, v_head_dim=2, state=3, groups=3, conv=2, norm_groups=1, eps=1e-5)))
    with pytest.raises(ValueError):
        build_part("feed_forward", PartSpec("moe", dict(hidden_size=8, intermediate_size=4, experts=2, top=1, activation="clamped")))
    with pytest.raises(ValueError):
        build_part("feed_forward", PartSpec("moe", dict(hidden_size=8, intermediate_size=4, experts=2, top=1, identity=1)))
    part = build_part("mixer", PartSpec("gated_linear", dict(hidden_size=8, num_heads=2, head_dim=3, v_head_dim=5, decay_rank=4, tau=2.0, eps=1e-5)))
    assert part.cache_need().state_shape == (2, 5, 3) and gla(2, 3, 5, 2.0, 4)["tau"] == part.tau
    assert dense(3)["ff"] == 3
