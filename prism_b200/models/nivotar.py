"""Nivotar: a small decoder whose ``config.json`` lists its layers one by one.
Its typed configuration, its layer plan and its entry in the architecture
registry; everything this engine knows about the design by name is here.

The design, as this file builds it from the parts:

* embedding rows as they are; the table is the head as well;
* every layer is an *outnorm* block: each sublayer reads the residual stream
  itself, and its result is RMS-normed (``norm1`` for the mixer, ``norm2`` for
  the feed-forward, which may be absent) before it is added;
* mixer ``parallel``: two mixers side by side on the same input, their results
  scaled by constants and added (``parts/recurrent.py: sum``).  Left: windowed
  grouped-query attention, q and k RMS-normed over the whole projection,
  rotated in halves, an explicit score scale (``parts/attention.py``).  Right:
  a state-space mixer (``parts/recurrent.py: state_space``);
* mixer ``lightning``: linear attention behind silu with a fixed decay per
  head from the configuration, one norm over all heads, a sigmoid gate;
* mixer ``gla``: linear attention with a decay per key channel from a low-rank
  product, a norm per head, a silu gate (``gated_linear``);
* feed-forward ``dense``: silu-gated with biases on all projections; ``moe``:
  the softmax over all experts, a correction on the scores for the choice
  only, the ``top`` best chosen, their scores as weights without a
  renormalisation, limited gated experts, and at the end of the list identity
  experts that return the layer's input;
* the final norm (``final.norm``).

The rank of a ``gla`` mixer's decay is the shape of ``a1`` in the model file
(``decay_rank`` in the mixer's configuration where there is no file).  The
design puts no limit on positions; block tables need a width, so
``max_positions`` (an engine knob, default 131072) may be given in the file.
"""

from __future__ import annotations

from dataclasses import dataclass
from typing import Optional, Tuple

from ..config.model_config import ConfigError
from ..model_registry import register_architecture
from ..parts.base import PartSpec
from .decoder import ModelSpec

ARCHITECTURE = "Nivotar"
DEFAULT_MAX_POSITIONS = 131072


def _need(d, key: str, where: str):
    if not isinstance(d, dict) or key not in d or d[key] is None:
        raise ConfigError(f"config.json: {where} has no '{key}'")
    return d[key]


def _pos_int(d, key: str, where: str) -> int:
    v = int(_need(d, key, where))
    if v < 1:
        raise ConfigError(f"config.json: {where}.{key} must be positive, got {v}")
    return v


def _divides(part: int, whole: int, what: str, of: str, where: str):
    if whole % part:
        raise ConfigError(f"config.json: {where}: {of} ({whole}) not divisible by {what} ({part})")


@dataclass(frozen=True)
class WindowAttentionConfig:
    heads: int
    kv_heads: int
    dim: int
    vdim: int
    scale: float
    window: Optional[int]         # None: every key before the query
    rot_dims: int
    rot_base: float


@dataclass(frozen=True)
class StateSpaceConfig:
    heads: int
    vdim: int
    state: int
    groups: int
    conv: int
    norm_groups: int


@dataclass(frozen=True)
class ParallelConfig:
    left: WindowAttentionConfig
    right: StateSpaceConfig
    left_scale: float
    right_scale: float


@dataclass(frozen=True)
class LightningConfig:
    heads: int
    dim: int
    vdim: int
    decay: Tuple[float, ...]      # one per head


@dataclass(frozen=True)
class GLAConfig:
    heads: int
    dim: int
    vdim: int
    tau: float
    decay_rank: int


@dataclass(frozen=True)
class DenseConfig:
    ff: int


@dataclass(frozen=True)
class RoutedConfig:
    ff: int
    limit: float
    experts: int
    identity: int
    top: int


@dataclass(frozen=True)
class NivotarLayer:
    type: str                     # "parallel" | "lightning" | "gla"
    mixer: object
    mlp: object                   # DenseConfig, RoutedConfig or None


def _left(mx, where: str) -> WindowAttentionConfig:
    heads, dim = _pos_int(mx, "heads", where), _pos_int(mx, "dim", where)
    kvh = int(mx.get("kv_heads") or heads)
    if kvh < 1:
        raise ConfigError(f"config.json: {where}.kv_heads must be positive, got {kvh}")
    _divides(kvh, heads, "kv_heads", "heads", where)
    rot = mx.get("rot") or {}
    dims = int(rot.get("dims", dim) or 0) if rot else 0
    if dims % 2 or not 0 <= dims <= dim:
        raise ConfigError(f"config.json: {where}.rot.dims = {dims}: must be even and at most dim ({dim})")
    base = float(_need(rot, "base", where + ".rot")) if dims else 1.0
    if not base > 0:
        raise ConfigError(f"config.json: {where}.rot.base must be positive, got {base}")
    mask = mx.get("mask") or {}
    window = _pos_int(mask, "size", where + ".mask") if mask else None
    return WindowAttentionConfig(heads, kvh, dim, int(mx.get("vdim") or dim), float(_need(mx, "scale", where)), window, dims, base)


def _right(mx, where: str) -> StateSpaceConfig:
    c = StateSpaceConfig(*(_pos_int(mx, k, where) for k in ("heads", "vdim", "state", "groups", "conv", "norm_groups")))
    _divides(c.groups, c.heads, "groups", "heads", where)
    _divides(c.norm_groups, c.heads * c.vdim, "norm_groups", "heads * vdim", where)
    return c


def _mixer(kind: str, mx, where: str, prefix: str, shapes):
    if kind == "parallel":
        return ParallelConfig(_left(_need(mx, "left", where), where + ".left"), _right(_need(mx, "right", where), where + ".right"),
                              float(_need(mx, "left_scale", where)), float(_need(mx, "right_scale", where)))
    if kind not in ("lightning", "gla"):
        raise ConfigError(f"config.json: {where}: type {kind!r}: this design has 'parallel', 'lightning' and 'gla' mixers")
    heads, dim = _pos_int(mx, "heads", where), _pos_int(mx, "dim", where)
    vdim = int(mx.get("vdim") or dim)
    if kind == "lightning":
        decay = tuple(float(d) for d in _need(mx, "decay", where))
        if len(decay) != heads:
            raise ConfigError(f"config.json: {where}.decay has {len(decay)} entries for {heads} heads")
        return LightningConfig(heads, dim, vdim, decay)
    tau = float(_need(mx, "tau", where))
    if not tau > 0:
        raise ConfigError(f"config.json: {where}.tau must be positive, got {tau}")
    rank = mx.get("decay_rank")
    if shapes is not None:
        shape = shapes.get(prefix + "mix.a1")
        if shape is None or len(shape) != 2:
            raise ConfigError(f"the model file has no matrix '{prefix}mix.a1', whose rows are the decay's rank")
        rank = shape[0]
    if rank is None:
        raise ConfigError(f"config.json: {where} has no 'decay_rank' (without a model file nothing else gives it)")
    return GLAConfig(heads, dim, vdim, tau, int(rank))


def _mlp(mlp, where: str):
    if mlp is None:
        return None
    kind = mlp.get("kind", "dense")
    if kind == "dense":
        return DenseConfig(_pos_int(mlp, "ff", where))
    if kind != "moe":
        raise ConfigError(f"config.json: {where}.kind = {kind!r}: this design has 'dense' and 'moe' feed-forwards")
    router, expert = _need(mlp, "router", where), _need(mlp, "expert", where)
    rw, ew = where + ".router", where + ".expert"
    experts, top, identity = _pos_int(router, "experts", rw), _pos_int(router, "top", rw), int(router.get("identity") or 0)
    if identity < 0:
        raise ConfigError(f"config.json: {rw}.identity must not be negative, got {identity}")
    if top > experts + identity:
        raise ConfigError(f"config.json: {rw}: top ({top}) exceeds experts and identity experts ({experts + identity})")
    limit = float(_need(expert, "limit", ew))
    if not limit > 0:
        raise ConfigError(f"config.json: {ew}.limit must be positive, got {limit}")
    return RoutedConfig(_pos_int(expert, "ff", ew), limit, experts, identity, top)


@dataclass(frozen=True)
class NivotarConfig:
    vocab: int
    width: int
    eps: float
    layers: Tuple[NivotarLayer, ...]
    max_positions: int = DEFAULT_MAX_POSITIONS
    eos_token_id: Tuple[int, ...] = ()

    @classmethod
    def from_dict(cls, raw: dict, tensor_shapes: Optional[dict] = None) -> "NivotarConfig":
        vocab, width = _pos_int(raw, "vocab", "the model"), _pos_int(raw, "width", "the model")
        eps = float(_need(_need(raw, "norm", "the model"), "eps", "norm"))
        layers_raw = _need(raw, "layers", "the model")
        if not isinstance(layers_raw, list) or not layers_raw:
            raise ConfigError("config.json: 'layers' must be a list with at least one layer")
        layers = []
        for i, lr in enumerate(layers_raw):
            where = f"layers[{i}]"
            kind, mx = _need(lr, "type", where), _need(lr, "mixer", where)
            layers.append(NivotarLayer(kind, _mixer(kind, mx, where + ".mixer", f"l{i}.", tensor_shapes),
                                       _mlp(lr.get("mlp"), where + ".mlp")))
        eos = raw.get("eos_token_id")
        eos = () if eos is None else tuple(int(e) for e in (eos if isinstance(eos, (list, tuple)) else [eos]))
        return cls(vocab, width, eps, tuple(layers), int(raw.get("max_positions") or DEFAULT_MAX_POSITIONS), eos)


def nivotar_spec(cfg: NivotarConfig) -> ModelSpec:
    W = cfg.width
    norm = lambda tensor, prefix, **kw: PartSpec("rmsnorm", dict(width=W, eps=cfg.eps, tensor=tensor, **kw), prefix=prefix)
    layers = []
    for i, layer in enumerate(cfg.layers):
        p, m = f"l{i}.", layer.mixer
        if layer.type == "parallel":
            a, s = m.left, m.right
            left = PartSpec("gqa_attention", dict(
                hidden_size=W, num_heads=a.heads, num_kv_heads=a.kv_heads, head_dim=a.dim, v_head_dim=a.vdim, qkv_bias=False,
                o_bias=False, scale=a.scale, window=a.window, qk_norm_eps=cfg.eps, qk_norm_whole=True,
                position=None if not a.rot_dims else PartSpec("rotary_yarn", dict(rotary_dim=a.rot_dims, theta=a.rot_base,
                                                                                  interleaved=False)),
                names=dict(q="q", k="k", v="v", o="o", q_norm="q.norm", k_norm="k.norm")), prefix=p + "mix.left.")
            right = PartSpec("state_space", dict(hidden_size=W, num_heads=s.heads, v_head_dim=s.vdim, state=s.state, groups=s.groups,
                                                 conv=s.conv, norm_groups=s.norm_groups, eps=cfg.eps), prefix=p + "mix.right.")
            mixer = PartSpec("sum", dict(mixers=[left, right], scales=[m.left_scale, m.right_scale]))
        elif layer.type == "lightning":
            mixer = PartSpec("lightning", dict(hidden_size=W, num_heads=m.heads, head_dim=m.dim, v_head_dim=m.vdim, decay=m.decay,
                                               eps=cfg.eps), prefix=p + "mix.")
        else:
            mixer = PartSpec("gated_linear", dict(hidden_size=W, num_heads=m.heads, head_dim=m.dim, v_head_dim=m.vdim,
                                                  decay_rank=m.decay_rank, tau=m.tau, eps=cfg.eps), prefix=p + "mix.")
        ff = None
        if isinstance(layer.mlp, DenseConfig):
            ff = PartSpec("swiglu", dict(hidden_size=W, intermediate_size=layer.mlp.ff, names=("gate", "up", "down"),
                                         biases=("gate.b", "up.b", "down.b")), prefix=p + "mlp.")
        elif isinstance(layer.mlp, RoutedConfig):
            r = layer.mlp
            ff = PartSpec("moe", dict(hidden_size=W, intermediate_size=r.ff, experts=r.experts, top=r.top, softmax=True,
                                      scale_input=False, activation="clamped", limit=r.limit, correction="correction",
                                      identity=r.identity), prefix=p + "mlp.")
        layers.append(PartSpec("outnorm", dict(mixer=mixer, mixer_post=norm("norm1", p), feed_forward=ff,
                                               ff_post=norm("norm2", p, **({} if ff is not None else dict(optional=True)))), prefix=p))
    return ModelSpec(
        architecture=ARCHITECTURE, hidden_size=W, vocab_size=cfg.vocab, max_positions=cfg.max_positions,
        embedding=PartSpec("token", dict(vocab_size=cfg.vocab, hidden_size=W, tensor="embed")),
        layers=layers, final_norm=norm("norm", "final."),
        head=PartSpec("linear", dict(vocab_size=cfg.vocab, hidden_size=W, tied_to="embedding.weight", tensor="head")),
        eos_token_id=cfg.eos_token_id)


register_architecture(ARCHITECTURE, NivotarConfig.from_dict, nivotar_spec, sizes_from_tensors=True)
