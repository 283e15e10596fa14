"""Limatar: a small decoder whose ``config.json`` lists its layers one by one.
Its typed configuration, its layer plan and its entry in the architecture
registry; everything this engine knows about the design by name is here.

The design, as this file builds it from the parts:

* embedding rows, normed (``embed.norm``); every norm of the model's width is
  an RMS norm whose weight is stored around zero;
* every layer is a *sandwich* block: a norm before and after each sublayer
  (``norm1`` / ``norm1b`` around the mixer, ``norm2`` / ``norm2b`` around the
  feed-forward, which may be absent);
* ``loop``: layers ``start .. stop - 1`` run ``times`` times in a row with the
  same weights, each pass with a cache and a state of its own;
* mixer ``latent_attention``: queries and keys/values through low-rank latents,
  a rotated key part shared by all heads (interleaved pairs, frequencies under
  YaRN scaling), an explicit score scale, a learned sink per head in the
  softmax's denominator, a sigmoid gate on the concatenated heads
  (``parts/attention.py``); the cache holds the latent and the rotated part;
* mixer ``retention``: linear attention with a fixed decay per head from the
  configuration, rotated in halves, a norm per head and a silu gate
  (``parts/recurrent.py``);
* feed-forward ``dense``: gate and up limited, ``g sigmoid(1.702 g) (u + 1)``;
  ``moe``: the ``top`` largest logits of a router with a bias, weights their
  softmax, gated silu experts, and a shared expert of the same form;
* the final norm (``final.norm``) and the embedding table as the head.

The design puts no limit on positions; block tables need a width, so
``max_positions`` (an engine knob, default 131072) may be given in the file.
"""

from __future__ import annotations

from dataclasses import dataclass
from typing import Optional, Tuple

from ..config.model_config import ConfigError
from ..model_registry import register_architecture
from ..parts.base import PartSpec
from .decoder import ModelSpec, ScheduleEntry

ARCHITECTURE = "Limatar"
DEFAULT_MAX_POSITIONS = 131072
DEFAULT_ROT_BASE = 10000.0


def _need(d, key: str, where: str):
    if not isinstance(d, dict) or key not in d or d[key] is None:
        raise ConfigError(f"config.json: {where} has no '{key}'")
    return d[key]


def _pos_int(d, key: str, where: str) -> int:
    v = int(_need(d, key, where))
    if v < 1:
        raise ConfigError(f"config.json: {where}.{key} must be positive, got {v}")
    return v


@dataclass(frozen=True)
class RotationConfig:
    dims: int                     # entries of a head that turn
    base: float
    scaling: Optional[Tuple[float, float, float, float]]     # factor, original, fast, slow


@dataclass(frozen=True)
class LatentConfig:
    heads: int
    dim: int                      # unrotated query/key size per head
    rot_dim: int                  # rotated part per head
    vdim: int
    q_rank: int
    kv_rank: int
    scale: float
    rot: RotationConfig


@dataclass(frozen=True)
class RetentionConfig:
    heads: int
    dim: int
    vdim: int
    decay: Tuple[float, ...]      # one per head
    rot: RotationConfig


@dataclass(frozen=True)
class DenseConfig:
    ff: int
    limit: float


@dataclass(frozen=True)
class RoutedConfig:
    ff: int
    experts: int
    top: int
    shared_ff: Optional[int]


@dataclass(frozen=True)
class LimatarLayer:
    type: str                     # "latent_attention" | "retention"
    mixer: object
    mlp: object                   # DenseConfig, RoutedConfig or None


def _rotation(mx, width: int, what: str, where: str) -> RotationConfig:
    rot = mx.get("rot") or {}
    dims = int(rot.get("dims", width) or 0) if rot else 0
    if dims % 2 or not 0 <= dims <= width:
        raise ConfigError(f"config.json: {where}.rot.dims = {dims}: must be even and at most {what} ({width})")
    sc = rot.get("scaling")
    scaling = None
    if sc:
        scaling = tuple(float(_need(sc, k, where + ".rot.scaling")) for k in ("factor", "original", "fast", "slow"))
        if min(scaling) <= 0:
            raise ConfigError(f"config.json: {where}.rot.scaling: factor, original, fast and slow must be positive")
    return RotationConfig(dims, float(rot.get("base", DEFAULT_ROT_BASE)), scaling)


def _mixer(kind: str, mx, where: str):
    heads, dim, vdim = _pos_int(mx, "heads", where), _pos_int(mx, "dim", where), int(mx.get("vdim") or mx["dim"])
    if kind == "latent_attention":
        rot_dim = int(mx.get("rot_dim") or 0)
        return LatentConfig(heads, dim, rot_dim, vdim, _pos_int(mx, "q_rank", where), _pos_int(mx, "kv_rank", where),
                            float(_need(mx, "scale", where)), _rotation(mx, rot_dim, "rot_dim", where))
    if kind == "retention":
        decay = tuple(float(d) for d in _need(mx, "decay", where))
        if len(decay) != heads:
            raise ConfigError(f"config.json: {where}.decay has {len(decay)} entries for {heads} heads")
        return RetentionConfig(heads, dim, vdim, decay, _rotation(mx, dim, "dim", where))
    raise ConfigError(f"config.json: {where}: type {kind!r}: this design has 'latent_attention' and 'retention' mixers")


def _mlp(mlp, where: str):
    if mlp is None:
        return None
    kind = mlp.get("kind", "dense")
    if kind == "dense":
        limit = float(_need(mlp, "limit", where))
        if not limit > 0:
            raise ConfigError(f"config.json: {where}.limit must be positive, got {limit}")
        return DenseConfig(_pos_int(mlp, "ff", where), limit)
    if kind != "moe":
        raise ConfigError(f"config.json: {where}.kind = {kind!r}: this design has 'dense' and 'moe' feed-forwards")
    router = _need(mlp, "router", where)
    experts, top = _pos_int(router, "experts", where + ".router"), _pos_int(router, "top", where + ".router")
    if top > experts:
        raise ConfigError(f"config.json: {where}.router: top ({top}) exceeds experts ({experts})")
    shared = mlp.get("shared")
    return RoutedConfig(_pos_int(_need(mlp, "expert", where), "ff", where + ".expert"), experts, top,
                        None if not shared else _pos_int(shared, "ff", where + ".shared"))


@dataclass(frozen=True)
class LimatarConfig:
    vocab: int
    width: int
    eps: float
    layers: Tuple[LimatarLayer, ...]
    loop: Optional[Tuple[int, int, int]] = None     # start, stop, times
    max_positions: int = DEFAULT_MAX_POSITIONS
    eos_token_id: Tuple[int, ...] = ()

    @classmethod
    def from_dict(cls, raw: dict) -> "LimatarConfig":
        vocab, width = _pos_int(raw, "vocab", "the model"), _pos_int(raw, "width", "the model")
        eps = float(_need(_need(raw, "norm", "the model"), "eps", "norm"))
        layers_raw = _need(raw, "layers", "the model")
        if not isinstance(layers_raw, list) or not layers_raw:
            raise ConfigError("config.json: 'layers' must be a list with at least one layer")
        layers = []
        for i, lr in enumerate(layers_raw):
            where = f"layers[{i}]"
            kind, mx = _need(lr, "type", where), _need(lr, "mixer", where)
            layers.append(LimatarLayer(kind, _mixer(kind, mx, where + ".mixer"), _mlp(lr.get("mlp"), where + ".mlp")))
        loop = raw.get("loop")
        if loop:
            start, stop, times = (int(_need(loop, k, "loop")) for k in ("start", "stop", "times"))
            if not 0 <= start <= stop <= len(layers) or times < 1:
                raise ConfigError(f"config.json: loop: layers {start} .. {stop - 1}, {times} times: the model has {len(layers)} "
                                  f"layers, and they run at least once")
            loop = (start, stop, times)
        eos = raw.get("eos_token_id")
        eos = () if eos is None else tuple(int(e) for e in (eos if isinstance(eos, (list, tuple)) else [eos]))
        return cls(vocab, width, eps, tuple(layers), loop or None, int(raw.get("max_positions") or DEFAULT_MAX_POSITIONS), eos)

    def run_order(self) -> list:
        """Indices of the layers in the order they run."""
        order = list(range(len(self.layers)))
        if self.loop is None:
            return order
        start, stop, times = self.loop
        return order[:start] + order[start:stop] * times + order[stop:]


def _rotary(rot: RotationConfig, interleaved: bool) -> Optional[PartSpec]:
    if not rot.dims:
        return None
    return PartSpec("rotary_yarn", dict(
        rotary_dim=rot.dims, theta=rot.base, interleaved=interleaved,
        scaling=None if rot.scaling is None else dict(zip(("factor", "original", "fast", "slow"), rot.scaling))))


def limatar_spec(cfg: LimatarConfig) -> ModelSpec:
    W = cfg.width
    norm = lambda tensor, prefix, **kw: PartSpec("rmsnorm", dict(width=W, eps=cfg.eps, tensor=tensor, centred=True, **kw), prefix=prefix)
    layers = []
    for i, layer in enumerate(cfg.layers):
        p, m = f"l{i}.", layer.mixer
        if layer.type == "latent_attention":
            mixer = PartSpec("latent_attention", dict(
                hidden_size=W, num_heads=m.heads, head_dim=m.dim, rot_dim=m.rot_dim, v_head_dim=m.vdim, q_rank=m.q_rank,
                kv_rank=m.kv_rank, eps=cfg.eps, scale=m.scale, sink=True, gate=True, rope_dims=0, position=_rotary(m.rot, True),
                names=dict(dq="dq", dq_norm="dq.norm", uq="uq", dkv="dkv", dkv_norm="dkv.norm", uk="uk", uv="uv", o="o",
                           sink="sink", g="g")), prefix=p + "mix.")
        else:
            mixer = PartSpec("retention", dict(hidden_size=W, num_heads=m.heads, head_dim=m.dim, v_head_dim=m.vdim,
                                               decay=m.decay, eps=cfg.eps, position=_rotary(m.rot, False)), prefix=p + "mix.")
        ff = None
        if isinstance(layer.mlp, DenseConfig):
            ff = PartSpec("swiglu", dict(hidden_size=W, intermediate_size=layer.mlp.ff, names=("gate", "up", "down"),
                                         activation="clamped", limit=layer.mlp.limit), prefix=p + "mlp.")
        elif isinstance(layer.mlp, RoutedConfig):
            r = layer.mlp
            shared = None if r.shared_ff is None else PartSpec(
                "swiglu", dict(hidden_size=W, intermediate_size=r.shared_ff, names=("gate", "up", "down")), prefix=p + "mlp.shared.")
            # the softmax over the chosen logits is the softmax over all of them, divided by the sum of the chosen
            ff = PartSpec("moe", dict(hidden_size=W, intermediate_size=r.ff, experts=r.experts, top=r.top, softmax=True,
                                      renorm=True, scale_input=False, router_bias="router.b", shared=shared), prefix=p + "mlp.")
        extra = {} if ff is not None else dict(optional=True)
        layers.append(PartSpec("sandwich", dict(mixer=mixer, mixer_norm=norm("norm1", p), mixer_post=norm("norm1b", p),
                                                feed_forward=ff, ff_norm=norm("norm2", p, **extra),
                                                ff_post=norm("norm2b", p, **extra)), prefix=p))
    return ModelSpec(
        architecture=ARCHITECTURE, hidden_size=W, vocab_size=cfg.vocab, max_positions=cfg.max_positions,
        embedding=PartSpec("token", dict(vocab_size=cfg.vocab, hidden_size=W, tensor="embed", norm=norm("norm", "embed."))),
        layers=layers, schedule=[ScheduleEntry(i) for i in cfg.run_order()], final_norm=norm("norm", "final."),
        head=PartSpec("linear", dict(vocab_size=cfg.vocab, hidden_size=W, tied_to="embedding.weight", tensor="head")),
        eos_token_id=cfg.eos_token_id)


register_architecture(ARCHITECTURE, LimatarConfig.from_dict, limatar_spec)
