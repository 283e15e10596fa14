"""Interfaces of the parts a decoder is put together from, and the registry
that maps a part's kind (a string in the layer plan) to its class.

andre-fu/prism writes the whole forward pass inline, three times over
(engine/executor.py:77-130, 132-162, 239-270).  Here each piece of that
loop is a part with its sizes and constants as constructor parameters:

====================  =========================================================
category              interface (see the class of that name below)
====================  =========================================================
``norm``              ``forward(ctx, residual, delta, rows=None) -> normed``
``position``          ``rotary() -> RotaryParams | None`` and ``apply(ctx, q, k)``
``mixer``             ``cache_need()``, ``forward(ctx, x, cache) -> delta``
``feed_forward``      ``forward(ctx, x) -> delta``
``block``             ``forward(ctx, residual, delta, cache) -> (residual, delta)``
``embedding``         ``forward(ctx) -> residual``
``head``              ``forward(ctx, normed_rows) -> float32 logits``
====================  =========================================================

A part never learns which model it is in: the architecture gives it a name
prefix for its tensors and nothing else.
"""

from __future__ import annotations

from dataclasses import dataclass, field
from typing import Callable, Dict, List, Optional, Tuple


# --------------------------------------------------------------------------
# weights a part asks for
# --------------------------------------------------------------------------

@dataclass(frozen=True)
class WeightSource:
    """One tensor of the model file: its name relative to the part's prefix,
    its shape, and how random-weights mode draws it
    (``matrix`` | ``bias`` | ``norm`` | ``eye``: a square matrix near the identity).  ``absolute``: the name is the file's
    full name already (a tensor that another part has handed over)."""
    name: str
    shape: Tuple[int, ...]
    init: str = "matrix"
    absolute: bool = False


@dataclass(frozen=True)
class ParamSpec:
    """One parameter of a part as the kernels see it: the file tensors in
    ``sources`` stacked along dim 0 (the fused qkv and gate_up buffers of
    engine/weight_pool.py:169-182,194-197), or with ``axis=1`` side by side
    along dim 1 (projections whose results are added: one product over the
    joined inputs).  ``optional``: all sources may be
    absent together, and then ``absent`` says what the part gets: ``"zeros"``
    or ``"none"``.  ``alias_of`` names another parameter (qualified) whose
    storage is shared when every source is absent (a tied head)."""
    name: str
    sources: Tuple[WeightSource, ...]
    optional: bool = False
    absent: str = "none"
    alias_of: Optional[str] = None
    axis: int = 0

    @property
    def shape(self) -> Tuple[int, ...]:
        first = self.sources[0].shape
        if self.axis == 1:
            return (first[0], sum(s.shape[1] for s in self.sources)) + tuple(first[2:])
        return (sum(s.shape[0] for s in self.sources),) + tuple(first[1:])


# --------------------------------------------------------------------------
# what a mixer needs from the cache manager
# --------------------------------------------------------------------------

@dataclass(frozen=True)
class CacheNeed:
    """``paged``: keys and values of ``num_kv_heads x head_dim`` per token in
    pages; ``window`` None keeps every key, an integer keeps the last
    ``window`` positions (older pages are given back); ``chunk``: queries see
    only the keys of their own block of ``chunk`` positions (counted from 0),
    so the pages of earlier blocks are given back.  ``v_head_dim``: size of a
    value when it differs from a key's (None: the same; 0: no value plane at
    all, the values are read out of the key rows).  ``keep_first``: under a
    window, the first ``keep_first`` positions stay visible to every later
    query, so the pages that hold them are never given back.  ``state``: one
    tensor of ``state_shape`` per request, in a slot.  ``none``: nothing.

    A mixer that needs several of these (pages for its attention half and
    state for its recurrent half, or two state tensors of different shapes)
    lists them in ``Mixer.cache_needs()`` and gets one view for each."""
    kind: str = "none"
    num_kv_heads: int = 0
    head_dim: int = 0
    window: Optional[int] = None
    state_shape: Tuple[int, ...] = ()
    state_dtype: str = "float32"
    v_head_dim: Optional[int] = None
    chunk: Optional[int] = None
    keep_first: int = 0

    @property
    def value_dim(self) -> int:
        return self.head_dim if self.v_head_dim is None else int(self.v_head_dim)

    def first_kept(self, length: int) -> int:
        """The first position that the query at position ``length`` (the next one of a request holding
        ``length`` tokens) can still see, the kept first positions aside; the pages wholly before it (and
        wholly after the kept positions) may be given back."""
        lo = 0
        if self.window is not None:
            lo = max(lo, length - self.window + 1)
        if self.chunk is not None:
            lo = max(lo, length // self.chunk * self.chunk)
        return lo

    def group_key(self):
        return (self.kind, self.num_kv_heads, self.head_dim, self.window,
                tuple(self.state_shape), self.state_dtype, self.value_dim, self.chunk, self.keep_first)


@dataclass
class RotaryParams:
    """What the fused rotate-and-store kernel needs of a position encoding:
    a float32 table of ``rotary_dim/2`` inverse frequencies on the device."""
    inv_freq: object          # torch.Tensor [rotary_dim // 2] float32
    rotary_dim: int
    interleaved: bool = False # pairs (2i, 2i + 1) instead of (i, i + rotary_dim / 2)
    amplitude: float = 1.0    # a factor on cosine and sine


@dataclass
class StreamUpdate:
    """A sublayer's result that a block with several residual streams has left open: ``delta`` (``[T, W]`` or a stack
    of partial sums) together with the weights that spread it over the streams, ``x_j <- sum_i mix[i, j] x_i +
    out[j] delta``.  The next norm carries the update out in the launch that reads the streams anyway."""
    delta: object
    mix: object
    out: object


@dataclass
class NormedDelta:
    """A sublayer's result that is normed before it joins the residual stream, left open: ``x <- x + rmsnorm(delta) *
    weight`` (``delta``: ``[T, W]`` or a stack of partial sums).  The next norm carries it out in its own launch."""
    delta: object
    weight: object
    eps: float

    def carry_out(self, residual, copy):
        """The sum alone, in place on the float32 rows; ``copy`` (None: not wanted) receives the new rows in its dtype."""
        from .. import ops
        ops.add_normed_rmsnorm(residual, self.delta, self.weight, self.eps, None, 0.0, copy)


@dataclass(frozen=True)
class DetachedProjection:
    """A projection that a part hands to the block around it: its weight's file tensors (names relative to
    the block's prefix; several are stacked along dim 0), their biases if any, and its width - the columns
    it reads (an output projection) or the rows it produces (an input projection).  ``float32``: the part
    reads its input projection's result in float32 (it feeds norms, gates or a recurrence)."""
    weights: Tuple[WeightSource, ...]
    biases: Tuple[WeightSource, ...]
    width: int
    float32: bool = False


# --------------------------------------------------------------------------
# part base classes
# --------------------------------------------------------------------------

@dataclass
class PartSpec:
    """One entry of a layer plan: which kind of part, its constructor
    arguments (sizes and constants, nested ``PartSpec`` for sub-parts), and the
    prefix of its tensors' names in the model file."""
    kind: str
    args: dict = field(default_factory=dict)
    prefix: str = ""


class Part:
    """Common life cycle: constructed from the layer plan's arguments, asked
    for its ``params()`` (own) and ``children`` (sub-parts), then ``bind``
    receives one device tensor per own parameter (None for an absent optional
    one) and is called on the children in turn."""

    category = ""
    prefix = ""

    @property
    def children(self) -> Dict[str, "Part"]:
        return getattr(self, "_children", {})

    def add_child(self, name: str, part: "Part") -> "Part":
        if not hasattr(self, "_children"):
            self._children = {}
        self._children[name] = part
        return part

    def params(self) -> List[ParamSpec]:
        return []

    def named_params(self, path: str = ""):
        """Yield ``(qualified name, ParamSpec with absolute tensor names)`` for
        this part and everything below it."""
        for p in self.params():
            srcs = tuple(WeightSource(s.name if s.absolute else self.prefix + s.name, s.shape, s.init, True)
                         for s in p.sources)
            yield path + p.name, ParamSpec(p.name, srcs, p.optional, p.absent, p.alias_of, p.axis)
        for cname, child in self.children.items():
            yield from child.named_params(f"{path}{cname}.")

    def bind(self, tensors: Dict[str, object], device, dtype, path: str = "") -> None:
        """``tensors`` maps qualified names to device tensors."""
        self.device = device
        self.dtype = dtype
        self.w = {p.name: tensors.get(path + p.name) for p in self.params()}
        for cname, child in self.children.items():
            child.bind(tensors, device, dtype, f"{path}{cname}.")
        self.on_bound()

    def on_bound(self) -> None:
        """Hook: create device buffers that are not weights (tables, scratch)."""

    def handed_over(self, *sources: WeightSource) -> Tuple[WeightSource, ...]:
        """Own file tensors under their full names, for a ``DetachedProjection``."""
        return tuple(WeightSource(s.name if s.absolute else self.prefix + s.name, s.shape, s.init, True) for s in sources)

    def walk(self):
        """This part and every part below it."""
        yield self
        for child in self.children.values():
            yield from child.walk()


class Norm(Part):
    category = "norm"

    def forward(self, ctx, residual, delta, rows=None):
        """``residual += delta`` (float32, in place; ``delta`` may be None or a
        stack of split partial sums) and return the normed rows in the compute
        dtype.  ``rows``: device int32 indices of the rows wanted (all if None)."""
        raise NotImplementedError


class PositionEncoding(Part):
    category = "position"

    def rotary(self) -> Optional[RotaryParams]:
        """Parameters for the fused rotate-and-store kernel, or None when this
        encoding is not a rotary one (then ``apply`` is called instead)."""
        return None

    def apply(self, ctx, q, k) -> None:
        """Encode positions into ``q [T, nh, hd]`` and ``k [T, nkv, hd]`` in place."""
        raise NotImplementedError


class Mixer(Part):
    category = "mixer"
    detachable_out = False      # whether detach_out_projection / detach_in_projection hand anything over
    detachable_in = False
    # Whether a pure-decode step with this mixer may be replayed from a captured CUDA graph.  Inside a
    # graph there is no host copy of the step (``ctx.host`` and ``StateCacheView.host_slots`` are None)
    # and every value must come from device arrays.  None: yes unless the mixer keeps per-request state
    # (``cache_need().kind == "state"``); a state mixer that works from ``cache.slots`` alone sets True.
    graph_safe: Optional[bool] = None
    # True: ``forward`` wants the float32 residual rows themselves as ``x`` where the block has them (a block
    # whose residual stream is normed), not their copy in the compute dtype.
    reads_float32 = False

    def cache_need(self) -> CacheNeed:
        return CacheNeed()

    def cache_needs(self) -> Tuple[CacheNeed, ...]:
        """Everything this mixer keeps between steps.  The default is the single ``cache_need()`` (or
        nothing); a mixer with several needs overrides this, and ``forward`` then gets a tuple of views in
        the same order instead of one view."""
        need = self.cache_need()
        return () if need.kind == "none" else (need,)

    def forward(self, ctx, x, cache):
        """``x [T, H]`` normed rows -> ``delta [T, H]`` (or split partial sums
        ``[k, T, H]`` float32) to be added to the residual stream.  ``cache`` is
        the view of this layer's cache plane for this step (``None`` if the
        mixer needs none; a tuple of views if ``cache_needs()`` lists several)."""
        raise NotImplementedError

    # A block that adds the results of several sublayers may take over their last projections and run them
    # as one product over the joined inputs (see ``parts/blocks.py``), and likewise their first projections
    # of the same input.  A part that can hand them over implements these; the default is that it cannot.
    def detach_out_projection(self) -> Optional["DetachedProjection"]:
        """Give up the output projection: from now on ``params()`` leaves it out and ``forward_inner`` is
        called instead of ``forward``.  None: this part keeps it."""
        return None

    def detach_in_projection(self) -> Optional["DetachedProjection"]:
        """Give up the first projection of the layer's input (only after ``detach_out_projection``):
        ``forward_inner`` then gets its columns of the joint product as ``proj``."""
        return None

    def forward_inner(self, ctx, x, cache, out, proj=None) -> None:
        """The sublayer up to its output projection, written into ``out [T, inner]`` (a view whose rows may
        have a stride of their own)."""
        raise NotImplementedError


class FeedForward(Part):
    category = "feed_forward"
    detachable_out = False
    detachable_in = False
    # True: ``forward`` takes the float32 rows that ``x`` is the copy of as well (``rows32``), where the block has them
    reads_float32_too = False

    def forward(self, ctx, x):
        raise NotImplementedError

    def detach_out_projection(self) -> Optional["DetachedProjection"]:
        return None

    def detach_in_projection(self) -> Optional["DetachedProjection"]:
        return None

    def forward_inner(self, ctx, x, out, proj=None) -> None:
        raise NotImplementedError


class Block(Part):
    """Arrangement of a mixer, a feed-forward and their norms."""
    category = "block"

    def cache_need(self) -> CacheNeed:
        return self.mixer.cache_need()

    def cache_needs(self) -> Tuple[CacheNeed, ...]:
        return self.mixer.cache_needs()

    def forward(self, ctx, residual, delta, cache):
        raise NotImplementedError


class Embedding(Part):
    category = "embedding"

    def forward(self, ctx):
        raise NotImplementedError


class Head(Part):
    category = "head"

    def forward(self, ctx, normed_rows):
        raise NotImplementedError


# --------------------------------------------------------------------------
# registry of part kinds
# --------------------------------------------------------------------------

_PARTS: Dict[Tuple[str, str], Callable] = {}

CATEGORIES = ("norm", "position", "mixer", "feed_forward", "block", "embedding", "head")


def register_part(category: str, kind: str):
    """Class decorator: ``@register_part("mixer", "gqa_attention")``."""
    if category not in CATEGORIES:
        raise ValueError(f"unknown part category {category!r}; one of {CATEGORIES}")

    def deco(cls):
        _PARTS[(category, kind)] = cls
        return cls
    return deco


def part_class(category: str, kind: str):
    try:
        return _PARTS[(category, kind)]
    except KeyError:
        known = sorted(k for (c, k) in _PARTS if c == category)
        raise KeyError(f"no {category} part of kind {kind!r}; registered: {known}") from None


def build_part(category: str, spec: PartSpec) -> Part:
    """Construct the part a ``PartSpec`` names and give it its tensor prefix."""
    part = part_class(category, spec.kind)(**spec.args)
    part.prefix = spec.prefix
    return part


def registered_parts(category: Optional[str] = None):
    return sorted(k for k in _PARTS if category is None or k[0] == category)
