"""What a model is made of, and the registries that turn a description into it.

A model is described as data (``ModelSpec``): a list of layers, each naming the
kind and the numbers of its mixer, feed-forward, norms and block arrangement,
and a run order (``RunSpec`` list) that may name a layer twice or let a run
read the cache another run writes.  ``build`` functions look the kinds up in
the registries below; parts get their sizes and constants as arguments and
their tensors by name.  No part knows which model it is in.

Interfaces (all tensors are CUDA tensors; T tokens in the step, H width):

``Norm``
    ``apply(resid, delta=None, rows=None) -> normed``: adds ``delta`` into the
    32-bit residual stream ``resid`` [T, H] when given, returns the normed rows
    in the activations' type.  With ``rows`` it norms those rows only and
    leaves ``resid`` unchanged.
``PositionEncoding``
    ``encode_and_store(qkv, geometry, ctx, kv, write)``: encodes the queries
    (in place) and keys of the fused projection rows and, if ``write``, stores
    keys and values in the paged cache ``kv``.  One that cannot work in place
    (a convolution over time reads earlier rows) offers ``encode_rows(qkv,
    geometry, ctx, cache) -> queries`` instead, with ``extra_state_needs()``
    and ``tile_sizes()`` as a mixer has them.
``Mixer``
    ``cache_need() -> KVNeed | None`` and ``state_need() -> StateNeed | None``
    say what the cache manager must hold for it; ``forward(x, ctx, cache) ->
    y`` mixes the tokens of the step (x, y: [T, H] activations) using
    ``cache.kv`` (pages) and/or ``cache.state`` (one row per state slot).
    State: request b of the step owns row ``ctx.state_slots[b]`` of
    ``cache.state``.  Before the step's first layer the framework zeroes the
    rows of requests whose ``ctx.ctx_before[b]`` is 0 (a new request, or one
    recomputed after pre-emption), so a mixer reads its row unconditionally
    and writes it back.  Rows of a step that stand for no request (padding of a
    fixed-shape batch) carry slot -1: a kernel uses the buffer's last row for
    them, which belongs to nobody, or skips them.  Steps of a model whose
    mixers keep state are never padded with dummy tokens behind a request's
    own.  ``tile_sizes()`` names the query-tile sizes its kernels want listed
    in the step's integers (``ctx.tiles``).
``InputFilter``
    ``forward(x, ctx, state) -> x'``: what a block puts between a norm and the
    sub-layer that reads it (a short convolution over time, say); it may keep
    per-request state of its own (``state_need()``), which the block hands it.
    Optional: ``after_norm(norm, resid, delta, ctx, state) -> x' | None`` runs
    the norm before it and itself as one kernel where it can (None: it cannot).
``FeedForward``
    ``forward(x, ctx) -> y``.
``StreamInput``
    ``forward(stream, ctx)``: adds something to the residual stream that
    depends on the step's token ids or on nothing but learned vectors (an
    embedding per layer behind a gate, what a pass over a stretch of layers adds
    before its first layer).  A block may run one after its sub-layers; a
    ``RunSpec`` may name one that runs before its layer.
``Block``
    ``forward(stream, ctx, cache)``: arranges norms, mixer and feed-forward
    around the residual stream (``stream.resid`` 32-bit plus a ``pending``
    delta not yet added).
Every part also has ``tensors() -> list[TensorDecl]`` (what it reads from the
checkpoint, with shapes, for checking and for random weights) and
``bind(get, runtime)`` (takes its tensors, already on the device).

The reference's modules read a shared config object in their constructors
(python/lyapunov_engine/models/llama.py:35-48,110-117,126-134).
"""
from __future__ import annotations

from dataclasses import dataclass, field
from typing import Any, Callable


# ---------------------------------------------------------------- description
@dataclass(frozen=True)
class PartSpec:
    kind: str
    params: dict = field(default_factory=dict)


@dataclass(frozen=True)
class LayerSpec:
    """One layer: a block arrangement over a mixer and a feed-forward.  All
    sizes, constants and tensor names sit in the parts' params."""
    block: PartSpec


@dataclass(frozen=True)
class RunSpec:
    """One entry of the run order: run ``layer``; ``reads_cache_of`` names an
    earlier entry (by its index in the run order) whose cache this run reads
    instead of writing one of its own; ``entry``: a stream input that runs
    right before the layer (what a pass over a stretch of layers adds before its
    first one)."""
    layer: int
    reads_cache_of: int | None = None
    entry: PartSpec | None = None


@dataclass(frozen=True)
class ModelSpec:
    architecture: str
    hidden_size: int
    vocab_size: int
    max_positions: int
    embedding: PartSpec
    layers: tuple[LayerSpec, ...]
    run_order: tuple[RunSpec, ...]
    final_norm: PartSpec
    head: PartSpec
    eos_token_ids: tuple[int, ...] = ()
    bos_token_id: int | None = None
    config_json: dict = field(default_factory=dict, compare=False)


# ---------------------------------------------------------------- tensors
@dataclass(frozen=True)
class TensorDecl:
    """A checkpoint tensor a part reads.  ``role`` decides the type it is kept
    in: "matrix" in the engine's compute type (bfloat16 or float32); "vector"
    (norm weights and the like) always 32-bit, so one stored in 32 bits stays
    exactly so; "int_table" as int32.  ``init`` is how random weights fill it:
    "normal", "ones", "ones_jitter", "zeros", "taps" (small numbers around
    zero), "eye" (the identity matrix) or "share" (1 / count in every entry).  ``alias_of`` names the tensor
    that stands in when the checkpoint has none of this name (a tied head).
    ``std_scale``: random matrices are N(0, std * std_scale)."""
    name: str
    shape: tuple[int, ...]
    role: str = "matrix"
    init: str = "normal"
    alias_of: str | None = None
    std_scale: float = 1.0


@dataclass(frozen=True)
class KVNeed:
    """Keys and values in pages.  ``window`` w: a query reads the last w keys
    only; ``chunk`` c: a query reads the keys of its own chunk of c positions
    only (chunks counted from position 0); neither: every key is kept.
    ``values`` False: one pool serves as keys and as values (a mixer that
    attends over one latent vector per token).  ``keep_first`` n (with a
    window): the keys at positions below n stay visible to every later query,
    so the pages that hold them are never given back while the request lives."""
    num_kv_heads: int
    head_dim: int
    window: int | None = None
    chunk: int | None = None
    values: bool = True
    keep_first: int = 0


@dataclass(frozen=True)
class StateNeed:
    """Per-request state of fixed size: one row of ``shape`` per slot."""
    shape: tuple[int, ...]
    dtype: Any = None  # torch dtype; None: float32


class Part:
    def tensors(self) -> list[TensorDecl]:
        return []

    def bind(self, get: Callable[[str], Any], runtime) -> None:
        pass


class Norm(Part):
    def apply(self, resid, delta=None, rows=None):
        raise NotImplementedError

    def apply_stream(self, stream, read=None, rows=None, workspace=None, key="normed"):
        """The norm of what a sub-layer reads from ``stream`` (a
        ``ResidualStream``), after the pending output has entered it.  A
        stream in one copy with a plain addition pending is what every norm
        takes; a norm that also takes a stream in several copies overrides
        this (``read``: the reading sub-layer's ``StreamLink``; None: the sum
        of the copies).  Without ``rows`` the pending output is consumed."""
        if stream.copies != 1 or stream.update is not None or read is not None:
            raise ValueError(f"{type(self).__name__} reads a residual stream in one copy only")
        out = self.apply(stream.resid, stream.pending, rows=rows, workspace=workspace, key=key)
        if rows is None:
            stream.pending = None
        return out


class PositionEncoding(Part):
    def encode_and_store(self, qkv, geometry, ctx, kv, write: bool) -> None:
        raise NotImplementedError


class Mixer(Part):
    # a bias [H] (32-bit) on the output that forward() leaves to the block that adds the output to the stream (named
    # by ``o_bias_name``; blocks that add none refuse such a mixer)
    o_bias_name: str | None = None
    output_bias = None
    # True: the mixer writes no keys of its own, its runs must read another run's
    reads_only = False

    def cache_need(self) -> KVNeed | None:
        return None

    def state_need(self) -> StateNeed | None:
        return None

    def extra_state_needs(self) -> dict[str, "StateNeed"]:
        """More per-request state than the one buffer of ``state_need()``, by
        names of the mixer's choosing; the block lists them among its own
        (``Block.extra_state_needs()``) and ``cache.extra[name]`` holds each."""
        return {}

    def tile_sizes(self) -> list[int]:
        """Query-tile sizes its kernels want: for each, ``ctx.tiles[size]`` lists
        (request of each tile, first query token of the tile within the
        request, number of tiles, how many of them belong to requests that
        bring several tokens), those of several tokens first."""
        return []

    def decode_variant(self, fill: int, num_decode: int, context_bound: int):
        """What of this mixer's launches depends on how many of a step's
        ``num_decode`` one-token requests are real (``fill``; the others pad
        the step to a fixed shape): any hashable, None if nothing.  Steps of
        fixed shape that are captured once and replayed are kept apart by it;
        ``forward`` finds the same number in ``ctx.decode_fill`` and must make
        the same choice from it."""
        return None

    def forward(self, x, ctx, cache):
        raise NotImplementedError


class InputFilter(Part):
    def state_need(self) -> StateNeed | None:
        return None

    def tile_sizes(self) -> list[int]:
        return []

    def forward(self, x, ctx, state):
        raise NotImplementedError


class FeedForward(Part):
    def forward(self, x, ctx):
        raise NotImplementedError


class StreamInput(Part):
    # True: forward() wants the stream's rows in the activations' type (``copy``), for a product that reads them
    reads_stream = False

    def forward(self, stream, ctx, copy=None) -> None:
        raise NotImplementedError


class NormedAddend:
    """How a pending output enters the stream when it is normed on the way:
    with y = pending + ``input_bias``,
        resid += (y - mean) / sqrt(var + eps) * weight + bias
    where var is the mean of the squared deviations; not ``centered``: mean is
    0, a root mean square norm.  ``weight`` [W], ``bias`` and ``input_bias`` [W]
    or None, all 32-bit; a factor on what enters is a factor on weight and
    bias.  A norm that reads such a stream applies it in its own kernel."""
    __slots__ = ("weight", "eps", "bias", "centered", "input_bias")

    def __init__(self, weight, eps: float, bias=None, centered: bool = False, input_bias=None):
        self.weight, self.eps, self.bias, self.centered, self.input_bias = weight, float(eps), bias, bool(centered), input_bias

    def plain(self) -> bool:
        """Whether it is a root mean square norm with a weight alone."""
        return self.bias is None and self.input_bias is None and not self.centered


class ScaledAddend:
    """How a pending output enters the stream when every column has a learned
    factor (a layer scale): resid += weight * pending (weight [W], 32-bit),
    applied by the norm that reads the stream, in its own kernel."""
    __slots__ = ("weight",)

    def __init__(self, weight):
        self.weight = weight


class SecondAddend:
    """How a pending output enters the stream when another sub-layer's output
    enters beside it: resid += pending + other (``other`` as a pending output:
    a tensor or float32 partial sums); the norm that reads the stream adds both
    in its own kernel."""
    __slots__ = ("other",)

    def __init__(self, other):
        self.other = other


class Block(Part):
    mixer: Mixer

    def extra_state_needs(self) -> dict[str, StateNeed]:
        """Per-request state that parts of the block other than the mixer keep
        (and what the mixer keeps beyond its one buffer), by a name of the
        block's choosing; ``cache.extra[name]`` holds each buffer when the
        block runs (rows by state slot, as the mixer's)."""
        return dict(self.mixer.extra_state_needs())

    def tile_sizes(self) -> list[int]:
        return list(self.mixer.tile_sizes())

    def forward(self, stream, ctx, cache) -> None:
        raise NotImplementedError


class ResidualStream:
    """The 32-bit residual stream of a step and the last sub-layer's output
    that has not entered it yet (the next norm adds it).  ``resid`` is [T, W],
    or [T, copies, W] where a block arrangement keeps several copies of the
    stream; ``update`` says how ``pending`` enters: None: resid += pending;
    a ``StreamLink`` whose ``mix`` [copies, copies] and ``post`` [copies]
    give copy j <- sum_s mix[s, j] copy_s + post[j] * pending; a
    ``NormedAddend``: resid += pending normed with a weight; a
    ``ScaledAddend``: resid += weight * pending; a ``SecondAddend``: resid +=
    pending + its ``other``."""
    __slots__ = ("resid", "pending", "update", "copies")

    def __init__(self, resid, pending=None):
        self.resid = resid
        self.pending = pending
        self.update = None
        self.copies = 1


# ---------------------------------------------------------------- registries
class Registry:
    def __init__(self, what: str):
        self.what = what
        self._items: dict[str, Callable] = {}

    def register(self, kind: str, factory: Callable | None = None):
        def put(f):
            self._items[kind] = f
            return f
        return put(factory) if factory is not None else put

    def build(self, spec: PartSpec, **extra):
        if spec.kind not in self._items:
            raise KeyError(f"no {self.what} of kind {spec.kind!r} is registered "
                           f"(known: {', '.join(sorted(self._items)) or 'none'})")
        return self._items[spec.kind](**spec.params, **extra)

    def __contains__(self, kind: str) -> bool:
        return kind in self._items

    def kinds(self) -> list[str]:
        return sorted(self._items)


NORMS = Registry("norm")
POSITION_ENCODINGS = Registry("position encoding")
MIXERS = Registry("mixer")
FEED_FORWARDS = Registry("feed-forward")
INPUT_FILTERS = Registry("input filter")
STREAM_INPUTS = Registry("stream input")
BLOCKS = Registry("block arrangement")
EMBEDDINGS = Registry("embedding")
HEADS = Registry("output head")

register_norm = NORMS.register
register_position_encoding = POSITION_ENCODINGS.register
register_mixer = MIXERS.register
register_feed_forward = FEED_FORWARDS.register
register_input_filter = INPUT_FILTERS.register
register_stream_input = STREAM_INPUTS.register
register_block = BLOCKS.register
register_embedding = EMBEDDINGS.register
register_head = HEADS.register
