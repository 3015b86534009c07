"""What every part is, and the registries that turn a plan's kinds into parts.

A part owns its constants (given as arguments, never read from a model class),
names the tensors it needs, loads them, and runs on the flat rows of one step.
No part knows which model it is in: a mixer sees rows, the step's per-token and
per-sequence tables (:class:`StepContext`) and its own cache line.

Interfaces
----------
``Norm.forward(ctx, x, delta=None, rows=None, want32=False, write_back=True)``
    x is the float32 residual stream [T, width]; ``delta`` (float32) is added to
    it first (and stored back when ``write_back``); returns the normed rows in the
    model dtype and, if ``want32``, in float32 too.
``Mixer.forward(ctx, act, line, writes_cache)`` -> float32 update [T, width]
    ``line`` is the :class:`~fieldrun_b200.cache.LineView` of the run's cache line.
``Mixer.cache_need()`` -> :class:`~fieldrun_b200.cache.CacheNeed`
``FeedForward.forward(ctx, act, act32)`` -> float32 update [T, width]
``Position.tables(num_positions, device)`` -> (cos, sin) float32 [positions, dim/2]
``Block.forward(ctx, x, pending, line, writes_cache)`` -> (x, pending)
    ``pending`` is an update not yet added to x, so that the next norm adds it.
``Norm.add_normed(ctx, update, x)`` -> x in the model dtype
    the other place of a norm: x <- x + norm(update), for blocks whose sublayers read x itself.
``Norm.normed(ctx, update)`` -> norm(update) in float32
    a norm behind a sublayer whose block also has one in front (``NormedUpdate`` carries the pair to the next norm).
``Norm.forward_copies(ctx, x, update, streams, gather=..., store=...)`` -> (x, rows, rows in float32)
    the norm of a weighted sum of the copies of a stream that is kept several times (blocks with hyper-connections).
``Connector.forward(ctx, x, pending, first, index)`` -> the new stream [T, width] (float32)
    a part between two runs that rewrites the whole stream; ``first`` holds the embedding's rows.
    ``forward_deferred`` -> (stream, pending): for one that only adds and may leave the sum to the next norm.
``MixerInput.forward(ctx, norm, x, pending, line, offset)`` -> (x, act)
    a part between the mixer's norm and the mixer: it runs the norm and gives the rows that the mixer reads.
``Addition.forward(ctx, x, pending)`` -> (x, pending)
    a part behind a layer's block that adds to the stream once more (a further input per layer and token).
"""
from __future__ import annotations

import json
import weakref
from typing import Any, Callable, Mapping, Optional

import torch

from ..cache import CacheNeed, LineView
from ..config.plan import PartSpec
from ..weights.loader import TensorNeed, TensorSource


class Part:
    """Base of all parts: constants in, tensors by name, rows through.

    ``replayable`` says that the part's ``forward`` reads the step's tables only on the device
    (``ctx.tok_pos`` and the like, never the host lists) and makes every decision from shapes.  A step of
    such parts can be recorded once as a CUDA graph and run again with other positions and slots.  A part
    that leaves it False is always run directly."""

    replayable: bool = False
    # the libraries of kernels (groups of ``csrc/build.py``) that the part launches from; a model compiles and loads
    # the groups of its parts, and no others, before its first step
    kernel_groups: tuple[str, ...] = ("common", "streams")

    def __init__(self, spec: PartSpec, dtype: torch.dtype):
        self.spec = spec
        self.dtype = dtype

    def tensor_needs(self) -> list[TensorNeed]:
        return []

    def load(self, source: TensorSource) -> None:
        pass

    def children(self) -> list["Part"]:
        """Parts that this part is put together from (a mixer made of two mixers); the model counts their tensors,
        kernels and ``replayable`` with its own."""
        return []

    def name_of(self, local: str) -> str:
        try:
            return self.spec.tensors[local]
        except KeyError:
            raise KeyError(f"part {self.spec.kind!r} was given no checkpoint name for its tensor {local!r}") from None


class DeferredUpdate:
    """An update of the residual stream that its maker has not summed up yet, so that the norm which adds it
    can do the sum while it reads the stream.  ``materialize`` gives the plain float32 tensor [T, width]; any
    norm can take any deferred update that way."""

    def materialize(self, ctx) -> torch.Tensor:
        raise NotImplementedError


class WeightedRows(DeferredUpdate):
    """The one deferred form that norms may sum themselves: update[t] = sum over r < k, in the order of r, of
    ``weights[t, r] * rows[row_map[t * k + r]]`` (float32 ``rows`` [N, width], float32 ``weights`` [T, k],
    int32 ``row_map`` [T * k]).  Any part may make one: routed experts do (a token's experts in rank order,
    src/minimax.rs:121-123), and so may a mixer that blends several candidates per token.  A norm that
    cannot take it, or not with this ``k``, calls ``materialize``."""

    def __init__(self, rows: torch.Tensor, weights: torch.Tensor, row_map: torch.Tensor):
        self.rows, self.weights, self.row_map = rows, weights, row_map

    @property
    def top_k(self) -> int:
        return int(self.weights.shape[-1])

    def materialize(self, ctx) -> torch.Tensor:
        from ..csrc import ops
        out = ctx.buffer("weighted_rows.sum", (self.weights.shape[0], self.rows.shape[1]), torch.float32)
        ops.expert_combine(self.rows, self.weights, self.row_map, out)
        return out


class BiasedRows(DeferredUpdate):
    """A float32 tensor [T, width] and a vector [width] that every row of it still has to get (the bias of a projection
    that ends a sublayer), so that the norm which takes the update can add it while it reads the rows."""

    def __init__(self, rows: torch.Tensor, vector: torch.Tensor):
        self.rows, self.vector = rows, vector

    def materialize(self, ctx) -> torch.Tensor:
        from ..csrc import ops
        ops.add_row_vector(self.rows, self.vector, self.rows)
        return self.rows


class UpdateSum(DeferredUpdate):
    """Several updates of one stream that are added together: float32 tensors [T, width], at most one
    :class:`WeightedRows` and at most one :class:`BiasedRows`.  A block whose sublayers all read the same x leaves their
    outputs in this form, so that the norm which reads the stream next adds them while it reads (a norm that does not
    know the form gets their sum from ``materialize``)."""

    def __init__(self, updates):
        biased = [u for u in updates if isinstance(u, BiasedRows)]
        self.tensors = [u.rows if isinstance(u, BiasedRows) else u for u in updates if isinstance(u, (torch.Tensor, BiasedRows))]
        self.vector = biased[0].vector if biased else None
        self.weighted = [u for u in updates if isinstance(u, WeightedRows)]
        other = [u for u in updates if u is not None and not isinstance(u, (torch.Tensor, WeightedRows, BiasedRows))]
        if other or len(self.weighted) > 1 or len(biased) > 1:
            raise ValueError("an UpdateSum holds float32 tensors, at most one WeightedRows and at most one BiasedRows")

    def materialize(self, ctx) -> torch.Tensor:
        from ..csrc import ops
        total = None
        for update in self.tensors + [w.materialize(ctx) for w in self.weighted]:
            if total is None:
                total = update
            else:
                ops.add_rows(total, update)
        if self.vector is not None:
            ops.add_row_vector(total, self.vector, total)
        return total


class WeightedPair(DeferredUpdate):
    """Two float32 tensors [T, width] with a constant weight each, not yet summed: update = wa * a + wb * b.  A mixer
    made of two mixers whose outputs are weighted by constants leaves them in this form, so that the norm which takes
    the update can do the sum while it reads the rows."""

    def __init__(self, a: torch.Tensor, b: torch.Tensor, wa: float, wb: float):
        self.a, self.b, self.wa, self.wb = a, b, float(wa), float(wb)

    def materialize(self, ctx) -> torch.Tensor:
        from ..csrc import ops
        out = ctx.buffer("weighted_pair.sum", tuple(self.a.shape), torch.float32)
        ops.weighted_pair(self.a, self.b, out, self.wa, self.wb)
        return out


class NormedUpdate(DeferredUpdate):
    """A sublayer's output that goes through a norm of its own before it is added to the stream (a block with a norm
    behind each sublayer as well as in front of it): update = norm(inner), ``inner`` a float32 tensor or any deferred
    form.  A norm that reads the stream next and knows the form norms ``inner``, adds and norms the sum in one pass;
    any other norm gets the plain tensor from ``materialize``."""

    def __init__(self, inner, norm: "Norm"):
        self.inner, self.norm = inner, norm

    def materialize(self, ctx) -> torch.Tensor:
        return self.norm.normed(ctx, as_tensor(ctx, self.inner))


class CopiesUpdate:
    """What sublayers left for a stream that is kept as several copies: v_t = sum_s mix[s, t] x_s + first_out[t] * first +
    second_out[t] * second.  ``first`` and ``second`` are float32 tensors [T, width] or any deferred form (or None); ``mix``
    [S, S] and the weights [S] are float32 tensors on the device."""

    def __init__(self, mix: torch.Tensor, first=None, first_out: Optional[torch.Tensor] = None, second=None,
                 second_out: Optional[torch.Tensor] = None):
        self.mix, self.first, self.first_out, self.second, self.second_out = mix, first, first_out, second, second_out

    def kernel_args(self, ctx) -> dict:
        """The update as ``ops.stream_copies`` takes it: its first part one tensor, its second one summed there if it can be."""
        from ..csrc import ops
        tensors, experts = (), None
        second = self.second
        if isinstance(second, WeightedRows) and second.top_k <= ops.COPIES_MAX_SUMMED_ROWS:
            experts = (second.rows, second.weights, second.row_map)
        elif (isinstance(second, UpdateSum) and second.vector is None and len(second.tensors) <= 2
                and all(w.top_k <= ops.COPIES_MAX_SUMMED_ROWS for w in second.weighted)):
            tensors = tuple(second.tensors)
            experts = next(((w.rows, w.weights, w.row_map) for w in second.weighted), None)
        elif second is not None:
            tensors = (as_tensor(ctx, second),)
        first = (as_tensor(ctx, self.first), self.first_out) if self.first is not None else None
        return dict(mix=self.mix, first=first, second=tensors, experts=experts, second_out=self.second_out)


def as_tensor(ctx, update):
    """The update as a float32 tensor, whatever form it came in (None stays None)."""
    return update.materialize(ctx) if isinstance(update, DeferredUpdate) else update


class Norm(Part):
    accepts_deferred: bool = False       # whether ``delta`` may be a DeferredUpdate of a kind this norm knows

    def forward(self, ctx, x: torch.Tensor, *, delta=None,
                rows: Optional[torch.Tensor] = None, want32: bool = False, write_back: bool = True):
        raise NotImplementedError

    def add_normed(self, ctx, update: torch.Tensor, x: torch.Tensor) -> torch.Tensor:
        """For a block whose norm sits on the sublayer's output: x <- x + norm(update) in float32, in place;
        returns the new x in the model dtype (x itself in float32 mode), which the next sublayer reads."""
        raise NotImplementedError(f"norm {self.spec.kind!r} has no form that norms a sublayer's output")

    def normed(self, ctx, update: torch.Tensor) -> torch.Tensor:
        """norm(update) as a float32 tensor [T, width]: the norm of rows that are not the stream (a sublayer's output)."""
        raise NotImplementedError(f"norm {self.spec.kind!r} has no form that norms rows other than the stream")


    def forward_copies(self, ctx, x: torch.Tensor, update: Optional[CopiesUpdate], streams: int, *,
                       gather: Optional[torch.Tensor] = None, rows: Optional[torch.Tensor] = None, want32: bool = False,
                       store: bool = False):
        """norm(sum_t gather[t] v_t) over the copies v of the stream with ``update`` in them (without ``gather`` their plain
        sum); with ``store`` the v are kept.  ``x`` is [T, streams, width], or [T, width] while all copies are equal.
        Returns (the stream, the rows in the model dtype, the rows in float32 if ``want32``)."""
        from ..csrc import ops
        count = rows.numel() if rows is not None else x.shape[0]
        args = update.kernel_args(ctx) if update is not None else {}
        kept = self.copies_buffer(ctx, x, streams) if store else None
        summed = ctx.buffer("stream.copies_sum", (count, x.shape[-1]), torch.float32)
        ops.stream_copies(x, streams, gather=gather, rows=rows, store=kept, out32=summed, **args)
        act, act32 = self.forward(ctx, summed, want32=want32)
        return x if kept is None else kept, act, act32

    @staticmethod
    def copies_buffer(ctx, x: torch.Tensor, streams: int) -> torch.Tensor:
        """Where the copies are kept: x itself once it holds them, else a buffer beside the one row that stood for them."""
        return x if x.dim() == 3 else ctx.buffer("stream.copies", (x.shape[0], streams, x.shape[-1]), torch.float32)


class Position:
    """A position encoding handed to a mixer: it fills the tables the mixer's kernel rotates with.
    ``build_position`` gives mixers whose position arguments are equal one and the same object, and
    ``shared_tables`` makes that object's tables once per (length, device): the layers of a model read one
    pair of tables, not one pair each."""

    rotary_dim: int = 0
    interleaved: bool = False

    def tables(self, num_positions: int, device) -> tuple[Optional[torch.Tensor], Optional[torch.Tensor]]:
        raise NotImplementedError

    def shared_tables(self, num_positions: int, device) -> tuple[Optional[torch.Tensor], Optional[torch.Tensor]]:
        made = self.__dict__.setdefault("_tables_made", {})
        key = (int(num_positions), str(torch.device(device)))
        if key not in made:
            made.clear()                      # one length at a time: a model's cache is sized once
            made[key] = self.tables(num_positions, device)
        return made[key]


class Mixer(Part):
    def cache_need(self) -> CacheNeed:
        return CacheNeed()

    def prepare(self, num_positions: int, device) -> None:
        """Called once the cache's size is known (tables over positions are made here)."""

    def forward(self, ctx, act: torch.Tensor, line: LineView, writes_cache: bool) -> torch.Tensor:
        raise NotImplementedError


class FeedForward(Part):
    wants_float32_input: bool = False

    def forward(self, ctx, act: torch.Tensor, act32: Optional[torch.Tensor]) -> torch.Tensor:
        raise NotImplementedError

    def forward_deferred(self, ctx, act: torch.Tensor, act32: Optional[torch.Tensor]):
        """Like ``forward``, but may return a :class:`DeferredUpdate`."""
        return self.forward(ctx, act, act32)


class Connector(Part):
    """A part that stands between two runs of the run order and rewrites the stream as a whole."""

    def forward(self, ctx, x: torch.Tensor, pending, first: torch.Tensor, index: int) -> torch.Tensor:
        raise NotImplementedError

    def forward_deferred(self, ctx, x: torch.Tensor, pending, first: torch.Tensor, index: int):
        """Like ``forward``, but returns (stream, pending) and may leave an addition to the next norm."""
        return self.forward(ctx, x, pending, first, index), None


class MixerInput(Part):
    """A part between a mixer's norm and the mixer.  It may keep a float32 state per sequence, twice (``state_floats``
    floats behind the mixer's own state, see ``CacheNeed.with_state_behind``; ``offset`` says where they begin)."""

    state_floats: int = 0

    def forward(self, ctx, norm: "Norm", x: torch.Tensor, pending, line: LineView, offset: int):
        """Norms x + pending and returns (the stream with the sum in it, the rows that the mixer reads)."""
        raise NotImplementedError


class Addition(Part):
    """A part behind a layer's block that adds to the stream once more; it may read the step's token ids
    (``ctx.step_tokens``, on the device).  ``forward(ctx, x, pending)`` gets the stream and the update that the block
    left unsummed, and returns the two in the same form."""

    def forward(self, ctx, x: torch.Tensor, pending):
        raise NotImplementedError


class StreamConnection(Part):
    """The constants with which a layer's sublayers read the copies of a stream and spread their outputs over them."""


def shared_fetch(source: TensorSource, need: TensorNeed) -> torch.Tensor:
    """A tensor that several parts read (one table with a share per layer): fetched once per source and kept with it."""
    try:
        kept = source.__dict__.setdefault("_shared_tensors", {})
    except AttributeError:
        return source.fetch(need)
    key = (need.name, need.role)
    if key not in kept:
        kept[key] = source.fetch(need)
    return kept[key]


class Block:
    def __init__(self, mixer: Mixer, feed_forward: FeedForward, mixer_norm: Norm, feed_forward_norm: Norm,
                 mixer_out_norm: Optional[Norm] = None, feed_forward_out_norm: Optional[Norm] = None):
        self.mixer, self.feed_forward = mixer, feed_forward
        self.mixer_norm, self.feed_forward_norm = mixer_norm, feed_forward_norm
        # norms behind the sublayers, for the arrangements that have them
        self.mixer_out_norm, self.feed_forward_out_norm = mixer_out_norm, feed_forward_out_norm
        self.mixer_input: Optional[MixerInput] = None
        self.connections: Optional[StreamConnection] = None

    takes_connections: bool = False      # whether the arrangement runs on a stream that is kept as several copies

    def set_connections(self, part: StreamConnection) -> None:
        if not self.takes_connections:
            raise ValueError(f"{type(self).__name__} runs on a single stream, not on copies of it")
        self.connections = part

    takes_mixer_input: bool = False      # whether the arrangement has a place for a part in front of the mixer

    def set_mixer_input(self, part: MixerInput) -> None:
        if not self.takes_mixer_input:
            raise ValueError(f"{type(self).__name__} has no place for a part between the norm and the mixer")
        self.mixer_input = part

    def parts(self) -> list[Part]:
        """The block's parts; a layer without a feed-forward has neither it nor its norms."""
        return [part for part in (self.connections, self.mixer_norm, self.mixer_input, self.mixer, self.mixer_out_norm, self.feed_forward_norm,
                                  self.feed_forward, self.feed_forward_out_norm) if part is not None]

    def cache_need(self) -> CacheNeed:
        """What a run of the block needs of its cache line: the mixer's keys, values and state, and behind that state
        the one of the part in front of the mixer."""
        need = self.mixer.cache_need()
        return need.with_state_behind(self.mixer_input.state_floats) if self.mixer_input is not None else need

    def input_offset(self) -> int:
        """Where, in a copy of the line's state, the part in front of the mixer has its own."""
        return self.mixer.cache_need().copy_floats

    def forward(self, ctx, x, pending, line: LineView, writes_cache: bool):
        raise NotImplementedError


_REGISTRIES: dict[str, dict[str, Callable[..., Any]]] = {
    "mixer": {}, "feed_forward": {}, "norm": {}, "position": {}, "block": {}, "embedding": {}, "head": {},
    "connector": {}, "addition": {}, "mixer_input": {}, "stream_connection": {},
}


def register_part(category: str, kind: str, factory: Callable[..., Any], *, replace: bool = False) -> None:
    """Make ``kind`` buildable.  ``factory(spec, dtype)`` for parts with tensors, ``factory(args)`` for a
    position encoding, ``factory(mixer, feed_forward, mixer_norm, feed_forward_norm)`` for a block."""
    table = _REGISTRIES[category]
    if kind in table and not replace:
        raise ValueError(f"{category} {kind!r} is already registered")
    table[kind] = factory


def registered(category: str) -> list[str]:
    return sorted(_REGISTRIES[category])


def _factory(category: str, kind: str):
    try:
        return _REGISTRIES[category][kind]
    except KeyError:
        raise KeyError(f"no {category} of kind {kind!r} is registered; registered: {registered(category)}") from None


def build_part(category: str, spec: PartSpec, dtype: torch.dtype):
    return _factory(category, spec.kind)(spec, dtype)


_POSITIONS: "weakref.WeakValueDictionary[str, Position]" = weakref.WeakValueDictionary()


def build_position(args: Optional[Mapping[str, Any]]) -> Optional[Position]:
    """The position encoding of ``args``; equal arguments give the same object while a mixer still holds it."""
    if not args:
        return None
    factory = _factory("position", args["kind"])
    try:
        key = f"{id(factory)}:" + json.dumps(dict(args), sort_keys=True, default=repr)
    except (TypeError, ValueError):
        return factory(args)
    position = _POSITIONS.get(key)
    if position is None:
        position = factory(args)
        try:
            _POSITIONS[key] = position
        except TypeError:                     # an object that cannot be weakly referenced is simply not shared
            pass
    return position


def build_block(kind: str, mixer, feed_forward, mixer_norm, feed_forward_norm, mixer_out_norm=None,
                feed_forward_out_norm=None) -> Block:
    """``mixer_out_norm`` and ``feed_forward_out_norm``: the norms behind the sublayers, for a layer that names them."""
    if mixer_out_norm is None and feed_forward_out_norm is None:
        return _factory("block", kind)(mixer, feed_forward, mixer_norm, feed_forward_norm)
    return _factory("block", kind)(mixer, feed_forward, mixer_norm, feed_forward_norm, mixer_out_norm, feed_forward_out_norm)
