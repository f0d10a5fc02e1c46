"""Interfaces of the parts a decoder is assembled from, and the registries that map a part's kind
(a string in the model plan) to its class.

A part knows its own sizes and constants (constructor parameters), the tensors it needs by name
(`weight_specs`), what it wants from the cache manager (`cache_need`, mixers only) and how to run
on a step's tokens (`forward`). No part knows which model it is in, and none reads a model config.

Adding a part means subclassing one of the interfaces below and calling the matching `register_*`
function; the decoder, the loader, the cache manager and the step function find it through the plan.
"""
from __future__ import annotations

from dataclasses import dataclass
from typing import TYPE_CHECKING, Callable, Optional

import torch

if TYPE_CHECKING:
    from ..engine.context import StepContext
    from ..engine.runtime import Runtime


# ------------------------------------------------------------------ what a part asks of the loader
@dataclass(frozen=True)
class WeightSpec:
    """One tensor a part reads by name. `role` decides precision on the device and random init:
    "matrix": kept in bfloat16 unless stored in 32-bit; random ~ N(0, std)
    "norm":   per-channel scale used in float32; random 1 + U(-0.1, 0.1)
    "norm_offset": the same stored around zero (the scale is 1 + w); random U(-0.2, 0.2)
    "gate_floor": lower bounds of a forget gate, used in float32; random U(0, 0.9)
    "unit":   per-channel mixing weights, used in float32; random U(0, 1)
    "log_rate": logarithms of decay rates, used in float32; random log U(0.5, 8)
    "decay_bias": what a decay exp(-exp(z)) adds to z, used in float32; random U(-6, 0)
    "keep_bias": what a forget gate's pre-activation gets added so that it mostly keeps, used in float32; random U(2, 6)
    "mix":    weights of an average over the n entries of the tensor's last axis, used in float32; random around 1 / n
    "table":  integer table, int32.
    `free` lists the axes whose size the checkpoint decides (the shape's entry there is what random weights are made with)."""
    name: str
    shape: tuple[int, ...]
    role: str = "matrix"
    std: float = 0.02
    free: tuple[int, ...] = ()

    def fits(self, shape) -> bool:
        return len(shape) == len(self.shape) and all(a == b or i in self.free for i, (a, b) in enumerate(zip(shape, self.shape)))


# ------------------------------------------------------------------ what a mixer asks of the cache
@dataclass(frozen=True)
class PagedKV:
    """Keys and values for every token (or for the last `window` tokens and the first `keep_first`) of a request, in pages."""
    kv_heads: int
    head_dim: int
    window: Optional[int] = None
    keep_first: int = 0     # with a window: the positions 0 .. keep_first - 1 stay for as long as the request lives


@dataclass(frozen=True)
class PagedRows:
    """One row of `width` values for every token of a request, in pages (what latent attention keeps: a
    compressed latent and a rotated key part that all heads share)."""
    width: int
    window: Optional[int] = None


@dataclass(frozen=True)
class FixedState:
    """Per-request state of fixed size, zeroed when a request is admitted."""
    shape: tuple[int, ...]
    dtype: torch.dtype = torch.float32


@dataclass(frozen=True)
class Several:
    """More than one thing for one execution (a block with state of its own beside its mixer's cache): the execution gets a tuple
    of views in the order of `needs`, None where an item is None."""
    needs: tuple


CacheNeed = Optional[object]  # PagedKV | PagedRows | FixedState | Several | None


def flat_needs(needs) -> list:
    """Every single need (no None, no `Several`) among an execution list's needs."""
    out = []
    for n in needs:
        for m in (n.needs if isinstance(n, Several) else (n,)):
            if m is not None:
                out.append(m)
    return out


class Part:
    """Common life cycle: construct from sizes -> weight_specs() -> bind(weights, runtime)."""

    prefix: str = ""

    def weight_specs(self) -> list[WeightSpec]:
        return []

    def bind(self, weights: dict[str, torch.Tensor], rt: "Runtime") -> None:
        """Take this part's tensors (device tensors, in their stored precision) and prepare them
        for the runtime's mode (fuse, convert, upload derived tables)."""


@dataclass
class NormedDelta:
    """A contribution to the residual stream that still has to go through a norm of its own before it is added: what a block leaves for the
    next norm when its sublayers' outputs are normed (x += norm(sum of `delta` + `bias`)). A norm that is given one as `delta` applies `norm`
    (same kind, same epsilon) to it first; `Norm.takes_normed_delta` says whether it can."""
    delta: torch.Tensor                     # float32 [P, T, H]
    norm: "Norm"
    bias: Optional[torch.Tensor] = None     # float32 [H], added to the summed partial sums before the norm


@dataclass
class ScaledDelta:
    """A contribution to the residual stream that is multiplied by a constant where it is added: x += scale * (sum of `delta`). What a block
    with a residual multiplier leaves for the next norm; `Norm.takes_scaled_delta` says whether a norm can add one."""
    delta: torch.Tensor     # float32 [P, T, H]
    scale: float


@dataclass
class SummedDelta:
    """Two contributions to the residual stream that are added one after the other: what a block whose sublayers run side by side leaves for
    the next norm; `Norm.takes_summed_delta` says whether a norm can add one."""
    first: torch.Tensor     # float32 [P, T, H]
    second: torch.Tensor    # float32 [P2, T, H]


class Norm(Part):
    takes_summed_delta = False   # True: `forward` takes a `SummedDelta` as delta
    takes_scaled_delta = False   # True: `forward` takes a `ScaledDelta` as delta
    takes_normed_delta = False   # True: `forward` takes a `NormedDelta` as delta

    def forward(self, ctx: "StepContext", x: torch.Tensor, delta: Optional[torch.Tensor], rows: Optional[torch.Tensor] = None) -> torch.Tensor:
        """x: float32 residual stream [T, H], updated in place by `delta` (float32 [P, T, H] or None);
        returns the normalised rows in the runtime's activation dtype. With `rows` only those
        source rows are produced and x is left as it is."""
        raise NotImplementedError

    def add_normed(self, ctx: "StepContext", x: torch.Tensor, delta: torch.Tensor, mult: float) -> torch.Tensor:
        """The norm applied to a sublayer's output instead of its input: x += mult * norm(sum of `delta`), in place
        (delta: float32 [P, T, H]); returns x in the runtime's activation dtype, for the next sublayer to read."""
        raise NotImplementedError


class PositionEncoding(Part):
    def tables(self, ctx: "StepContext") -> tuple[Optional[torch.Tensor], Optional[torch.Tensor]]:
        """(cos, sin), float32 [T, rotary_dim/2], for the step's tokens; (None, None) for no rotation."""
        raise NotImplementedError


class Mixer(Part):
    adds_to_residual = False   # True: forward takes `residual=` and may add its contribution there itself
    runs_norm = False          # True: the block calls `forward_normed(ctx, norm, x, pending, cache)` instead of running its input norm and `forward`:
                               # a mixer that reads the normed rows in more than one form (several shifted mixes of them) makes them in its own kernels
    out_bias: Optional[torch.Tensor] = None   # float32 [H], set at bind: a vector that belongs to every row of the contribution and that the
                                              # kernel which adds the contribution to the stream adds with it (only blocks that say so take such a mixer)

    def cache_need(self) -> CacheNeed:
        return None

    def forward(self, ctx: "StepContext", h: torch.Tensor, cache) -> torch.Tensor:
        """h: normalised activations [T, H]; cache: what the cache manager gave this execution
        (a KvLayerView for PagedKV and PagedRows, a StateView for FixedState, None otherwise).
        Returns the residual contribution, float32 [P, T, H] (P partial sums, added in order).
        A part with `adds_to_residual` is called with `residual=x` (float32 [T, H]) as well: it may
        add its contribution to x in place and return None, or leave x alone and return the partial sums."""
        raise NotImplementedError


class FeedForward(Part):
    adds_to_residual = False   # as for a mixer

    def forward(self, ctx: "StepContext", h: torch.Tensor) -> torch.Tensor:
        """Returns the residual contribution, float32 [P, T, H]."""
        raise NotImplementedError


class Embedding(Part):
    def forward(self, ctx: "StepContext") -> torch.Tensor:
        """Returns the float32 residual stream [T, H] for ctx.token_ids."""
        raise NotImplementedError


class Head(Part):
    def forward(self, ctx: "StepContext", h: torch.Tensor) -> torch.Tensor:
        """h: normalised rows [K, H] -> float32 logits [K, V]."""
        raise NotImplementedError


class StreamPart(Part):
    """A part that works on the residual stream itself between two executions of the schedule (the entry of a pass over looped layers,
    for instance). A plan names it in `stream_parts`; a schedule entry's `enter = (part, occurrence)` runs it right before that entry."""

    needs_embedding = False   # True: `forward` is given the embedding's output of the step as x0

    def forward(self, ctx: "StepContext", x: torch.Tensor, pending: Optional[torch.Tensor], x0: Optional[torch.Tensor], occurrence: int) -> Optional[torch.Tensor]:
        """x: float32 residual stream [T, H] (in place); pending: a contribution not yet added to it. Returns the contribution it leaves
        for the next norm to add (or None)."""
        raise NotImplementedError


class Block:
    """An arrangement of norm, mixer and feed-forward around the residual stream."""

    def __init__(self, mixer_norm: Norm, mixer: Mixer, feed_forward_norm: Norm, feed_forward: FeedForward):
        self.mixer_norm, self.mixer, self.feed_forward_norm, self.feed_forward = mixer_norm, mixer, feed_forward_norm, feed_forward

    takes_out_bias = False   # True: the arrangement adds a mixer's `out_bias` where it adds the mixer's contribution

    def parts(self) -> list[Part]:
        return [self.mixer_norm, self.mixer, self.feed_forward_norm, self.feed_forward]

    def cache_need(self) -> CacheNeed:
        """What an execution of this block asks of the cache manager: its mixer's need, unless the arrangement has state of its own."""
        return self.mixer.cache_need()

    def forward(self, ctx: "StepContext", x: torch.Tensor, pending: Optional[torch.Tensor], cache) -> Optional[torch.Tensor]:
        """Runs the block on x (in place). `pending` is a contribution not yet added to x; the
        return value is the block's own last contribution, left for the next norm to add."""
        raise NotImplementedError


# ------------------------------------------------------------------ registries
MIXERS: dict[str, Callable[..., Mixer]] = {}
FEED_FORWARDS: dict[str, Callable[..., FeedForward]] = {}
NORMS: dict[str, Callable[..., Norm]] = {}
POSITION_ENCODINGS: dict[str, Callable[..., PositionEncoding]] = {}
EMBEDDINGS: dict[str, Callable[..., Embedding]] = {}
HEADS: dict[str, Callable[..., Head]] = {}
BLOCKS: dict[str, Callable[..., Block]] = {}
STREAM_PARTS: dict[str, Callable[..., StreamPart]] = {}


def _register(table: dict, what: str):
    def register(kind: str, factory=None):
        def put(f):
            table[kind] = f
            return f
        return put(factory) if factory is not None else put
    register.__doc__ = f"Register a {what} under a kind name; usable as a decorator."
    return register


register_mixer = _register(MIXERS, "mixer")
register_feed_forward = _register(FEED_FORWARDS, "feed-forward")
register_norm = _register(NORMS, "norm")
register_position_encoding = _register(POSITION_ENCODINGS, "position encoding")
register_embedding = _register(EMBEDDINGS, "embedding")
register_head = _register(HEADS, "head")
register_block = _register(BLOCKS, "block arrangement")
register_stream_part = _register(STREAM_PARTS, "stream part")


def make(table: dict, what: str, kind: str, **params):
    if kind not in table:
        raise KeyError(f"no {what} of kind {kind!r} is registered (known: {', '.join(sorted(table)) or 'none'})")
    return table[kind](**params)
