"""Interfaces of the parts and the registries that map a spec's `kind` to a class.

A part is built from its spec, its tensors and the kernel set (`ops`); it never sees
the model it sits in.  A mixer tells the cache manager what it has to remember
through `cache_need`: keys and values per token in pages (`PagedNeed`), a record of
fixed size per request (`StateNeed`), or nothing.

Buffers for activation rows that a matrix product will read (`[tokens, width]` outputs of
a norm, an activation, a mixer's inner stage) come from `ops.new_rows(n, width, dtype,
device)` rather than `torch.empty`: the kernel set may leave room behind them so that the
matrix library is shown row counts it has met before.  Any tensor still works as a
product's input; it is then copied once.

Adding a part: subclass the interface, give `params` and (for a mixer) `cache_need`,
and call the matching `register_*` with the `kind` string its spec carries.  Nothing
else in the package has to change.
"""
from __future__ import annotations

from dataclasses import dataclass
from typing import Callable, Dict, Optional, Tuple

from .spec import ParamDecl


@dataclass(frozen=True)
class PagedNeed:
    """Keys and values of every token, in pages.  `window`: only the last `window` positions
    are ever read again; `chunk`: only the positions of the newest chunk of `chunk` positions
    (counted from position 0) are.  Both tell the cache manager which pages it may take
    back early; neither changes the layout.  `v_head_dim`: size of a value head when it is
    not the key size.  `values` false: one row per token is all there is (a latent row that
    keys and values are both made from); no value pages exist.  `every` > 1: one row per `every`
    tokens (made from them when the last of them is written) instead of one per token.  `block`:
    the rows of the newest incomplete block of `block` positions are read once more when it
    completes, so their pages stay until then whatever the window says.  `keep_first`: the first so
    many positions stay visible whatever the window says, and so do their pages."""
    num_kv_heads: int
    head_dim: int
    window: Optional[int] = None
    chunk: Optional[int] = None
    v_head_dim: Optional[int] = None
    values: bool = True
    every: int = 1
    block: Optional[int] = None
    keep_first: int = 0

    @property
    def value_dim(self) -> int:
        if not self.values:
            return 0
        return self.v_head_dim if self.v_head_dim else self.head_dim

    def layout(self):
        """What two calls must agree on to share pages."""
        return (self.num_kv_heads, self.head_dim, self.value_dim, self.every)

    def rows(self, tokens: int) -> int:
        """Rows that the first `tokens` positions of a request have."""
        return tokens // self.every


@dataclass(frozen=True)
class SeveralNeeds:
    """What a mixer made of several mixers has to remember: one need (or None) per branch, in
    the branches' order.  The call's cache view then has `parts`, one view (or None) each.  A part
    may itself be several."""
    parts: Tuple[object, ...]


@dataclass(frozen=True)
class StateNeed:
    """A float32 record of this shape per live request.  The cache manager hands a request
    its slot with the record cleared to zero, so the state before position 0 is zero
    without the mixer's doing."""
    shape: Tuple[int, ...]


class Mixer:
    """mixer(normed[N, hidden], ctx, cache) -> [N, hidden]

    `ctx` is the step's `StepContext` (token positions, request boundaries, the
    kernels); `cache` is the `CacheView` of this call in the run order or None.
    """

    @staticmethod
    def params(spec, owns_cache: bool = True) -> Dict[str, ParamDecl]:
        """Tensors by local name.  `owns_cache` is false when every call of the block
        reads another call's cache, so tensors that only fill a cache are not needed."""
        raise NotImplementedError

    @staticmethod
    def cache_need(spec):
        return None

    @staticmethod
    def workspace_bytes(spec, ops, max_requests: int, max_context: int) -> int:
        """Bytes of kernel scratch the mixer's launches can need at most with
        `max_requests` requests of up to `max_context` cached tokens in a step.  The
        runner reserves the largest answer once, before it captures any launch sequence."""
        return 0

    def __init__(self, spec, tensors, ops, dtype):
        raise NotImplementedError

    def forward(self, normed, ctx, cache):
        raise NotImplementedError


class FeedForward:
    """feed_forward(normed[N, hidden], ctx) -> [N, hidden]"""

    @staticmethod
    def params(spec) -> Dict[str, ParamDecl]:
        raise NotImplementedError

    def __init__(self, spec, tensors, ops, dtype):
        raise NotImplementedError

    def forward(self, normed, ctx):
        raise NotImplementedError


class Norm:
    """norm.add_norm(resid, delta, ctx, rows=None, delta_norm=None) adds `delta` (or
    nothing) to the float32 residual stream in place and returns the normalised rows in the
    compute dtype; with `rows` it reads only those rows and leaves the stream untouched.
    `delta_norm` is a norm that `delta` still has to pass through before it is added (a norm
    placed after a sub-layer): a class that can do both in one kernel does, any other calls
    `delta_norm.norm` first (`_normed_delta`).
    norm.norm(x, ctx) normalises rows that are not part of the stream."""

    @staticmethod
    def params(spec) -> Dict[str, ParamDecl]:
        raise NotImplementedError

    def __init__(self, spec, tensors, ops, dtype):
        raise NotImplementedError

    def add_norm(self, resid, delta, ctx, rows=None, delta_norm=None):
        raise NotImplementedError

    @staticmethod
    def _normed_delta(delta, delta_norm, ctx):
        if delta is None or delta_norm is None:
            return delta
        return delta_norm.norm(delta, ctx)

    def norm(self, x, ctx):
        """The normalised rows of `x` (compute dtype), with no residual stream involved:
        what a norm placed after a sub-layer applies to its output."""
        raise NotImplementedError

    def scale_output(self, factor: float) -> None:
        """From now on the normalised rows come out times `factor` (the weights take it in)."""
        raise NotImplementedError


class PositionEncoding:
    """A position encoding the attention mixer can apply to q and k.

    `rotation_table()` returns (cos, sin), float32 [max_position, head_dim/2], of a
    rotation that pairs dimension i with i + head_dim/2, or None for no encoding.
    """

    def __init__(self, spec, device):
        raise NotImplementedError

    def rotation_table(self):
        raise NotImplementedError


class Arrangement:
    """How a block wires norm, mixer and feed-forward around the residual stream.

    `cache_need(spec)` is what one call of the block has to remember: the mixer's need unless
    the arrangement itself keeps something between steps.  `fresh_stream`: the block's first norm
    leaves the residual rows it is given as they are and goes on with new ones.

    forward(stream, ctx, cache) -> stream, where `stream` is a `Stream`: the float32
    residual plus the last sub-layer's output that is still to be added (so that the
    addition can be fused into the next norm).
    """

    @staticmethod
    def params(spec, owns_cache: bool = True) -> Dict[str, ParamDecl]:
        """Full tensor names -> declarations for one block."""
        raise NotImplementedError

    fresh_stream = False

    @staticmethod
    def cache_need(spec):
        return mixer_class(spec.mixer.kind).cache_need(spec.mixer)

    def __init__(self, spec, tensors, ops, dtype):
        raise NotImplementedError

    def forward(self, stream, ctx, cache):
        raise NotImplementedError


@dataclass
class Stream:
    resid: object                   # float32 [N, hidden]
    pending: Optional[object]       # [N, hidden], not yet added
    pending_norm: Optional[object] = None   # a Norm `pending` has to pass through first
    pending_hyper: Optional[tuple] = None   # (mix [S, S], out [S]): how `pending` enters the
                                            # streams of a block with hyper-connections
    pending_scale: Optional[object] = None  # float32 [hidden]: `pending` is multiplied by it,
                                            # channel by channel, as it is added
    pending_add: Optional[object] = None    # float32 [hidden]: one vector that every row of the
                                            # stream still has to receive
    pending_rows: Optional[object] = None   # float32 [N, hidden]: rows still to be added as well


_MIXERS: Dict[str, type] = {}
_FEED_FORWARDS: Dict[str, type] = {}
_NORMS: Dict[str, type] = {}
_POSITIONS: Dict[str, type] = {}
_ARRANGEMENTS: Dict[str, type] = {}


def _register(table: Dict[str, type], what: str) -> Callable:
    def register(kind: str, cls: type, replace: bool = False) -> type:
        if kind in table and table[kind] is not cls and not replace:
            raise ValueError(f"{what} kind {kind!r} is already registered")
        table[kind] = cls
        return cls
    return register


def _lookup(table: Dict[str, type], what: str) -> Callable:
    def lookup(kind: str) -> type:
        if kind not in table:
            raise KeyError(f"unknown {what} kind {kind!r} (registered: {sorted(table)})")
        return table[kind]
    return lookup


register_mixer = _register(_MIXERS, "mixer")
register_feed_forward = _register(_FEED_FORWARDS, "feed-forward")
register_norm = _register(_NORMS, "norm")
register_position = _register(_POSITIONS, "position encoding")
register_arrangement = _register(_ARRANGEMENTS, "arrangement")
mixer_class = _lookup(_MIXERS, "mixer")
feed_forward_class = _lookup(_FEED_FORWARDS, "feed-forward")
norm_class = _lookup(_NORMS, "norm")
position_class = _lookup(_POSITIONS, "position encoding")
arrangement_class = _lookup(_ARRANGEMENTS, "arrangement")
