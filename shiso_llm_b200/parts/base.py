"""Interfaces of the parts a model is put together from, and their registries.

A part is built from a ``PartSpec`` (its sizes and constants) and a ``BuildEnv``
(compute dtype, device, the kernel table).  It lists the tensors it needs, is
handed them by name after loading, says what cache it needs, and runs on the
rows of one step.  No part knows which model it is in.

Kinds of part and what each must provide:

``Norm``             ``apply(x)``, ``add_apply(residual, delta, rows=None)``, optional ``add_apply_linear``
``PositionEncoding`` ``rotary()`` - the per-pair frequencies the fused kernel rotates by
``Mixer``            ``cache_spec()``, ``forward(x, step, cache)`` -> tensor or ``DeferredLinear``
``FeedForward``      ``forward(x, step)`` -> tensor or ``DeferredLinear``
                     (both: ``takes_deferred_norm = True`` to get ``x`` as a ``DeferredNorm``)
``Block``            ``forward(stream, step, cache)`` - the arrangement of the above
``Embedding``        ``forward(step)`` -> float32 residual rows
``Head``             ``forward(x)`` -> float32 logits
``SideInput``        ``forward(rows, step)`` -> something to add to the stream behind a layer
"""

from __future__ import annotations

from dataclasses import dataclass
from typing import Any, Callable, Optional

import torch

from ..weights.spec import TensorSpec
from .plan import PartSpec


@dataclass
class BuildEnv:
    """What every part needs to know about where it runs."""

    dtype: torch.dtype  # compute dtype: activations between kernels, 16-bit weights
    device: torch.device
    ops: Any  # the kernel table (shiso_llm_b200.kernels.ops, or a stand-in in CPU tests)

    def empty(self, shape, dtype=None) -> torch.Tensor:
        return torch.empty(shape, dtype=dtype or self.dtype, device=self.device)


# --------------------------------------------------------------------------- cache needs


@dataclass(frozen=True)
class PagedKV:
    """Keys and values of every position, in pages.  ``window`` = how many of the most
    recent positions are ever read again (None: all of them).  Values may have another width
    than keys (``v_head_dim``; None: the same), and the entry may ask for an element type of
    its own (``dtype``; None: the engine's compute type).  ``every`` > 1 asks for one row per
    complete run of that many positions instead of one per position (summaries of blocks of
    tokens): a request of ``n`` positions then holds ``n // every`` rows.  ``keep_first`` > 0
    (with a window) says that the first so many positions are read for the request's whole life:
    the pages that hold them never go back while the window moves on.

    A mixer that needs more than one cache returns a tuple of needs from ``cache_spec`` and
    is handed a tuple of views in the same order."""

    num_kv_heads: int
    head_dim: int
    window: Optional[int] = None
    v_head_dim: Optional[int] = None
    dtype: Optional[torch.dtype] = None
    every: int = 1
    keep_first: int = 0
    num_v_heads: Optional[int] = None  # fewer value heads than key heads: neighbouring key heads share one (None: as many)

    @property
    def value_dim(self) -> int:
        return self.head_dim if self.v_head_dim is None else self.v_head_dim

    @property
    def value_heads(self) -> int:
        return self.num_kv_heads if self.num_v_heads is None else self.num_v_heads


@dataclass(frozen=True)
class FixedState:
    """Per-request state of fixed size, zero for a new request; float32 unless the entry asks
    for another element type."""

    shape: tuple[int, ...]
    dtype: torch.dtype = torch.float32

    @property
    def numel(self) -> int:
        n = 1
        for d in self.shape:
            n *= d
        return n

    @property
    def nbytes(self) -> int:
        return self.numel * self.dtype.itemsize


# --------------------------------------------------------------------------- part classes


class Part:
    """Common protocol: tensors wanted, tensors bound.

    ``graph_safe``: the part's launches depend on the step only through device arrays
    (positions, tables, slots), never through host values that change from step to step,
    so a captured decode step can be replayed.  A part that loops on the host over the
    step's sequences sets it to False and its model runs decode steps without graphs."""

    graph_safe = True

    def __init__(self, spec: PartSpec, env: BuildEnv):
        self.spec = spec
        self.env = env

    def tensor_specs(self) -> list[TensorSpec]:
        return []

    def bind(self, tensors: dict[str, torch.Tensor]) -> None:
        """Receives every loaded tensor by name; keep what ``tensor_specs`` named."""

    def sub_parts(self) -> list["Part"]:
        return []


class Norm(Part):
    def apply(self, x: torch.Tensor) -> torch.Tensor:
        """Normalises float32 rows ``x[T, size]``; returns compute-dtype rows."""
        raise NotImplementedError

    def add_apply(self, residual: torch.Tensor, delta: torch.Tensor, rows: Optional[torch.Tensor] = None):
        """``residual += delta`` (float32, in place) and returns norm(residual).

        With ``rows`` (int32 row numbers) only those rows are summed and normalised,
        into a ``[len(rows), size]`` result, and ``residual`` is left untouched."""
        raise NotImplementedError


class PositionEncoding(Part):
    # Which two elements of a head form rotation pair i: False - (i, i + rotary_dim/2), the
    # half-split pairing; True - the neighbours (2i, 2i + 1).
    interleaved = False
    # Cosine and sine of every angle are multiplied by this (1: a plain rotation).  Only kernels
    # that take a magnitude honour another value; a mixer whose kernels do not must refuse it.
    magnitude = 1.0

    def rotary(self):
        """``(inv_freq, rotary_dim)``: the encoding rotates pair i of every query and key head
        (see ``interleaved``) by the angle ``position * inv_freq[i]`` (float32
        ``[rotary_dim / 2]`` on the device); ``(None, 0)`` leaves heads as they are.
        The fused norm + rotate + store kernel applies it."""
        raise NotImplementedError


class Mixer(Part):
    def cache_spec(self):
        """``PagedKV``, ``FixedState`` or ``None``."""
        return None

    def forward(self, x: torch.Tensor, step, cache) -> torch.Tensor:
        """``x[T, hidden]`` (compute dtype, already normalised) -> mixer output ``[T, hidden]``.

        ``cache`` is this run entry's view of the cache (``PagedKVView`` or
        ``FixedStateView``), or ``None``; ``cache.owner`` is False when the entry
        borrows another entry's cache and must not write it."""
        raise NotImplementedError


class FeedForward(Part):
    def forward(self, x: torch.Tensor, step) -> torch.Tensor:
        raise NotImplementedError


class Embedding(Part):
    def cache_spec(self):
        """``FixedState`` when the embedding keeps something per request (it is then handed the
        view as ``forward(step, cache)``), else None."""
        return None

    def forward(self, step) -> torch.Tensor:
        """Float32 residual rows ``[T, hidden]`` for ``step.token_ids``."""
        raise NotImplementedError

    def table(self) -> torch.Tensor:
        raise NotImplementedError


class Head(Part):
    def forward(self, x: torch.Tensor) -> torch.Tensor:
        """``x[R, hidden]`` (compute dtype) -> float32 logits ``[R, vocab]``.  A head that sets
        ``takes_deferred_norm = True`` may be handed a ``DeferredNorm`` and starts with ``project``."""
        raise NotImplementedError


class SideInput(Part):
    def forward(self, rows: torch.Tensor, step, scale: float):
        """``rows[T, hidden]``: the stream itself in the compute type, not normed.  Returns what waits
        on the stream (a tensor, ``DeferredLinear`` or ``NormedOutput``), already times ``scale``."""
        raise NotImplementedError


class DeferredLinear:
    """A block's output projection that has not run yet: ``x @ w^T``.

    A mixer or feed-forward may return this instead of a tensor; the stream then runs the
    product together with the residual add and the next norm when the norm can
    (``Norm.add_apply_linear``), which for decode-sized steps is one launch instead of two.
    ``materialize()`` runs it on its own."""

    def __init__(self, ops, x: torch.Tensor, w: torch.Tensor, out_dtype: torch.dtype):
        self.ops, self.x, self.w, self.out_dtype = ops, x, w, out_dtype

    def materialize(self) -> torch.Tensor:
        return self.ops.linear(self.x, self.w, self.out_dtype)


class NormedPair:
    """A mixer output that is not formed yet: ``scale * (norm(left) * left_w + norm(right) * right_w)``,
    the RMS norms of two branches' rows over the model width (``eps`` inside the root).

    The next norm of the stream adds it to the residual and normalises the sum in one kernel when
    it can (``takes_pairs``: its ``add_apply`` is handed this object as the block output).
    ``materialize()`` gives the float32 rows."""

    def __init__(self, ops, left, right, left_w, right_w, scale: float, eps: float):
        self.ops, self.left, self.right, self.left_w, self.right_w, self.scale, self.eps = ops, left, right, left_w, right_w, scale, eps

    def materialize(self) -> torch.Tensor:
        return self.ops.normed_pair(self.left, self.right, self.left_w, self.right_w, self.scale, self.eps)


class NormedOutput:
    """A sublayer output that is not formed yet: ``scale * norm(y) * w``, the RMS norm of its rows over
    the model width (``eps`` inside the root).  It waits on the stream as a ``NormedPair`` does, and the
    same norms take it."""

    def __init__(self, ops, y, w, scale: float, eps: float):
        self.ops, self.y, self.w, self.scale, self.eps = ops, y, w, scale, eps

    def materialize(self) -> torch.Tensor:
        return self.ops.normed_pair(self.y, None, self.w, None, self.scale, self.eps)


class DeferredNorm:
    """The normed rows a mixer or feed-forward is about to read, not computed yet:
    ``norm(residual + pending)`` of a stream.

    A part that sets ``takes_deferred_norm = True`` is handed this instead of a tensor and
    starts with ``project(ops, x, w, ...)``.  Where the block output waiting to be added is a
    product (``DeferredLinear``), the norm is an RMS norm and the kernel table has the pair
    ``linear_into_stream`` / ``linear_scaled`` (a handful of rows), the two products run with
    nothing between them: the first adds into the stream and leaves unscaled rows, the second
    applies the row scale.  Else the norm runs first, as it always did.  ``materialize()``
    gives the rows themselves."""

    def __init__(self, stream: "Stream", norm: Norm):
        self.stream, self.norm = stream, norm

    def materialize(self) -> torch.Tensor:
        return self.stream.normed(self.norm)

    def _scaled_rows(self):
        """The rows without their scale (``ScaledRows`` of the kernel table) when the block output
        waiting to be added is a product that the table can send straight into the stream;
        else None, and nothing has happened."""
        stream, norm = self.stream, self.norm
        ops = norm.env.ops
        waiting = stream.pending
        into_stream = getattr(ops, "linear_into_stream", None)
        params = norm.rms_params() if hasattr(norm, "rms_params") else None
        if isinstance(waiting, DeferredLinear) and into_stream is not None and params is not None:
            result = into_stream(waiting.x, waiting.w, stream.residual, params[0], params[1])
            if result is not None:
                stream.residual, rows = result
                stream.pending = None
                return rows
        return None

    def linear(self, w: torch.Tensor, out_dtype: torch.dtype, glu: bool = False, act=None) -> torch.Tensor:
        ops = self.norm.env.ops
        if act is not None:  # the fused pair knows the silu pair only
            return ops.linear_glu(self.stream.normed(self.norm), w, out_dtype, act[0], act[1])
        rows = self._scaled_rows()
        if rows is not None:
            return ops.linear_scaled(rows, w, out_dtype, glu)  # this product scales the rows by itself
        x = self.stream.normed(self.norm)
        return ops.linear_swiglu(x, w, out_dtype) if glu else ops.linear(x, w, out_dtype)

    def linear_short_conv(self, in_proj: torch.Tensor, taps, bias, state, step) -> torch.Tensor:
        """``ops.linear_short_conv`` of these rows (the input projection of a gated short
        convolution and the convolution behind it)."""
        ops = self.norm.env.ops
        rows = self._scaled_rows()
        return ops.linear_short_conv(rows if rows is not None else self.stream.normed(self.norm), in_proj, taps, bias, state, step)


def project(ops, x, w: torch.Tensor, out_dtype: torch.dtype, glu: bool = False, act=None) -> torch.Tensor:
    """``x @ w^T`` (or SwiGLU over the gate/up pair ``w``) for rows ``x`` that are a tensor or a
    ``DeferredNorm``.  ``act = (kind, limit)`` names another activation of a gated pair than silu
    (``ops.linear_glu``)."""
    if isinstance(x, DeferredNorm):
        return x.linear(w, out_dtype, glu, act) if act is not None else x.linear(w, out_dtype, glu)
    if act is not None:
        return ops.linear_glu(x, w, out_dtype, act[0], act[1])
    return ops.linear_swiglu(x, w, out_dtype) if glu else ops.linear(x, w, out_dtype)


class Stream:
    """The residual stream between blocks.

    ``residual`` is float32 ``[T, hidden]``.  ``pending`` is a block output not yet
    added (or a tuple of them, from a layer whose sublayers run side by side): the next norm
    adds it while it normalises (one fused kernel), which is how
    the reference closes every block (crates/shiso-engine/src/layers.rs:2476-2498)."""

    def __init__(self, residual: torch.Tensor, observer: Optional[Callable] = None):
        self.residual = residual
        self.pending: Optional[torch.Tensor] = None
        self.observer = observer  # a diagnostic: called with the stream after every ``add``
        # A block arrangement that keeps several copies of the stream (hyper-connections) holds
        # them here, float32 ``[copies, T, hidden]``; None while there is one stream, and then
        # ``residual`` stands for every copy.  ``lane_update = (y, mix, out)`` is a sublayer
        # output not yet written into the copies: the next read writes it in the same kernel.
        self.lanes: Optional[torch.Tensor] = None
        self.lane_update = None
        # The residual rows in the compute type, when a kernel that updated the residual also
        # wrote them out (a layer whose sublayers read the residual itself); dropped by ``add``.
        self.current: Optional[torch.Tensor] = None

    def rows(self, env) -> torch.Tensor:
        """The residual rows, up to date, in the compute type of ``env``: what a sublayer that
        reads the stream itself (no norm before it) is given."""
        delta = self.take_pending()
        if delta is not None:
            for d in delta if isinstance(delta, tuple) else (delta,):
                self.residual += d.to(self.residual.dtype)
            self.current = None
        if env.dtype == torch.float32:
            return self.residual
        if self.current is None:
            self.current = env.ops.unary(self.residual, "copy", env.dtype)
        return self.current

    def lane_values(self) -> Optional[torch.Tensor]:
        """The copies with the waiting update applied, computed on the side (a diagnostic);
        None while there is one stream."""
        if self.lanes is None and self.lane_update is None:
            return None
        if self.lanes is not None:
            lanes = self.lanes
        else:
            lanes = self.residual.unsqueeze(0).expand(self.lane_update[1].shape[0], -1, -1)
        if self.lane_update is None:
            return lanes.clone()
        y, mix, out = self.lane_update
        return torch.einsum("sr,std->rtd", mix.to(lanes.dtype), lanes) + out.to(lanes.dtype)[:, None, None] * y.to(lanes.dtype)[None]

    def merge_lanes(self, ops) -> None:
        """Ends the copies: ``residual`` becomes their sum (with the waiting update applied)."""
        if self.lanes is None and self.lane_update is None:
            return
        if self.lane_update is None:
            self.residual = ops.hyper_mix_sum(self.lanes, None, None, None)
        else:
            y, mix, out = self.lane_update
            self.residual = ops.hyper_mix_sum(self.lanes if self.lanes is not None else self.residual, y, mix, out)
        self.lanes = self.lane_update = None

    def normed(self, norm: Norm, deferred: bool = False):
        """The normed rows; with ``deferred`` a ``DeferredNorm`` that computes them when (and how)
        its reader wants."""
        if deferred:
            return DeferredNorm(self, norm)
        if self.pending is None:
            return norm.apply(self.residual)
        delta, self.pending = self.pending, None
        if isinstance(delta, tuple):
            if not getattr(norm, "takes_several", False):
                raise RuntimeError(f"{type(norm).__name__} adds one block output at a time, {len(delta)} are waiting")
            return norm.add_apply(self.residual, tuple(d.materialize() if isinstance(d, DeferredLinear) else d for d in delta))
        if isinstance(delta, (NormedPair, NormedOutput)) and not getattr(norm, "takes_pairs", False):
            self.residual = norm.env.ops.stream_add(self.residual, (delta.materialize(),), None)
            return norm.apply(self.residual)
        if isinstance(delta, DeferredLinear):
            fused = getattr(norm, "add_apply_linear", None)
            if fused is not None:
                return fused(self.residual, delta)
            delta = delta.materialize()
        return norm.add_apply(self.residual, delta)

    def take_pending(self, norm: Optional[Norm] = None) -> Optional[torch.Tensor]:
        """The block output still waiting to be added, as a tensor (or None); a tuple of tensors
        where a layer left several.  A ``NormedPair`` or ``NormedOutput`` stays one where ``norm`` says it
        takes those."""
        delta, self.pending = self.pending, None
        if isinstance(delta, (NormedPair, NormedOutput)):
            return delta if norm is not None and getattr(norm, "takes_pairs", False) else delta.materialize()
        if isinstance(delta, tuple):
            return tuple(d.materialize() if isinstance(d, DeferredLinear) else d for d in delta)
        if isinstance(delta, DeferredLinear):
            delta = delta.materialize()
        return delta

    def add_now(self, deltas, scale: float, env, want_rows: bool) -> Optional[torch.Tensor]:
        """``residual += scale * sum(deltas)`` at once, in float32 and in place; returns the new rows in
        the compute type of ``env`` where they are wanted (for a part that reads the stream itself)."""
        if self.pending is not None:
            raise RuntimeError("a block output is already waiting to be added to the residual")
        deltas = tuple(d.materialize() if isinstance(d, DeferredLinear) else d for d in deltas)
        self.current = env.ops.stream_add_rows(self.residual, deltas, scale, env.dtype if want_rows else None)
        if self.observer is not None:
            self.observer(self)
        return self.current

    def add(self, delta) -> None:
        if self.pending is not None:
            raise RuntimeError("a block output is already waiting to be added to the residual")
        self.pending = delta
        self.current = None
        if self.observer is not None:
            self.observer(self)


class Block(Part):
    def mixer_part(self) -> Mixer:
        raise NotImplementedError

    def forward(self, stream: Stream, step, cache) -> None:
        raise NotImplementedError


# --------------------------------------------------------------------------- registries


class Registry:
    """Name -> factory(spec, env, ...) for one kind of part."""

    def __init__(self, what: str):
        self.what = what
        self._factories: dict[str, Callable] = {}

    def register(self, kind: str, factory: Callable = None):
        def add(f):
            if kind in self._factories:
                raise ValueError(f"{self.what} {kind!r} is registered already")
            self._factories[kind] = f
            return f

        return add if factory is None else add(factory)

    def unregister(self, kind: str) -> None:
        self._factories.pop(kind, None)

    def build(self, spec: PartSpec, env: BuildEnv, *args, **kwargs):
        factory = self._factories.get(spec.kind)
        if factory is None:
            raise KeyError(
                f"no {self.what} named {spec.kind!r}; registered: {', '.join(sorted(self._factories))}"
            )
        return factory(spec, env, *args, **kwargs)

    def kinds(self) -> list[str]:
        return sorted(self._factories)


NORMS = Registry("norm")
POSITION_ENCODINGS = Registry("position encoding")
MIXERS = Registry("mixer")
FEED_FORWARDS = Registry("feed-forward")
BLOCKS = Registry("block arrangement")
EMBEDDINGS = Registry("embedding")
HEADS = Registry("head")
SIDES = Registry("side input")
