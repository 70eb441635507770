"""Interfaces of the parts a model is put together from, and their registries.

A model is an embedding, a list of blocks, a final norm and an output head; a block
arranges a mixer, a feed-forward and their norms; a mixer may use a position
encoding.  Every part gets its sizes and constants as parameters, declares the
weights it wants by name, says what cache it needs, and runs on the rows of a step.
No part knows which model it is in.

A part kind is registered under a name in its category; a model description
(``ModelSpec``) names kinds and parameters only, so a new embedding, mixer,
feed-forward, norm, position encoding or head is added by registering it: no
framework file changes.

What a sub-layer hands to the residual stream is a *delta*: a tensor ``[rows, width]``
of the activation type, or a ``SplitSum`` -- the fp32 slices of a matrix product that
was split over k, whose sum is the delta.  A producer may return either; a consumer
that cannot add slices itself calls ``dense_delta`` first.  Nobody has to know who
comes next.
"""
from __future__ import annotations

import os
from dataclasses import dataclass, field
from typing import Any, Callable

import torch

from ..csrc import ops
from ..csrc.ops import SplitSum


# ---------------------------------------------------------------------------
# what a part is described by
# ---------------------------------------------------------------------------
@dataclass(frozen=True)
class PartSpec:
    """Kind name plus keyword parameters of one part."""
    kind: str
    params: dict = field(default_factory=dict)

    def with_params(self, **more) -> "PartSpec":
        return PartSpec(self.kind, {**self.params, **more})


def join_name(prefix: str, name: str) -> str:
    """Checkpoint name of ``name`` below ``prefix``; either may be empty (a part whose only tensor
    carries the part's own name declares it as ``""``)."""
    return f"{prefix}.{name}" if prefix and name else (prefix or name)


@dataclass
class WeightDecl:
    """One tensor a part expects from the checkpoint.

    ``name`` is relative to the part's prefix.  ``role`` decides how it is kept:
    ``matrix`` in the run's element type, ``vector`` always in fp32 (a tensor stored
    in 32 bits stays so; bf16 widens exactly), ``table_int`` in int32.  ``dest`` is
    the device storage the loader copies into, usually a slice of a packed buffer.
    ``init`` is the random-weights rule: ``normal`` ~ N(0, std), ``one_plus_normal``
    ~ 1 + N(0, 0.1), ``eye_plus_normal`` ~ I + N(0, std), ``wide_normal`` ~ N(0, 0.4), ``zeros``.
    """
    name: str
    shape: tuple[int, ...]
    role: str = "matrix"
    init: str = "normal"
    dest: torch.Tensor | None = None


# ---------------------------------------------------------------------------
# what a part may need from the cache manager
# ---------------------------------------------------------------------------
@dataclass(frozen=True)
class PagedKV:
    """Keys and values for every token (or the last ``window`` tokens), in pages.  ``v_head_dim``: the size of
    a value row where it differs from a key row's (``None``: the same).  ``values_are_keys``: a position's value is
    its key; one set of pages serves as both.  ``chunk``: positions are counted off in chunks of that many from the
    request's start, and only keys of the chunk that is being filled are needed (not together with ``window``)."""
    kv_heads: int
    head_dim: int
    window: int | None = None
    v_head_dim: int | None = None
    values_are_keys: bool = False
    chunk: int | None = None

    @property
    def value_dim(self) -> int:
        return self.head_dim if self.v_head_dim is None else self.v_head_dim

    @property
    def span(self) -> int | None:
        """The most keys a token sees; None: all before it."""
        return self.window if self.chunk is None else self.chunk

    def first_needed(self, position: int) -> int:
        """The first position whose key a token at ``position`` sees (tokens behind it see none before that either)."""
        if self.chunk is not None:
            return position - position % self.chunk
        return 0 if self.window is None else max(0, position - self.window + 1)


@dataclass(frozen=True)
class FixedState:
    """A state of fixed size per request (``numel`` elements of ``dtype``)."""
    numel: int
    dtype: torch.dtype = torch.float32


@dataclass(frozen=True)
class SeveralNeeds:
    """What a mixer made of several mixers needs: each member's own need (``None`` for one that needs nothing),
    in the members' order.  The cache manager answers with a ``SeveralViews`` in the same order."""
    needs: tuple


def flat_needs(need) -> list:
    """The paged and fixed-size needs inside ``need``, whatever its nesting."""
    if need is None:
        return []
    if isinstance(need, SeveralNeeds):
        return [x for member in need.needs for x in flat_needs(member)]
    return [need]


# ---------------------------------------------------------------------------
# run-time handles
# ---------------------------------------------------------------------------
@dataclass
class Runtime:
    """Where and in which element type a model lives."""
    device: torch.device
    dtype: torch.dtype

    def empty(self, *shape, dtype=None) -> torch.Tensor:
        return poisoned(torch.empty(*shape, dtype=dtype or self.dtype, device=self.device))


def poison_new_buffers() -> bool:
    """TESSWEAVE_POISON_BUFFERS=1 (the tests set it): every buffer that is allocated without a value --
    workspace, weight storage before loading -- is filled with NaN (integers with a large negative
    number), so that a kernel that reads what nobody wrote gives NaN instead of whatever the memory held.
    Fresh device memory is often zero, or holds the same values an earlier run left there, and hides
    such a read."""
    return os.environ.get("TESSWEAVE_POISON_BUFFERS", "0") == "1"


def poisoned(t: torch.Tensor) -> torch.Tensor:
    if poison_new_buffers():
        t.fill_(float("nan") if t.is_floating_point() else -(2 ** 30))
    return t


class Workspace:
    """Named scratch tensors that only ever grow; shared by all parts of a model.

    A buffer asked for under one name is reused by every layer, so the memory of a
    step does not grow with depth, and addresses stay fixed for CUDA graphs.
    """

    def __init__(self, device: torch.device):
        self.device = device
        self._buffers: dict[str, torch.Tensor] = {}
        self.frozen = False
        self.prefix = ""        # put before every name: a part that runs several parts side by side gives each buffers of its own

    def get(self, name: str, shape: tuple[int, ...], dtype: torch.dtype, zero: bool = False) -> torch.Tensor:
        """The buffer ``name`` with at least ``shape`` elements.  ``zero`` fills it with zeros when it
        is (re)allocated -- for state that kernels keep zero between launches, such as counters."""
        numel = 1
        for s in shape:
            numel *= int(s)
        name = self.prefix + name
        buf = self._buffers.get(name)
        if buf is None or buf.dtype != dtype or buf.numel() < numel:
            if self.frozen:
                raise RuntimeError(f"workspace buffer {name!r} would have to grow while a CUDA graph holds its address")
            if zero:
                buf = torch.zeros(max(numel, 1), dtype=dtype, device=self.device)
            else:
                buf = poisoned(torch.empty(max(numel, 1), dtype=dtype, device=self.device))
            self._buffers[name] = buf
        return buf[:numel].view(*shape)

    def reserve(self, name: str, shape: tuple[int, ...], dtype: torch.dtype) -> None:
        self.get(name, shape, dtype)

    def bytes(self) -> int:
        return sum(b.numel() * b.element_size() for b in self._buffers.values())


@dataclass
class PagedView:
    """One cache layer of a paged group, as a mixer sees it."""
    k_pages: torch.Tensor          # [pages, kv_heads, page_size, head_dim]
    v_pages: torch.Tensor
    block_table: torch.Tensor      # int32 [request slots, max blocks], -1 where no page is held
    page_size: int
    window: int | None
    host_tables: Any = None        # callable slot -> list[int], for parts that want the table on the host


@dataclass
class StateView:
    """One cache layer of fixed-size per-request state."""
    state: torch.Tensor            # [request slots, numel]


@dataclass
class SeveralViews:
    """The caches of a mixer made of several mixers, one per member (``None`` where a member needs none)."""
    views: tuple


@dataclass
class StepContext:
    """Everything a part may read about the step that is running.

    Device tensors are int32.  ``n_tokens`` rows are live; rows beyond belong to the
    padding of a fixed-size (graph) batch and have ``seq_of_token == -1``.
    """
    runtime: Runtime
    workspace: Workspace
    n_tokens: int                  # rows in this step (including padding rows)
    n_seqs: int
    token_ids: torch.Tensor        # [n_tokens]
    positions: torch.Tensor        # [n_tokens] absolute position of each row in its request
    seq_of_token: torch.Tensor     # [n_tokens] index into the per-sequence arrays, -1 = padding
    seq_slot: torch.Tensor         # [n_seqs] request slot (row of block tables and state)
    seq_q_start: torch.Tensor      # [n_seqs] first row of the sequence in this step
    seq_q_len: torch.Tensor        # [n_seqs] rows of the sequence in this step
    seq_kv_len: torch.Tensor       # [n_seqs] tokens the request holds after this step
    status: torch.Tensor           # int32 [1] error bits written by kernels
    # host copies of the per-sequence arrays, for parts that loop on the host
    host_slot: list[int] = field(default_factory=list)
    host_q_start: list[int] = field(default_factory=list)
    host_q_len: list[int] = field(default_factory=list)
    host_kv_len: list[int] = field(default_factory=list)
    max_q_len: int = 1
    max_kv_len: int = 1
    decode_only: bool = False      # every sequence brings exactly one token
    fixed_shape: bool = False      # the launch is being captured: sizes must not depend on host values of this step
    device_tokens: torch.Tensor | None = None   # int32: token ids the previous step left on the device (id -(i+1) -> [i])
    kept: dict = field(default_factory=dict)      # rows of this step that a layer leaves for later layers, by name
    upcoming_weights: torch.Tensor | None = None  # set by a block: what the part after the running one streams first


# ---------------------------------------------------------------------------
# part base classes
# ---------------------------------------------------------------------------
class Part:
    """Common behaviour: parameters in, weight declarations out."""
    graph_safe = True   # False if forward() syncs with the host or allocates

    def __init__(self, runtime: Runtime):
        self.runtime = runtime

    def weights(self) -> list[WeightDecl]:
        return []

    def redundant_names(self) -> list[str]:
        """Tensors a checkpoint may carry for this part that are not loaded because the part gets them
        another way (a tied head's copy of the embedding matrix).  Relative to the part's prefix."""
        return []

    def finalize(self) -> None:
        """Called once after every declared weight has been filled."""

    def streamed_first(self) -> torch.Tensor | None:
        """The contiguous weight this part's forward reads first and from end to end, or None.  A part that runs
        before it may ask the memory system to bring its head into L2 while its own last blocks finish."""
        return None

    def weight_bytes(self) -> int:
        seen, total = set(), 0
        for w in self.weights():
            if w.dest is not None:
                base = w.dest.untyped_storage().data_ptr()
                if (base, w.dest.storage_offset()) not in seen:
                    seen.add((base, w.dest.storage_offset()))
                    total += w.dest.numel() * w.dest.element_size()
        return total


def dense_delta(ctx: "StepContext", delta, dtype: torch.dtype, name: str = "delta.dense"):
    """``delta`` as a tensor: a ``SplitSum`` is added up (in slice order) into a workspace buffer."""
    if isinstance(delta, SplitSum):
        _, rows, width = delta.slices.shape
        return delta.dense(dtype, ctx.workspace.get(name, (rows, width), dtype))
    return delta


@dataclass(frozen=True)
class DeltaPair:
    """Two pending deltas (each a tensor or a ``SplitSum``) of sub-layers that read the same stream: their sum joins it."""
    first: object
    second: object


class Embedding(Part):
    """Turns the token ids of a step into the rows of the residual stream."""

    def forward(self, ctx: "StepContext") -> "ResidualStream":
        raise NotImplementedError

    def shared_matrix(self) -> torch.Tensor | None:
        """The [vocab, hidden] matrix an output head may share when the model ties the two, or None."""
        return None


class Head(Part):
    """Turns normalised rows into fp32 logits."""

    def forward(self, ctx: "StepContext", logits: torch.Tensor, y: torch.Tensor, n_rows: int) -> None:
        """logits[:n_rows] = head(y[:n_rows]); logits is fp32 [>= n_rows, vocab]."""
        raise NotImplementedError


class Norm(Part):
    """out = norm(resid [+ delta]); updates the fp32 residual stream in place.

    ``delta`` is None, a tensor of the activation type, a ``SplitSum``, or a ``DeltaPair`` of those.  A norm whose
    kernel adds the slices itself sets ``accepts_split_sum``, one whose kernel adds two deltas at once
    ``accepts_delta_pair``; callers go through ``apply``, which adds them up first for a norm that does not."""
    accepts_split_sum = False
    accepts_delta_pair = False

    def apply(self, ctx: "StepContext", out: torch.Tensor, resid: torch.Tensor, delta, n_rows: int,
              rows: torch.Tensor | None = None, delta_scale: float = 1.0) -> None:
        """``delta_scale``: the delta is multiplied by it (in fp32) as it joins the stream; a norm that cannot do
        that implements ``forward`` without the argument and is only ever asked for a scale of 1."""
        if isinstance(delta, DeltaPair) and not self.accepts_delta_pair:
            if delta_scale != 1.0:
                raise RuntimeError("a pair of deltas with a factor needs a norm whose kernel adds both")
            ops.add_delta(resid, delta.first, ctx.n_tokens)
            delta = delta.second
        if not self.accepts_split_sum:
            delta = dense_delta(ctx, delta, out.dtype)
        if delta_scale == 1.0:
            self.forward(ctx, out, resid, delta, n_rows, rows)
        else:
            self.forward(ctx, out, resid, delta, n_rows, rows, delta_scale=delta_scale)

    def forward(self, ctx: "StepContext", out: torch.Tensor, resid: torch.Tensor, delta, n_rows: int,
                rows: torch.Tensor | None = None, delta_scale: float = 1.0) -> None:
        raise NotImplementedError

    def apply_twice(self, ctx: "StepContext", out: torch.Tensor, other: "Norm", other_out: torch.Tensor, resid: torch.Tensor,
                    delta, n_rows: int, delta_scale: float = 1.0) -> None:
        """The delta joins the stream, and both this norm and ``other`` write their rows of it.  A kind whose kernel does
        both in one pass overrides this."""
        self.apply(ctx, out, resid, delta, n_rows, delta_scale=delta_scale)
        other.apply(ctx, other_out, resid, None, n_rows)

    def add_normed(self, ctx: "StepContext", resid: torch.Tensor, delta, n_rows: int,
                   copy: torch.Tensor | None = None) -> None:
        """resid += norm(delta), for a block that normalises what a sub-layer returns; ``copy`` (may be None)
        receives the new rows in the activation type.  ``delta`` as in ``apply``."""
        raise NotImplementedError(f"norm kind {getattr(self, 'kind', type(self).__name__)!r} cannot normalise into the residual stream")


@dataclass(frozen=True)
class RotaryPlan:
    """A rotation by ``position * inv_freq[i]`` of ``rot_dims / 2`` pairs at the start of every head: pair i is
    ``(2i, 2i + 1)`` when ``interleaved``, else ``(i, i + rot_dims / 2)``; dims from ``rot_dims`` on pass unchanged.
    With a ``magnitude`` other than 1 the rotated pairs are also scaled by it."""
    inv_freq: torch.Tensor          # fp32 [rot_dims / 2], on the device
    rot_dims: int
    interleaved: bool
    magnitude: float = 1.0          # cos and sin are both multiplied by this


class PositionEncoding(Part):
    """Encodes positions into queries and keys.

    ``apply`` rewrites the first ``n_heads`` heads of the packed rows (q heads, then k heads) in
    place; every encoding implements it, and a mixer needs to know nothing else.  An encoding that
    is a rotation by ``position * inv_freq[i]`` of the pairs ``(i, i + head_dim / 2)`` may also give
    that table through ``fused_rotary_table()``: a mixer that has a kernel which rotates while it
    does something else (writes the cache, attends) can then skip ``apply``.  ``None`` means
    "call apply()".
    """

    def apply(self, ctx: StepContext, qk: torch.Tensor, n_heads: int, head_dim: int) -> None:
        raise NotImplementedError

    def fused_rotary_table(self, head_dim: int) -> torch.Tensor | None:
        return None

    def rotary_plan(self, head_dim: int) -> RotaryPlan | None:
        """What a mixer needs to rotate inside a kernel of its own, for encodings that are a rotation of
        pairs (whole head or part of it, either pairing); ``None`` means "call apply()"."""
        return None


class Mixer(Part):
    """Mixes information between the tokens of a request (attention here)."""

    def cache_need(self) -> PagedKV | FixedState | SeveralNeeds | None:
        return None

    def forward(self, ctx: StepContext, h: torch.Tensor, cache: PagedView | StateView | SeveralViews | None,
                write_cache: bool):
        """h: [n_tokens, hidden] normalised rows.  Returns the delta for the residual stream
        (a tensor or a ``SplitSum``)."""
        raise NotImplementedError


class FeedForward(Part):
    """Token-wise transformation (dense or routed)."""

    def forward(self, ctx: StepContext, h: torch.Tensor):
        """Returns the delta for the residual stream (a tensor or a ``SplitSum``)."""
        raise NotImplementedError


class Block(Part):
    """Arrangement of a mixer and a feed-forward around the residual stream."""

    def forward(self, ctx: StepContext, stream: "ResidualStream", cache, write_cache: bool) -> None:
        raise NotImplementedError

    def parts(self) -> dict[str, Part]:
        raise NotImplementedError


@dataclass
class ResidualStream:
    """The fp32 residual rows plus a delta (tensor, ``SplitSum`` or ``DeltaPair``) the next norm still has to add.
    ``rounded``: the same rows (without the pending delta) in the activation type, if the part that wrote
    them last made that copy; whoever changes ``resid`` without renewing it sets it to None.
    ``copies``: fp32 [rows, copies, width] when a block keeps several parallel copies of the stream instead of
    ``resid``; such a block also sets ``fold``, which the model calls once behind the last block (and anyone who
    wants the single stream in between) to bring ``resid`` up to date: ``fold(ctx, stream)``.
    ``pending_scale``: what the pending delta is multiplied by when it is added (a design whose sub-layers join the
    stream through a constant factor); whoever takes ``pending`` honours it or refuses (``unscaled_pending``)."""
    resid: torch.Tensor
    pending: object = None
    pending_scale: float = 1.0
    rounded: torch.Tensor | None = None
    copies: torch.Tensor | None = None
    fold: Callable | None = None


def unscaled_pending(stream: ResidualStream, who: str):
    """The pending delta, for a block that adds it as it is; raises where the block before left one with a factor."""
    if stream.pending is not None and stream.pending_scale != 1.0:
        raise RuntimeError(f"{who}: the block before left a delta with the factor {stream.pending_scale}, which only a "
                           "block that knows such factors can add")
    return stream.pending


# ---------------------------------------------------------------------------
# registries
# ---------------------------------------------------------------------------
CATEGORIES = ("embedding", "norm", "position", "mixer", "feed_forward", "block", "head")
_REGISTRY: dict[str, dict[str, Callable[..., Part]]] = {c: {} for c in CATEGORIES}


def register_part(category: str, kind: str):
    """Class decorator: make ``kind`` buildable in ``category``."""
    if category not in _REGISTRY:
        raise KeyError(f"unknown part category {category!r}; one of {CATEGORIES}")

    def deco(cls):
        _REGISTRY[category][kind] = cls
        cls.kind = kind
        return cls
    return deco


def build_part(category: str, spec: PartSpec, runtime: Runtime, **extra) -> Part:
    try:
        cls = _REGISTRY[category][spec.kind]
    except KeyError:
        known = ", ".join(sorted(_REGISTRY.get(category, {}))) or "none"
        raise KeyError(f"no {category} part of kind {spec.kind!r} is registered (known: {known})") from None
    return cls(runtime, **spec.params, **extra)


def registered(category: str) -> list[str]:
    return sorted(_REGISTRY[category])
