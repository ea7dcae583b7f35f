"""Interfaces of the parts a layer is put together from, and the step context they run in.

A decoder layer here is a *block* that arranges a *mixer* (attention, or anything else that
moves information between positions), a *feed-forward*, *norms* and, inside the mixer, a
*position encoding*.  Every part receives its sizes and constants as constructor arguments and
its tensors from a weight source; no part knows which model it is in.  The reference decides
the same questions with per-architecture flags inside one forward pass
(src/SharpInference.Engine/ForwardPass.cs:1534-1757, flags from
src/SharpInference.Core/ModelGraph.cs:262-347); here they are parts chosen layer by layer.

Adding a part: subclass the interface below, give it a ``kind`` name with
:func:`register_part`, and use it from an architecture's builder (or a test's).  Contracts:

``Mixer.forward(ctx, slot, h) -> [T, H] float32``
    ``h`` are the normalised activations of the step's T rows in the activation dtype.
    ``slot`` is the cache manager's grant for this place in the layer schedule: the pages of its
    cache group (if ``cache_spec`` is not None) and the per-request state (if ``state_spec`` is
    not None).  The result is added to the residual stream by the block.
``FeedForward.forward(ctx, h, h32) -> [T, H] float32``
    ``h32`` is the unrounded float32 copy of ``h``, given when ``wants_fp32_input`` is true.
``Norm.apply(x, delta, rows, out_dtype, want_fp32) -> (h, h32)``
    ``x`` is the float32 residual stream; ``delta`` (float32 or None) is added to it first.
``PositionEncoding``
    either describes a rotation the attention kernel applies itself (``rotary()``), or edits q
    and k in place through ``apply(ctx, q, k)``.
"""
from __future__ import annotations

from dataclasses import dataclass, field
from types import SimpleNamespace
from typing import Any, Callable, Dict, Hashable, List, Optional, Sequence, Tuple

import torch


# ---------------------------------------------------------------------------------------
# What a mixer needs from the cache manager
# ---------------------------------------------------------------------------------------
@dataclass(frozen=True)
class CacheSpec:
    """Keys and values a mixer keeps per position, and which past positions stay visible.

    ``kind`` is ``"full"`` (every earlier position), ``"chunk"`` (positions of the same chunk of
    ``span`` positions) or ``"window"`` (the last ``span`` positions, the query's own included).
    Layers with equal specs share one group of pages and one block table per request.

    ``planes``: 2 when a page holds keys and values, 1 when it holds keys only and a value is its key row (the
    values are the keys, or both are readings of one cached latent).  ``keep_first`` (window kind): the first
    positions of a sequence stay visible whatever the window, so the pages that hold them are never given back.
    """

    kind: str
    span: int
    num_kv_heads: int
    head_dim: int
    planes: int = 2
    keep_first: int = 0

    def __post_init__(self):
        if self.kind not in ("full", "chunk", "window"):
            raise ValueError(f"cache kind '{self.kind}' is not one of full, chunk, window")
        if self.kind != "full" and self.span <= 0:
            raise ValueError(f"cache kind '{self.kind}' needs a positive span, found {self.span}")
        if self.planes not in (1, 2):
            raise ValueError(f"a page holds 1 or 2 planes, found {self.planes}")
        if self.keep_first < 0 or (self.keep_first and self.kind != "window"):
            raise ValueError(f"keep_first ({self.keep_first}) must not be negative and belongs to the window kind")

    def lowest_visible(self, pos: int) -> int:
        """The lowest position a query at ``pos`` may read."""
        if self.kind == "chunk":
            return (pos // self.span) * self.span
        if self.kind == "window":
            return max(0, pos - self.span + 1)
        return 0


@dataclass(frozen=True)
class StateSpec:
    """A tensor of fixed shape that a mixer keeps for every live request."""

    shape: Tuple[int, ...]
    dtype: torch.dtype = torch.float32


@dataclass
class LayerSlot:
    """What one entry of the layer schedule was granted by the cache manager."""

    index: int                              # place in the schedule
    layer: int                              # which block runs there
    group: Optional[int] = None             # id of the page group (key of StepContext.block_tables)
    kv: Optional[torch.Tensor] = None       # [pages, planes, kv_heads, page_size, head_dim]
    writes_cache: bool = True               # False: reads the cache that another entry writes
    state: Optional[torch.Tensor] = None    # [state_slots, *StateSpec.shape]
    page_size: int = 0
    # named per-request state of the block and its mixer (``state_specs``): name -> [state_slots, *shape]
    states: Dict[str, torch.Tensor] = field(default_factory=dict)


@dataclass
class StepContext:
    """One step's batch, as the parts see it.  Device tensors are int32."""

    num_tokens: int
    num_requests: int
    token_ids: torch.Tensor                 # [T]
    positions: torch.Tensor                 # [T] absolute position of every row
    row_request: torch.Tensor               # [T] index of the row's request within this step
    request_start: torch.Tensor             # [B] position of the request's first row in this step
    row_offsets: torch.Tensor               # [B + 1] first row of every request
    state_slots: torch.Tensor               # [B] state slot of every request
    block_tables: Dict[int, torch.Tensor]   # group id -> [B, max_blocks] page ids (-1: none)
    want_rows: Optional[torch.Tensor]       # [R] rows whose logits are wanted (None: no logits)
    slots: List[LayerSlot]                  # one per schedule entry
    # host-side copies, for grid sizing and for parts written in plain torch
    host_starts: List[int] = field(default_factory=list)
    host_lengths: List[int] = field(default_factory=list)
    host_state_slots: List[int] = field(default_factory=list)
    max_rows_per_request: int = 0
    max_context: int = 0                    # highest position + 1 over the step (an upper bound in a replayed graph)
    decode_only: bool = False               # every request brings exactly one row
    # what the mixers' step planners made of this step, by planner key: the arrays as int32 device tensors
    # (None where an array is empty) and the host-side values, as attributes (see StepPlanner)
    plans: Dict[Hashable, SimpleNamespace] = field(default_factory=dict)
    extras: Dict[str, Any] = field(default_factory=dict)
    # per-request state that belongs to the model and to no layer (``DecoderModel.state_specs``)
    model_states: Dict[str, torch.Tensor] = field(default_factory=dict)


# ---------------------------------------------------------------------------------------
# Per-step metadata that a kind of mixer brings along
# ---------------------------------------------------------------------------------------
@dataclass
class StepPlanData:
    """What a planner made of one step: int32 host arrays (any shape) that travel to the device in the
    step's one metadata copy, and host-side values (counts, bounds) that the mixer's launches use."""

    arrays: Dict[str, Any] = field(default_factory=dict)
    values: Dict[str, Any] = field(default_factory=dict)


class StepPlanner:
    """How a kind of mixer cuts a step's rows for its kernels.

    The step function knows requests, rows and block tables; how a mixer's kernels want the rows grouped
    (tiles of a prompt portion, single rows, segments of a scan) is the mixer's business.  A mixer that needs
    such metadata returns a planner from ``Mixer.step_planner(page_size)``.  Planners with equal ``key`` are
    one planner: they run once per step and every mixer with that key reads ``ctx.plans[key]``.

    ``plan(starts, lengths, bucket)`` gets, per request of the step, the position of its first row and its
    number of rows (rows of all requests lie end to end).  For decode-only steps that are replayed as a CUDA
    graph, ``bucket(starts, lengths)`` names what of the plan is baked into the graph (grid sizes, bounds):
    steps with the same number of requests and the same bucket share a graph, and ``plan`` is then called
    with that bucket and must return arrays of the same shapes, and values that hold for every such step.
    """

    key: Hashable = None

    def plan(self, starts: Sequence[int], lengths: Sequence[int], bucket: Hashable = None) -> StepPlanData:
        raise NotImplementedError

    def bucket(self, starts: Sequence[int], lengths: Sequence[int]) -> Hashable:
        return None


# ---------------------------------------------------------------------------------------
# Part interfaces
# ---------------------------------------------------------------------------------------
class Part:
    kind: str = ""


class Norm(Part):
    def apply(self, x: torch.Tensor, delta: Optional[torch.Tensor], *, rows: Optional[torch.Tensor],
              out_dtype: torch.dtype, want_fp32: bool = False):
        raise NotImplementedError


class PositionEncoding(Part):
    def rotary(self) -> Optional[Tuple[torch.Tensor, str]]:
        """``(inv_freq float32 [head_dim / 2], pairing)`` with pairing ``"interleaved"`` (pairs
        ``(2j, 2j+1)``) or ``"halves"`` (pairs ``(j, j + d/2)``) if the encoding is a rotation by
        ``position * inv_freq``; None otherwise."""
        return None

    def apply(self, ctx: StepContext, q: torch.Tensor, k: torch.Tensor) -> None:
        """Edit ``q`` [T, heads, d] and ``k`` [T, kv_heads, d] (float32) in place."""
        raise NotImplementedError


class Mixer(Part):
    cache_spec: Optional[CacheSpec] = None
    state_spec: Optional[StateSpec] = None
    # further per-request state by name (``slot.states[name]``); a block may declare ``state_specs`` too
    state_specs: Optional[Dict[str, StateSpec]] = None
    # True: ``h`` arrives as the unrounded float32 activations instead of the activation dtype
    wants_fp32_input: bool = False

    def step_planner(self, page_size: int) -> Optional[StepPlanner]:
        """The planner of this mixer's per-step metadata, or None if the step context is all it needs."""
        return None

    def step_planners(self, page_size: int) -> List[StepPlanner]:
        """All planners of this mixer: the one above, or several where a mixer is put together from mixers."""
        planner = self.step_planner(page_size)
        return [] if planner is None else [planner]

    def forward(self, ctx: StepContext, slot: LayerSlot, h: torch.Tensor) -> torch.Tensor:
        raise NotImplementedError


class ColumnMixer(Mixer):
    """A mixer that stands between two plain products: it reads columns of a projection of the layer's input and leaves
    the columns that an output projection reads (``in_columns``, ``out_columns``).  Alone, :meth:`forward` runs both
    products.  A part that holds several column mixers takes their weights over (:meth:`take_weights`), lays them side
    by side, runs one product in front of all and one behind, and calls :meth:`inner`.

    A subclass sets ``in_proj``, ``out_proj`` (``Linear``) and ``act_dtype`` and writes :meth:`inner`."""

    in_columns: int
    out_columns: int
    in_proj: Any = None
    out_proj: Any = None
    act_dtype: torch.dtype = torch.bfloat16

    def inner(self, ctx: StepContext, slot: LayerSlot, proj: torch.Tensor, out: torch.Tensor, scale: float = 1.0) -> None:
        """``proj`` float32 ``[T, in_columns]``, ``out`` ``[T, out_columns]`` in the activation dtype, either of them
        possibly a column range of a wider matrix; ``out`` receives the mixer's columns times ``scale``."""
        raise NotImplementedError

    def inner_from(self, ctx: StepContext, slot: LayerSlot, h: torch.Tensor, out: torch.Tensor) -> None:
        """From the layer's normalised input to the columns the output projection reads."""
        self.inner(ctx, slot, self.in_proj(h), out)

    def take_weights(self) -> Tuple[torch.Tensor, torch.Tensor]:
        """Hand the input and the output weight over; :meth:`forward` does not work afterwards."""
        w = (self.in_proj.weight, self.out_proj.weight)
        self.in_proj = self.out_proj = None
        return w

    def take_out_weight(self) -> torch.Tensor:
        """Hand the output weight over; the input product stays here (:meth:`inner_from`)."""
        w = self.out_proj.weight
        self.out_proj = None
        return w

    def forward(self, ctx: StepContext, slot: LayerSlot, h: torch.Tensor) -> torch.Tensor:
        out = torch.empty((h.shape[0], self.out_columns), dtype=self.act_dtype, device=h.device)
        self.inner_from(ctx, slot, h, out)
        return self.out_proj(out)


class FeedForward(Part):
    wants_fp32_input: bool = False

    def forward(self, ctx: StepContext, h: torch.Tensor, h32: Optional[torch.Tensor] = None) -> torch.Tensor:
        raise NotImplementedError


class StreamOp(Part):
    """Something done to the residual stream between two scheduled blocks (a re-injection of the embedding
    output before a pass over shared layers, for instance).  ``forward(ctx, x, pending, x0) -> (x, pending)``:
    ``x`` is the float32 residual stream, ``pending`` a float32 update not yet added to it (or None), ``x0`` the
    embedding output of the step's rows (float32, never written)."""

    graph_safe = False

    def forward(self, ctx: StepContext, x: torch.Tensor, pending: Optional[torch.Tensor], x0: torch.Tensor):
        raise NotImplementedError


class Block(Part):
    mixer: Mixer

    def forward(self, ctx: StepContext, slot: LayerSlot, x: torch.Tensor, pending: Optional[torch.Tensor]):
        """Returns ``(x, pending)``: the residual stream and a float32 update not yet added to it
        (the next norm adds it, fused)."""
        raise NotImplementedError


# ---------------------------------------------------------------------------------------
# Registry of part kinds
# ---------------------------------------------------------------------------------------
_PARTS: Dict[str, Dict[str, Callable[..., Part]]] = {
    "norm": {}, "position": {}, "mixer": {}, "feed_forward": {}, "block": {}, "stream": {},
}


def register_part(category: str, kind: str):
    """Class decorator: make ``kind`` constructible through :func:`make_part`."""
    if category not in _PARTS:
        raise ValueError(f"unknown part category '{category}' (known: {', '.join(_PARTS)})")

    def deco(cls):
        cls.kind = kind
        _PARTS[category][kind] = cls
        return cls

    return deco


def make_part(category: str, kind: str, **params) -> Part:
    try:
        cls = _PARTS[category][kind]
    except KeyError:
        known = ", ".join(sorted(_PARTS.get(category, {}))) or "(none)"
        raise ValueError(f"no {category} part of kind '{kind}' is registered; known: {known}") from None
    return cls(**params)


def part_kinds(category: str) -> List[str]:
    return sorted(_PARTS[category])
