"""The gated delta rule with a decay per key channel.

    q, k = silu(conv(Wq h)), silu(conv(Wk h))   (kv_heads x d) ;   v = silu(conv(Wv h))   (heads x dv)
    q, k as unit vectors per head, q times d^(-1/2) ;   b = sigmoid(Wb h)   per head
    g = exp(-exp(A) softplus(W2 (W1 h) + bias))   (heads x d)
    S <- g * S ;  u = b (v - S^T k) ;  S <- S + k u^T ;  o = S^T q   per head; several heads may share a q and a k
    y = rms(o) * w * sigmoid(G2 (G1 h))   head by head, projected by Wo

with ``conv`` a short causal convolution per channel.  The fused projection's columns are ``q | k | v | W1 G1 | b``; the two
low-rank maps go on through one product whose weight holds ``W2`` and ``G2`` on its diagonal (the low-rank columns are padded
to a multiple of 8).  Per-request state, float32: ``S`` (``state_specs["S"]``, a column of ``d`` numbers per value element) and
the convolutions' last ``taps - 1`` inputs (``state_specs["conv"]``).  Convolutions, unit norms, steps, decays, the state, all
its sums and the norm are float32 (``csrc/delta.cu``; a bfloat16 model's long portions form the products with the state on the
tensor cores, every operand in bfloat16 pieces of 24 bits together).  A request that brings few rows is walked row by row; longer portions
are cut into chunks (:class:`DeltaPlanner`).
"""
from __future__ import annotations

from typing import Hashable, Sequence

import numpy as np
import torch

from ..kernels import ops
from .base import LayerSlot, Mixer, StateSpec, StepContext, StepPlanData, StepPlanner, register_part
from .linear import Linear


def delta_columns(kv_heads: int, heads: int, d: int, dv: int, low: int):
    """(first low-rank column, first column of b, width padded to a multiple of 8) of the fused projection."""
    channels = 2 * kv_heads * d + heads * dv
    return channels, channels + low, (channels + low + heads + 7) // 8 * 8


class DeltaPlanner(StepPlanner):
    """``tiles`` int32 ``[n, 4]`` (first row, rows, request, 0): the step's rows in pieces for the kernel in front (left out when
    every request is a piece); ``walk``: the requests that are walked (left out when all are); ``chunks`` ``[n, 4]`` (first row,
    rows, request, 0), a request's one after the other, and ``spans`` ``[m, 4]`` (request, first chunk, chunks, 0).  Which of
    the two a request is depends on its own rows alone.  A tile has at least as many rows as a convolution looks back."""

    WALK_ROWS_UP_TO = 24        # (16 heads of 128 x 128: 16 rows 14 us walked, 19 us in chunks; 32 rows 23 and 20 us)
    TILE_ROWS = 8

    def __init__(self, taps: int, chunked: bool):
        self.tile = max(self.TILE_ROWS, taps - 1)
        self.chunked = bool(chunked)
        self.key = ("delta", self.tile, self.chunked)

    def plan(self, starts: Sequence[int], lengths: Sequence[int], bucket: Hashable = None) -> StepPlanData:
        tiles, walk, chunks, spans = [], [], [], []
        first = 0
        for b, n in enumerate(lengths):
            tiles.extend((first + r, min(self.tile, n - r), b, 0) for r in range(0, n, self.tile))
            if n <= self.WALK_ROWS_UP_TO or not self.chunked:
                walk.append(b)
            else:
                spans.append((b, len(chunks), (n + ops.DELTA_CHUNK - 1) // ops.DELTA_CHUNK, 0))
                chunks.extend((first + r, min(ops.DELTA_CHUNK, n - r), b, 0) for r in range(0, n, ops.DELTA_CHUNK))
            first += n
        num_walk, walk_rows = len(walk), max((lengths[b] for b in walk), default=0)
        if not spans:
            walk = []
        if len(tiles) == len(lengths):
            tiles = []
        return StepPlanData(arrays={"tiles": np.asarray(tiles, dtype=np.int32).reshape(-1, 4),
                                    "walk": np.asarray(walk, dtype=np.int32),
                                    "chunks": np.asarray(chunks, dtype=np.int32).reshape(-1, 4),
                                    "spans": np.asarray(spans, dtype=np.int32).reshape(-1, 4)},
                            values={"num_walk": num_walk, "walk_rows": walk_rows})


@register_part("mixer", "channel_delta")
class ChannelDelta(Mixer):
    graph_safe = True
    cache_spec = None

    def __init__(self, *, proj: Linear, up: Linear, out: Linear, conv_weight: torch.Tensor, dt_bias: torch.Tensor,
                 a_log: torch.Tensor, norm_weight: torch.Tensor, heads: int, kv_heads: int, dim: int, value_dim: int, low: int,
                 eps: float, act_dtype: torch.dtype = torch.bfloat16):
        """``proj``: rows as :func:`delta_columns` lays them out; ``up [heads * (dim + value_dim), low]``: from the low-rank
        columns to the decay's and the gate's; ``conv_weight`` float32 ``[taps, channels]``, the last tap the current
        token's."""
        if heads % kv_heads:
            raise ValueError(f"heads ({heads}) must be a multiple of kv heads ({kv_heads})")
        channels, _, width = delta_columns(kv_heads, heads, dim, value_dim, low)
        if proj.out_features != width or out.in_features != heads * value_dim:
            raise ValueError(f"projections have {proj.out_features} rows and {out.in_features} columns, expected {width} and "
                             f"{heads * value_dim}")
        if (up.out_features, up.in_features) != (heads * (dim + value_dim), low):
            raise ValueError(f"the low-rank product is [{up.out_features}, {up.in_features}], expected "
                             f"[{heads * (dim + value_dim)}, {low}]")
        if conv_weight.dim() != 2 or conv_weight.shape[1] != channels or conv_weight.shape[0] < 1:
            raise ValueError(f"the convolution is {tuple(conv_weight.shape)}, expected [taps, {channels}]")
        if dt_bias.numel() != heads * dim or a_log.numel() != heads or norm_weight.numel() != value_dim:
            raise ValueError("the decay's bias, A_log or the norm's weight disagree with heads, key or value size")
        if dim > ops.DELTA_MAX_KEY:
            raise ValueError(f"key size {dim} is beyond the {ops.DELTA_MAX_KEY} the kernels take")
        self.proj, self.up, self.out = proj, up, out
        self.conv_weight, self.dt_bias, self.a_log, self.norm_weight = conv_weight, dt_bias, a_log, norm_weight
        self.heads, self.kv_heads, self.dim, self.value_dim, self.low = heads, kv_heads, dim, value_dim, low
        self.taps, self.eps, self.act_dtype = int(conv_weight.shape[0]), float(eps), act_dtype
        self.state_specs = {"S": StateSpec((ops.delta_state_floats(heads, dim, value_dim),), torch.float32)}
        if self.taps > 1:
            self.state_specs["conv"] = StateSpec(((self.taps - 1) * channels,), torch.float32)
        self._planner = DeltaPlanner(self.taps, dim <= ops.DELTA_MAX_CHUNK_KEY)

    def step_planner(self, page_size: int) -> StepPlanner:
        return self._planner

    def forward(self, ctx: StepContext, slot: LayerSlot, h: torch.Tensor) -> torch.Tensor:
        plan = ctx.plans[self._planner.key]
        sizes = dict(kv_heads=self.kv_heads, heads=self.heads, d=self.dim, dv=self.value_dim)
        qkv, beta, low = ops.delta_prep(self.proj(h), conv_weight=self.conv_weight, conv_state=slot.states.get("conv"),
                                        row_offsets=ctx.row_offsets, state_slots=ctx.state_slots, tiles=plan.tiles, low=self.low,
                                        act_dtype=self.act_dtype, **sizes)
        z = self.up(low)                                             # [T, decay | gate] float32
        n = self.heads * self.dim
        y = ops.delta_rule(qkv, beta, z[:, :n], dt_bias=self.dt_bias, a_log=self.a_log, row_offsets=ctx.row_offsets,
                           state_slots=ctx.state_slots, state=slot.states["S"], num_requests=ctx.num_requests,
                           walk_requests=plan.walk, num_walk=plan.num_walk, chunks=plan.chunks, spans=plan.spans,
                           max_rows=plan.walk_rows, split=self.act_dtype == torch.bfloat16, **sizes)
        return self.out(ops.head_norm_gate(y, z[:, n:], self.norm_weight, self.eps, self.heads, self.act_dtype))
