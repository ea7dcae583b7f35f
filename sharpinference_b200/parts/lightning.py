"""Linear attention whose memory decays by a constant per head ("lightning attention").

    q, k = silu(Wq h), silu(Wk h)   (heads x d) ;   v = silu(Wv h)   (heads x dv)
    S_t = a_h S_(t-1) + k_t v_t^T ;   o_t = S_t^T q_t
    y = rms(all heads side by side) * w * sigmoid(Wg h) ,   projected by Wo

A :class:`ColumnMixer` whose projection columns are ``q | k | v | g`` (padded to a multiple of 8).  ``S`` is float32
per-request state (``state_specs["S"]``), zero at a sequence's start; the activations, the powers of the decay, all sums
and the norm are float32 (``csrc/lightning.cu``).  A request that brings few rows is walked row by row; longer portions
are cut into chunks that work side by side (:class:`LightningPlanner`).
"""
from __future__ import annotations

from typing import Hashable, Sequence

import numpy as np
import torch

from ..kernels import ops
from .base import ColumnMixer, LayerSlot, StateSpec, StepContext, StepPlanData, StepPlanner, register_part
from .linear import Linear


def lightning_columns(heads: int, d: int, dv: int):
    """First column of q, k, v, g in the fused projection, and its width (a multiple of 8)."""
    col_k = heads * d
    col_v = col_k + heads * d
    col_g = col_v + heads * dv
    return 0, col_k, col_v, col_g, (col_g + heads * dv + 7) // 8 * 8


class LightningPlanner(StepPlanner):
    """Which requests of a step are walked (int32 ``walk``, left out when all are) and which are cut into chunks: int32
    ``chunks`` ``[n, 4]`` (first row, rows, request, 0), a request's one after the other, and ``spans`` ``[m, 4]``
    (request, first chunk, chunks, 0).  Which of the two a request is depends on its own rows alone."""

    WALK_ROWS_UP_TO = 32        # (one head of 128 x 128 a block: 31 us walked, 44 us as a chunk)
    key = ("lightning",)

    def plan(self, starts: Sequence[int], lengths: Sequence[int], bucket: Hashable = None) -> StepPlanData:
        walk, chunks, spans = [], [], []
        first = 0
        for b, n in enumerate(lengths):
            if n <= self.WALK_ROWS_UP_TO:
                walk.append(b)
            else:
                mine = [(first + r, min(ops.LIGHTNING_CHUNK, n - r), b, 0) for r in range(0, n, ops.LIGHTNING_CHUNK)]
                spans.append((b, len(chunks), len(mine), 0))
                chunks.extend(mine)
            first += n
        num_walk = len(walk)
        if not spans:
            walk = []
        return StepPlanData(arrays={"walk": np.asarray(walk, dtype=np.int32),
                                    "chunks": np.asarray(chunks, dtype=np.int32).reshape(-1, 4),
                                    "spans": np.asarray(spans, dtype=np.int32).reshape(-1, 4)},
                            values={"num_walk": num_walk})


@register_part("mixer", "lightning_attention")
class LightningAttention(ColumnMixer):
    graph_safe = True
    cache_spec = None

    def __init__(self, *, proj: torch.Tensor, out: torch.Tensor, norm_weight: torch.Tensor, decay: Sequence[float],
                 heads: int, dim: int, value_dim: int, eps: float, act_dtype: torch.dtype = torch.bfloat16, name: str = ""):
        """``proj`` ``[columns, H]``: rows as :func:`lightning_columns` lays them out; ``out`` ``[H, heads * value_dim]``;
        ``decay``: one number a head."""
        cols = lightning_columns(heads, dim, value_dim)
        if proj.shape[0] != cols[-1] or out.shape[1] != heads * value_dim:
            raise ValueError(f"projections have {proj.shape[0]} rows and {out.shape[1]} columns, expected {cols[-1]} and "
                             f"{heads * value_dim}")
        if len(decay) != heads or norm_weight.numel() != heads * value_dim:
            raise ValueError(f"{len(decay)} decays and a norm of {norm_weight.numel()} for {heads} heads of {value_dim}")
        if dim > ops.LIGHTNING_MAX_KEY:
            raise ValueError(f"key size {dim} is beyond the {ops.LIGHTNING_MAX_KEY} the kernels take")
        self.in_proj, self.out_proj = Linear(proj, name + "qkvg"), Linear(out, name + "o")
        self.in_columns, self.out_columns = cols[-1], heads * value_dim
        self.col_q, self.col_k, self.col_v, self.col_g, _ = cols
        powers = ops.decay_powers(decay)
        self.powers = powers if proj.device.type == "meta" else powers.to(proj.device)
        self.norm_weight, self.eps, self.act_dtype = norm_weight, float(eps), act_dtype
        self.heads, self.dim, self.value_dim = heads, dim, value_dim
        self.state_spec = None
        self.state_specs = {"S": StateSpec((heads * dim * value_dim,), torch.float32)}

    def step_planner(self, page_size: int) -> StepPlanner:
        return LightningPlanner()

    def inner(self, ctx: StepContext, slot: LayerSlot, proj: torch.Tensor, out: torch.Tensor, scale: float = 1.0) -> None:
        plan = ctx.plans[LightningPlanner.key]
        y = ops.lightning(proj, col_q=self.col_q, col_k=self.col_k, col_v=self.col_v, powers=self.powers,
                          row_offsets=ctx.row_offsets, state_slots=ctx.state_slots, state=slot.states["S"],
                          heads=self.heads, d=self.dim, dv=self.value_dim, num_requests=ctx.num_requests,
                          walk_requests=plan.walk, num_walk=plan.num_walk, chunks=plan.chunks, spans=plan.spans,
                          fast_activations=self.act_dtype == torch.bfloat16)
        n = self.heads * self.value_dim
        ops.norm_sigmoid_gate(y, proj[:, self.col_g: self.col_g + n], self.norm_weight, self.eps, out, scale=scale)
