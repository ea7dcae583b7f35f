"""Two mixers side by side between one product in front and one behind.

``ScaledBranches``: ``left_scale * left(h) + right_scale * right(h)`` for two :class:`ColumnMixer` parts that read the same
input.  Their input weights are one matrix (rows of the left, then of the right), their output weights one matrix whose
inner size is both branches' columns, so the sum of the two outputs is formed inside the output product; the factors
multiply a branch's columns where they are written (in float32, before they are rounded to the activation dtype).  The
pair owns the cache of whichever branch keeps keys and values and the state of both (names prefixed ``left.`` /
``right.``, as :class:`BranchPair` has it).
"""
from __future__ import annotations

from typing import List

import torch

from .base import ColumnMixer, LayerSlot, StepContext, StepPlanner, register_part
from .linear import Linear
from .mamba import BranchPair
from .side import fork, join


def pad_columns(n: int) -> int:
    """Columns of a segment inside a wider product: a multiple of 8, so that the next one starts on 16 bytes."""
    return (n + 7) // 8 * 8


def side_by_side(weights) -> torch.Tensor:
    """Output weights ``[H, n_i]`` as one ``[H, sum of pad_columns(n_i)]``, zero columns behind each."""
    H = weights[0].shape[0]
    wide = torch.zeros((H, sum(pad_columns(w.shape[1]) for w in weights)), dtype=weights[0].dtype, device=weights[0].device)
    at = 0
    for w in weights:
        wide[:, at: at + w.shape[1]] = w
        at += pad_columns(w.shape[1])
    return wide


@register_part("mixer", "scaled_branches")
class ScaledBranches(ColumnMixer):
    def __init__(self, *, left: ColumnMixer, right: ColumnMixer, left_scale: float = 1.0, right_scale: float = 1.0,
                 act_dtype: torch.dtype = torch.bfloat16, name: str = ""):
        if left.cache_spec is not None and right.cache_spec is not None:
            raise ValueError("only one branch of a pair may keep keys and values")
        if left.in_columns % 8 or right.in_columns % 8:
            raise ValueError("a branch's projection columns come in multiples of 8")
        self.left, self.right = left, right
        self.left_scale, self.right_scale, self.act_dtype = float(left_scale), float(right_scale), act_dtype
        self.cache_spec = left.cache_spec if left.cache_spec is not None else right.cache_spec
        (lin, lout), (rin, rout) = left.take_weights(), right.take_weights()
        self.in_proj = Linear(torch.cat([lin, rin], dim=0).contiguous(), name + "left|right")
        self.out_proj = Linear(side_by_side([lout, rout]), name + "left.o|right.o")
        self.in_columns = left.in_columns + right.in_columns
        self._right_at = pad_columns(left.out_columns)
        self.out_columns = self._right_at + pad_columns(right.out_columns)
        self.state_spec = None
        self.state_specs = {prefix + name: spec for prefix, m in (("left.", left), ("right.", right))
                            for name, spec in (m.state_specs or {}).items()}
        self.graph_safe = bool(getattr(left, "graph_safe", False) and getattr(right, "graph_safe", False))

    def step_planners(self, page_size: int) -> List[StepPlanner]:
        return self.left.step_planners(page_size) + self.right.step_planners(page_size)

    def _branch(self, ctx, slot, m: ColumnMixer, prefix: str, proj, out, at: int, col: int, scale: float) -> None:
        m.inner(ctx, BranchPair._branch_slot(slot, prefix, m), proj[:, at: at + m.in_columns],
                out[:, col: col + m.out_columns], scale=scale)
        gap = pad_columns(m.out_columns) - m.out_columns
        if gap:                                            # the output weight has zero columns there: no NaN may stand in them
            out[:, col + m.out_columns: col + m.out_columns + gap].zero_()

    def inner(self, ctx: StepContext, slot: LayerSlot, proj: torch.Tensor, out: torch.Tensor, scale: float = 1.0) -> None:
        # the branches meet in the output product: the right one runs on a stream of its own
        side = fork(proj.device, "branch", ctx.decode_only)
        with torch.cuda.stream(side):
            self._branch(ctx, slot, self.right, "right.", proj, out, self.left.in_columns, self._right_at,
                         scale * self.right_scale)
        self._branch(ctx, slot, self.left, "left.", proj, out, 0, 0, scale * self.left_scale)
        join(side)
