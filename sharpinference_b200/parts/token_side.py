"""What a token brings along beside its embedding row: learned positions, and a small vector of its own for every layer.

``TableWithPositions``: ``x = embed[token] * scale + pos[position]``, a learned vector per position (of which there are as
many as the table has rows; the engine refuses longer sequences).

``TokenSide``: a table holds ``dim`` numbers per token and layer.  Behind a layer's feed-forward, with ``e`` the layer's slice
of the token's row,

    g = gelu_tanh(G x) * e ;   x += rms(P g) * w

``G [dim, H]`` reads the bare stream, ``P [H, dim]`` goes back.  The update before it is added, and the stream rounded for the
product, in one kernel; the gate is one more; the update that results is normed and added by whatever norm comes next.
"""
from __future__ import annotations

import torch

from ..kernels import ops
from .base import Part, StepContext
from .linear import Linear
from .norm import NormedUpdate


class TableWithPositions(Part):
    graph_safe = True
    state_specs = None

    def __init__(self, *, embed: torch.Tensor, pos: torch.Tensor, scale: float = 1.0):
        if pos.dim() != 2 or pos.shape[1] != embed.shape[1]:
            raise ValueError(f"the position table is {tuple(pos.shape)}, the embedding {tuple(embed.shape)}")
        self.embed, self.pos, self.scale = embed, pos, float(scale)

    @property
    def max_positions(self) -> int:
        return self.pos.shape[0]

    def forward(self, ctx: StepContext) -> torch.Tensor:
        return ops.embed_pos(ctx.token_ids, ctx.positions, self.embed, self.pos, self.scale)


class TokenSide(Part):
    def __init__(self, *, table: torch.Tensor, column: int, dim: int, gate: Linear, proj: Linear, norm_weight: torch.Tensor,
                 eps: float, act_dtype: torch.dtype = torch.bfloat16):
        """``table [vocab, *]``: the layer's slice starts at ``column``.  ``gate`` may have more than ``dim`` rows and ``proj`` as
        many columns: padding that stays zero."""
        if column < 0 or column + dim > table.shape[1] or gate.out_features < dim or proj.in_features != gate.out_features:
            raise ValueError(f"columns {column} .. {column + dim} of a table {tuple(table.shape)}, a gate of {gate.out_features} "
                             f"rows and a projection of {proj.in_features} columns do not fit together")
        if proj.out_features != gate.in_features or norm_weight.numel() != proj.out_features:
            raise ValueError("the side projection and its norm must have the stream's width")
        self.table, self.column, self.dim, self.gate, self.proj = table, int(column), int(dim), gate, proj
        self.norm_weight, self.eps, self.act_dtype = norm_weight, float(eps), act_dtype

    def update(self, ctx: StepContext, x: torch.Tensor, pending: NormedUpdate) -> NormedUpdate:
        """Adds ``pending`` to ``x`` and returns the side input's own update."""
        xa, _ = ops.add_normed(x, pending.y, pending.weight, None, pending.eps, self.act_dtype)
        g = ops.side_gate(self.gate(xa), ctx.token_ids, self.table, self.column, self.dim, self.act_dtype)
        return NormedUpdate(self.proj(g), self.norm_weight, self.eps)
