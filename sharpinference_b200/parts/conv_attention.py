"""Grouped-query attention over convolved projections, gated per head.

    q, k, v = Wq h, Wk h, Wv h ;   every channel of them:  y_t = sum_j w_j u_(t - taps + 1 + j)   (zeros before the start)
    the first ``rot_dims`` elements of every head of q and k turn by the position
    o = softmax over the earlier positions of (q . k * scale), times v
    head h of o is multiplied by sigmoid((Wg h)_h), the heads side by side are projected by Wo

A :class:`ColumnMixer`: the fused projection's columns are ``q | k | v | g`` (padded to a multiple of 8), unpadded heads.
One kernel (``sharpi_qkv_conv``) convolves, rotates, stores q and writes k and v into the pages, padding the heads there
to the one size that pages and attention kernels know; one kernel gates the heads and lays them side by side.  Pages,
masks, step planner and attention kernels are :class:`PagedAttention`'s.  The last ``taps - 1`` projected values of a
sequence are per-request state (``state_specs["conv"]``), float32.
"""
from __future__ import annotations

from typing import Optional

import torch

from ..kernels import ops
from .attention import PagedAttention, _PAIRING_CODE
from .base import CacheSpec, ColumnMixer, LayerSlot, PositionEncoding, StateSpec, StepContext, register_part
from .linear import Linear


def conv_attention_columns(heads: int, kv_heads: int, key_dim: int, value_dim: int):
    """(columns of q | k | v, columns in all: the gate's ``heads`` behind them, padded to a multiple of 8)."""
    channels = (heads + kv_heads) * key_dim + kv_heads * value_dim
    return channels, (channels + heads + 7) // 8 * 8


@register_part("mixer", "conv_attention")
class ConvAttention(ColumnMixer, PagedAttention):
    def __init__(self, *, proj: torch.Tensor, out: torch.Tensor, conv_weight: torch.Tensor, num_heads: int,
                 num_kv_heads: int, key_dim: int, value_dim: int, softmax_scale: float,
                 position: Optional[PositionEncoding] = None, mask: str = "full", span: int = 0,
                 act_dtype: torch.dtype = torch.bfloat16, name: str = ""):
        """``proj`` ``[columns, H]``: rows as :func:`conv_attention_columns` lays them out; ``out`` ``[H, heads *
        value_dim]``; ``conv_weight`` float32 ``[taps, channels]``, the last tap the current token's."""
        channels, columns = conv_attention_columns(num_heads, num_kv_heads, key_dim, value_dim)
        if num_heads % num_kv_heads:
            raise ValueError(f"heads ({num_heads}) must be a multiple of kv heads ({num_kv_heads})")
        if min(key_dim, value_dim) <= 0 or max(key_dim, value_dim) > 1024:
            raise ValueError(f"head sizes {key_dim} (keys) and {value_dim} (values) must be 1 .. 1024")
        if proj.shape[0] != columns or out.shape[1] != num_heads * value_dim:
            raise ValueError(f"projections have {proj.shape[0]} rows and {out.shape[1]} columns, expected {columns} and "
                             f"{num_heads * value_dim}")
        if conv_weight.dim() != 2 or conv_weight.shape[1] != channels or conv_weight.shape[0] < 1:
            raise ValueError(f"the convolution is {tuple(conv_weight.shape)}, expected [taps, {channels}]")
        self.rot_dims, self.inv_freq, self.inv_freq_low, self.pairing = 0, None, None, ops.ROPE_HALVES
        if position is not None:
            rot = position.rotary()
            if rot is None:
                raise ValueError("the convolution kernel takes rotary (or no) position encodings only")
            if getattr(position, "amplitude", 1.0) != 1.0:
                raise ValueError("a rotation with an amplitude is not built for this mixer")
            self.inv_freq, self.pairing = rot[0], _PAIRING_CODE[rot[1]]
            self.inv_freq_low = getattr(position, "inv_freq_low", None)
            self.rot_dims = 2 * rot[0].numel()
            if self.rot_dims > key_dim:
                raise ValueError(f"{self.rot_dims} rotated elements exceed the key size {key_dim}")
        D = max(key_dim, value_dim)
        D = (D + 15) // 16 * 16 if D <= 128 else D + (D & 1)
        self.in_proj, self.out_proj = Linear(proj, name + "qkvg"), Linear(out, name + "o")
        self.in_columns, self.out_columns = columns, num_heads * value_dim
        self.conv_weight, self.taps, self.channels = conv_weight, conv_weight.shape[0], channels
        self.num_heads, self.num_kv_heads, self.key_dim, self.value_dim, self.head_dim = (num_heads, num_kv_heads, key_dim,
                                                                                          value_dim, D)
        self.softmax_scale, self.act_dtype, self.position = float(softmax_scale), act_dtype, position
        self.cache_spec = CacheSpec(mask, span if mask != "full" else 0, num_kv_heads, D)
        self.state_spec = None
        self.state_specs = ({"conv": StateSpec(((self.taps - 1) * channels,), torch.float32)} if self.taps > 1 else {})
        # what the shared attention launch asks for beyond this
        self.softcap, self.sinks, self.values_are_keys, self.keep_first, self.distance_bias = 0.0, None, False, 0, None
        self._general_attention = False
        self.graph_safe = True

    def inner(self, ctx: StepContext, slot: LayerSlot, proj: torch.Tensor, out: torch.Tensor, scale: float = 1.0) -> None:
        plan = ctx.plans[("paged_attention", self.prefill_tile_rows(slot.page_size))]
        table = ctx.block_tables[slot.group]
        T, nq, C = ctx.num_tokens, self.num_heads, self.channels
        q = torch.empty((T, nq, self.head_dim), dtype=self.act_dtype, device=proj.device)
        ops.qkv_conv(proj[:, :C], q, slot.kv, weight=self.conv_weight, state=slot.states.get("conv"),
                     positions=ctx.positions, row_req=ctx.row_request, row_offsets=ctx.row_offsets,
                     state_slots=ctx.state_slots, block_table=table, nq=nq, nkv=self.num_kv_heads, D=self.head_dim,
                     key_dim=self.key_dim, value_dim=self.value_dim, page_size=slot.page_size, inv_freq=self.inv_freq,
                     inv_freq_low=self.inv_freq_low, rot_dims=self.rot_dims, pairing=self.pairing)
        o = self._attend(ctx, slot, plan, table, q)
        ops.gate_heads(o, proj[:, C: C + nq], out, heads=nq, D=self.head_dim, dv=self.value_dim, scale=scale)
