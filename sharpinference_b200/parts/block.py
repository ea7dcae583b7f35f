"""The arrangement of a layer's parts around the residual stream.

``PreNormBlock`` is the reference's order (src/SharpInference.Engine/ForwardPass.cs:1557-1714):
``x += mixer(norm1(x))``, then ``x += ffn(norm2(x))``.  The residual stream is float32; each
residual add is fused into the norm that follows it, so a block returns its feed-forward output
as ``pending`` and the next block's first norm (or the model's last) adds it.  A layer without a feed-forward
(``ffn=None``) leaves its mixer's output pending instead.

``ParallelBlock`` has one norm whose output both sublayers read: ``h = norm(x)``,
``x += mixer(h) + ffn(h)``; the feed-forward may be absent.  The sum of the two outputs is the
``pending`` update.

``ParallelPairBlock`` has two norms of the same stream: ``x += mixer(norm1(x)) + ffn(norm2(x))``.  Two RMS norms with one
``eps`` are one kernel.  Where the mixer and the feed-forward both end in a plain product (a :class:`ColumnMixer` beside a
feed-forward with ``out_columns``), their inner columns lie side by side in one matrix and one product forms the sum of
both outputs.

``SandwichBlock`` norms what a sublayer returns as well: ``x += scale1 * post1(mixer(norm1(x)))``, ``x += scale2 *
post2(ffn(norm2(x)))``, and may end with a token's own vector through a gate that reads the stream (:class:`TokenSide`).
All updates are :class:`NormedUpdate`: one kernel norms a sublayer's output, adds it and norms the stream for whatever
reads it next.
"""
from __future__ import annotations

from typing import Optional

import torch

from ..kernels import ops
from .base import Block, ColumnMixer, FeedForward, LayerSlot, Mixer, Norm, StepContext, register_part
from .branches import side_by_side, pad_columns
from .linear import Linear
from .norm import NormedUpdate, RMSNorm
from .side import fork, join
from .token_side import TokenSide


@register_part("block", "prenorm")
class PreNormBlock(Block):
    def __init__(self, *, mixer_norm: Norm, mixer: Mixer, ffn_norm: Optional[Norm], ffn: Optional[FeedForward],
                 act_dtype: torch.dtype = torch.bfloat16):
        self.mixer_norm, self.mixer, self.ffn_norm, self.ffn = mixer_norm, mixer, ffn_norm, ffn
        self.act_dtype = act_dtype

    def forward(self, ctx: StepContext, slot: LayerSlot, x: torch.Tensor, pending: Optional[torch.Tensor]):
        h, _ = self.mixer_norm.apply(x, pending, rows=None, out_dtype=self.act_dtype)
        mixed = self.mixer.forward(ctx, slot, h)
        if self.ffn is None:
            return x, mixed
        h, h32 = self.ffn_norm.apply(x, mixed, rows=None, out_dtype=self.act_dtype,
                                     want_fp32=self.ffn.wants_fp32_input)
        return x, self.ffn.forward(ctx, h, h32)


@register_part("block", "parallel")
class ParallelBlock(Block):
    def __init__(self, *, norm: Norm, mixer: Mixer, ffn: Optional[FeedForward], act_dtype: torch.dtype = torch.bfloat16):
        self.norm, self.mixer, self.ffn = norm, mixer, ffn
        self.act_dtype = act_dtype

    def forward(self, ctx: StepContext, slot: LayerSlot, x: torch.Tensor, pending: Optional[torch.Tensor]):
        want32 = self.ffn is not None and self.ffn.wants_fp32_input
        h, h32 = self.norm.apply(x, pending, rows=None, out_dtype=self.act_dtype, want_fp32=want32)
        mixed = self.mixer.forward(ctx, slot, h)
        if self.ffn is None:
            return x, mixed
        if getattr(self.ffn, "adds_to", False):          # the feed-forward's last kernel adds the mixer's output in
            return x, self.ffn.forward(ctx, h, h32, add_to=mixed)
        return x, ops.add(mixed, self.ffn.forward(ctx, h, h32), out=mixed)


@register_part("block", "parallel_pair")
class ParallelPairBlock(Block):
    def __init__(self, *, mixer_norm: Norm, mixer: Mixer, ffn_norm: Optional[Norm], ffn: Optional[FeedForward],
                 act_dtype: torch.dtype = torch.bfloat16):
        self.mixer_norm, self.mixer, self.ffn_norm, self.ffn, self.act_dtype = mixer_norm, mixer, ffn_norm, ffn, act_dtype
        self._pair_norm = (isinstance(mixer_norm, RMSNorm) and isinstance(ffn_norm, RMSNorm)
                           and mixer_norm.eps == ffn_norm.eps)
        self.joint_out = None
        if ffn is not None and isinstance(mixer, ColumnMixer) and hasattr(ffn, "take_out_weight"):
            self.joint_out = Linear(side_by_side([mixer.take_out_weight(), ffn.take_out_weight()]), "mixer.o|mlp.down")
            self._ffn_at = pad_columns(mixer.out_columns)

    def _norms(self, x: torch.Tensor, pending: Optional[torch.Tensor], want32: bool):
        if self._pair_norm:
            return ops.add_rmsnorm_pair(x, pending, self.mixer_norm.weight, self.ffn_norm.weight, self.mixer_norm.eps,
                                        self.act_dtype, want_fp32=want32)
        h1, _ = self.mixer_norm.apply(x, pending, rows=None, out_dtype=self.act_dtype)
        h2, h32 = self.ffn_norm.apply(x, None, rows=None, out_dtype=self.act_dtype, want_fp32=want32)
        return h1, h2, h32

    def forward(self, ctx: StepContext, slot: LayerSlot, x: torch.Tensor, pending: Optional[torch.Tensor]):
        if self.ffn is None:
            h, _ = self.mixer_norm.apply(x, pending, rows=None, out_dtype=self.act_dtype)
            return x, self.mixer.forward(ctx, slot, h)
        h1, h2, h32 = self._norms(x, pending, self.ffn.wants_fp32_input)
        # the mixer and the feed-forward meet in the last product or sum: the mixer runs on a stream of its own
        side = fork(x.device, "mixer", ctx.decode_only)
        if self.joint_out is not None:
            cols = torch.empty((x.shape[0], self.joint_out.in_features), dtype=self.act_dtype, device=x.device)
            with torch.cuda.stream(side):
                if self._ffn_at > self.mixer.out_columns:
                    cols[:, self.mixer.out_columns: self._ffn_at].zero_()
                self.mixer.inner_from(ctx, slot, h1, cols[:, : self.mixer.out_columns])
            self.ffn.inner(ctx, h2, cols[:, self._ffn_at:])
            join(side)
            return x, self.joint_out(cols)
        with torch.cuda.stream(side):
            mixed = self.mixer.forward(ctx, slot, h1)
        if getattr(self.ffn, "joins", False):              # adds the mixer's output in its last kernel, and waits for it there
            return x, self.ffn.forward(ctx, h2, h32, add_to=mixed, add_ready=side)
        y = self.ffn.forward(ctx, h2, h32)
        join(side)
        return x, ops.add(mixed, y, out=mixed)


@register_part("block", "sandwich")
class SandwichBlock(Block):
    """``mixer_post`` / ``ffn_post``: the weights of the norms behind the sublayers; ``mixer_scale`` / ``ffn_scale``: a factor
    per element of the stream (None: none), formed into the weights once, in float32.  ``side``: the layer's
    :class:`TokenSide` (None: none)."""

    def __init__(self, *, mixer_norm: RMSNorm, mixer: Mixer, mixer_post: RMSNorm, mixer_scale: Optional[torch.Tensor] = None,
                 ffn_norm: Optional[RMSNorm] = None, ffn: Optional[FeedForward] = None, ffn_post: Optional[RMSNorm] = None,
                 ffn_scale: Optional[torch.Tensor] = None, side: Optional[TokenSide] = None,
                 act_dtype: torch.dtype = torch.bfloat16):
        if (ffn is None) != (ffn_norm is None) or (ffn is None) != (ffn_post is None):
            raise ValueError("a feed-forward comes with the norms before and behind it, and only then")
        self.mixer_norm, self.mixer, self.ffn_norm, self.ffn, self.side = mixer_norm, mixer, ffn_norm, ffn, side
        self.act_dtype = act_dtype

        def scaled(norm: RMSNorm, scale):
            return norm.weight if scale is None else (norm.weight * scale.to(torch.float32)).contiguous()
        self.mixer_weight, self.mixer_eps = scaled(mixer_post, mixer_scale), mixer_post.eps
        if ffn is not None:
            self.ffn_weight, self.ffn_eps = scaled(ffn_post, ffn_scale), ffn_post.eps

    def forward(self, ctx: StepContext, slot: LayerSlot, x: torch.Tensor, pending):
        h, _ = self.mixer_norm.apply(x, pending, rows=None, out_dtype=self.act_dtype)
        pending = NormedUpdate(self.mixer.forward(ctx, slot, h), self.mixer_weight, self.mixer_eps)
        if self.ffn is not None:
            h, h32 = self.ffn_norm.apply(x, pending, rows=None, out_dtype=self.act_dtype, want_fp32=self.ffn.wants_fp32_input)
            pending = NormedUpdate(self.ffn.forward(ctx, h, h32), self.ffn_weight, self.ffn_eps)
        if self.side is not None:
            pending = self.side.update(ctx, x, pending)
        return x, pending

    def traced_stream(self, x: torch.Tensor, pending) -> torch.Tensor:
        return x + pending.value()
