"""The Radupel architecture, put together from parts, and its tensor names.

A decoder of parallel layers with two norms, ``x += mixer(norm1(x)) + ff(norm2(x))`` (:class:`ParallelPairBlock`), of which
a span may run several times with the same weights; before every such pass but the first the embedding output is added
to the stream (:class:`AddInput`).  Logits come from the embedding table and are capped by ``cap tanh(y / cap)``.

The mixer of every layer (``config.layers[i]``, each with sizes of its own) is :class:`ScaledBranches`: on the left
:class:`ConvAttention` (a short convolution on every channel of q, k and v, a rotation of the heads' leading elements in
the halves layout, a sigmoid gate per head), on the right :class:`LightningAttention` (linear attention with a constant
decay per head, a norm over all heads and an element-wise gate), each times a constant.

The feed-forward is absent, a dense gated network with biases (:class:`DenseSwiGLU`; its last product is one with the
mixer's) or a mixture routed by a softmax over all experts in groups, with identity experts, clamped gates and a gated
shared expert (:class:`MoESoftmaxGroups`).

Tensor names (linear weights ``[out, in]``): ``embed``, ``final.norm``; per layer ``l<i>.norm{1,2}``;
``l<i>.mix.left.{q,k,v}`` with ``.conv [channels, taps]`` each, ``l<i>.mix.left.{g,o}``, ``l<i>.mix.right.{q,k,v,g,o,norm}``;
``l<i>.mlp.{gate,up,down}`` with ``.b`` each, or ``l<i>.mlp.e<j>.{gate,up,down}``, ``l<i>.mlp.{router,correction}``,
``l<i>.mlp.shared.{gate,up,down,sg}``.
"""
from __future__ import annotations

import torch

from ..config.radupel import RadupelConfig, RadupelLayer
from ..parts import (AddInput, ConvAttention, DenseSwiGLU, GroupedLinear, LightningAttention, Linear, MoESoftmaxGroups,
                     ParallelPairBlock, RMSNorm, RotaryEncoding, ScaledBranches, conv_attention_columns,
                     leading_rotary_inv_freq_parts, lightning_columns)
from ..registry import register_architecture
from ..weights.source import WeightSource
from .model import DecoderModel, ScheduleEntry
from .notedra import _cat


def _padded(rows, count: int) -> torch.Tensor:
    """The rows of several matrices one after the other, zero rows behind them up to ``count``."""
    have = sum(t.shape[0] for t in rows)
    if have < count:
        rows = rows + [torch.zeros((count - have, rows[0].shape[1]), dtype=rows[0].dtype, device=rows[0].device)]
    return _cat(rows)


def _attention(c: RadupelConfig, layer: RadupelLayer, p: str, weights: WeightSource, act) -> ConvAttention:
    a, W = layer.left, c.width
    H, G, d, dv = a.heads, a.kv_heads, a.dim, a.vdim
    rows = [weights.matrix(p + "q", (H * d, W)), weights.matrix(p + "k", (G * d, W)), weights.matrix(p + "v", (G * dv, W))]
    stored = [(s, n) for s, n in (("q", H * d), ("k", G * d), ("v", G * dv))]
    if a.conv > 1 or weights.stored(p + "q.conv") is not False:
        taps = torch.cat([weights.vector(f"{p}{s}.conv", (n, a.conv), init="normal") for s, n in stored], dim=0)
    else:                                                # one tap and none stored: the projections as they are
        taps = torch.ones((sum(n for _, n in stored), 1), dtype=torch.float32, device=weights.device)
    rows.append(weights.matrix(p + "g", (H, W)))
    out = weights.matrix(p + "o", (W, H * dv))
    position = None
    if a.rot_dims:
        high, low = leading_rotary_inv_freq_parts(a.rot_dims, a.rot_base)
        if weights.device.type != "meta":
            high, low = high.to(weights.device), low.to(weights.device)
        position = RotaryEncoding(high, "halves", a.rot_dims, inv_freq_low=low)
    return ConvAttention(proj=_padded(rows, conv_attention_columns(H, G, d, dv)[1]), out=out,
                         conv_weight=taps.t().contiguous(), num_heads=H, num_kv_heads=G, key_dim=d, value_dim=dv,
                         softmax_scale=a.scale, position=position, act_dtype=act, name=p)


def _linear(c: RadupelConfig, layer: RadupelLayer, p: str, weights: WeightSource, act) -> LightningAttention:
    s, W = layer.right, c.width
    H, d, dv = s.heads, s.dim, s.vdim
    rows = [weights.matrix(p + "q", (H * d, W)), weights.matrix(p + "k", (H * d, W)), weights.matrix(p + "v", (H * dv, W)),
            weights.matrix(p + "g", (H * dv, W))]
    out = weights.matrix(p + "o", (W, H * dv))
    return LightningAttention(proj=_padded(rows, lightning_columns(H, d, dv)[-1]), out=out,
                              norm_weight=weights.vector(p + "norm", (H * dv,)), decay=s.decay, heads=H, dim=d,
                              value_dim=dv, eps=c.eps, act_dtype=act, name=p)


def _gated(weights: WeightSource, p: str, ff: int, W: int, act, limit: float = 0.0, biases: bool = False) -> DenseSwiGLU:
    def bias(name, n):
        return weights.vector(f"{p}{name}.b", (n,), init="normal") if biases else None
    gate, gate_b = weights.matrix(p + "gate", (ff, W)), bias("gate", ff)
    up, up_b = weights.matrix(p + "up", (ff, W)), bias("up", ff)
    down, down_b = weights.matrix(p + "down", (W, ff)), bias("down", W)
    return DenseSwiGLU(gate_up=Linear(_cat([gate, up]), p + "gate|up", bias=_cat([gate_b, up_b]) if biases else None),
                       down=Linear(down, p + "down", bias=down_b), act_dtype=act, limit=limit)


def _feed_forward(c: RadupelConfig, layer: RadupelLayer, p: str, weights: WeightSource, act):
    m, W = layer.mlp, c.width
    if m is None:
        return None
    if m.kind == "dense":
        return _gated(weights, p, m.ff, W, act, biases=True)
    gate_up, down = [], []
    for e in range(m.experts):                 # file order: e0.gate, e0.up, e0.down, e1.gate, ...
        gate_up.append(_cat([weights.matrix(f"{p}e{e}.gate", (m.ff, W)), weights.matrix(f"{p}e{e}.up", (m.ff, W))]))
        down.append(weights.matrix(f"{p}e{e}.down", (W, m.ff)))
    router = weights.vector(p + "router", (m.experts + m.identity, W), init="normal")
    correction = weights.vector(p + "correction", (m.experts + m.identity,), init="normal")
    shared = shared_gate = None
    if m.shared_ff:
        shared = _gated(weights, p + "shared.", m.shared_ff, W, act, limit=m.shared_limit)
        shared_gate = weights.vector(p + "shared.sg", (1, W), init="normal").reshape(W)
    return MoESoftmaxGroups(router=router, correction=correction,
                            experts_gate_up=GroupedLinear(torch.stack(gate_up).contiguous(), p + "experts.gate|up"),
                            experts_down=GroupedLinear(torch.stack(down).contiguous(), p + "experts.down"),
                            top_k=m.top, identity=m.identity, groups=m.groups, keep=m.keep, route_scale=m.scale,
                            limit=m.limit, shared=shared, shared_gate=shared_gate, act_dtype=act)


def build_radupel(config: RadupelConfig, weights: WeightSource) -> DecoderModel:
    c, act, W = config, weights.compute_dtype, config.width
    embedding = weights.matrix("embed", (c.vocab, W))
    blocks = []
    for i, layer in enumerate(c.layers):
        p = f"l{i}."
        norm1 = RMSNorm(weights.vector(p + "norm1", (W,)), c.eps)
        norm2 = None
        if layer.mlp is not None:
            norm2 = RMSNorm(weights.vector(p + "norm2", (W,)), c.eps)
        elif weights.stored(p + "norm2"):        # a folder may keep the norm of a feed-forward that is not there:
            weights.vector(p + "norm2", (W,))    # asked for so that the folder checks clean, and not used
        mixer = ScaledBranches(left=_attention(c, layer, p + "mix.left.", weights, act),
                               right=_linear(c, layer, p + "mix.right.", weights, act),
                               left_scale=layer.left_scale, right_scale=layer.right_scale, act_dtype=act, name=p + "mix.")
        ffn = _feed_forward(c, layer, p + "mlp.", weights, act)
        blocks.append(ParallelPairBlock(mixer_norm=norm1, mixer=mixer, ffn_norm=norm2, ffn=ffn, act_dtype=act))
    final_norm = RMSNorm(weights.vector("final.norm", (W,)), c.eps)
    runs = c.layer_runs()
    stream_ops = [AddInput()] if any(again for _, again in runs) else []
    schedule = [ScheduleEntry(i, before=0 if again else None) for i, again in runs]
    return DecoderModel(embedding=embedding, blocks=blocks, final_norm=final_norm, head=Linear(embedding, "embed"),
                        act_dtype=act, schedule=schedule, config=c, stream_ops=stream_ops, logit_softcap=c.logit_softcap)


register_architecture("Radupel", RadupelConfig, build_radupel)
