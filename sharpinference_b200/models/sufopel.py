"""The Sufopel architecture, put together from parts, and its tensor names.

A decoder with a norm before and behind every sublayer and a factor per element on what a sublayer adds
(:class:`SandwichBlock`), an embedding that is scaled and gets a learned vector per position
(:class:`TableWithPositions`), and behind every layer a slice of a per-token table through a gate that reads the stream
(:class:`TokenSide`).  Layers (``config.layers[i]``, every layer with sizes of its own) have one of two mixers:

* ``latent_attention``: :class:`LatentAttention` with a query latent, without a rotated part, with a gate per element; with
  ``kv_from`` the layer has no latent of its own and reads the ones an earlier layer cached (a schedule entry with
  ``cache_from``);
* ``channel_delta``: :class:`ChannelDelta`, the gated delta rule with a decay per key channel behind short convolutions.

The feed-forward is absent, a dense gated network (:class:`DenseSwiGLU`) or a mixture routed by sigmoid scores in groups
with clamped gates (:class:`MoESigmoidGroups`).  The logits are ``head x * logit_scale``.

Tensor names (linear weights ``[out, in]``): ``embed``, ``pos``, ``side.embed [vocab, layers * dim]``, ``final.norm``, ``head``;
per layer ``l<i>.norm{1,1b,2,2b}``, ``l<i>.ls{1,2}``, ``l<i>.side.{gate,proj,norm}``; for latent attention
``l<i>.mix.{dq,dq.norm,uq,uk,uv,g,o}`` and, unless the layer borrows, ``l<i>.mix.{dkv,dkv.norm}``; for the delta rule
``l<i>.mix.{q,k,v}`` with ``.conv [channels, taps]`` each and ``l<i>.mix.{b,A_log,norm,a1,a2,dt_bias,g1,g2,o}``;
``l<i>.mlp.{gate,up,down}``, or ``l<i>.mlp.e<j>.{gate,up,down}`` and ``l<i>.mlp.{router,correction}``.
"""
from __future__ import annotations

from typing import Optional

import torch

from ..config.sufopel import SufopelConfig, SufopelDelta, SufopelLatent, SufopelLayer
from ..parts import (ChannelDelta, DenseSwiGLU, GroupedLinear, LatentAttention, Linear, MoESigmoidGroups, RMSNorm, SandwichBlock,
                     TableWithPositions, TokenSide, delta_columns)
from ..registry import register_architecture
from ..weights.source import WeightSource
from .model import DecoderModel, ScheduleEntry
from .notedra import _cat
from .radupel import _padded


def _up8(n: int) -> int:
    return (n + 7) // 8 * 8


def _placed(pieces, rows: int, cols: int) -> torch.Tensor:
    """A matrix of zeros that holds ``(piece, first row, first column)``."""
    like = pieces[0][0]
    out = torch.zeros((rows, cols), dtype=like.dtype, device=like.device)
    if like.device.type != "meta":
        for piece, r, c in pieces:
            out[r: r + piece.shape[0], c: c + piece.shape[1]] = piece
    return out


def _latent(c: SufopelConfig, m: SufopelLatent, p: str, weights: WeightSource, act) -> LatentAttention:
    W, H, d, dv, r = c.width, m.heads, m.dim, m.vdim, m.kv_rank
    borrows = m.kv_from is not None
    rows = [weights.matrix(p + "dq", (m.q_rank, W))]
    q_norm, c_norm = weights.vector(p + "dq.norm", (m.q_rank,)), None
    up_q = weights.matrix(p + "uq", (H * d, m.q_rank))
    if not borrows:
        rows.append(weights.matrix(p + "dkv", (r, W)))
        c_norm = weights.vector(p + "dkv.norm", (r,))
    uk, uv = weights.matrix(p + "uk", (H * d, r)), weights.matrix(p + "uv", (H * dv, r))
    rows.append(weights.matrix(p + "g", (H * dv, W)))                # the gate rides in the fused projection
    out = weights.matrix(p + "o", (W, H * dv))
    return LatentAttention(down=Linear(_cat(rows), p + ("dq|g" if borrows else "dq|dkv|g")), q_norm_weight=q_norm,
                           c_norm_weight=c_norm, up_q=Linear(up_q, p + "uq"),
                           up_k=GroupedLinear(uk.reshape(H, d, r).transpose(1, 2).contiguous(), p + "uk"),
                           up_v=GroupedLinear(uv.reshape(H, dv, r).contiguous(), p + "uv"), out=Linear(out, p + "o"),
                           num_heads=H, dim=d, rot_dim=0, value_dim=dv, q_rank=m.q_rank, kv_rank=r, eps=c.eps,
                           softmax_scale=m.scale, act_dtype=act, element_gate=True, borrows=borrows)


def _rank(weights: WeightSource, name: str, given: int, otherwise: int) -> int:
    return (weights.shape_of(name) or (given or otherwise,))[0]


def _delta(c: SufopelConfig, m: SufopelDelta, p: str, weights: WeightSource, act) -> ChannelDelta:
    W, H, G, d, dv = c.width, m.heads, m.kv_heads, m.dim, m.vdim
    rows, taps = [], []
    for s, n in (("q", G * d), ("k", G * d), ("v", H * dv)):         # file order: every projection with its convolution
        rows.append(weights.matrix(p + s, (n, W)))
        if m.conv > 1 or weights.stored(f"{p}{s}.conv") is not False:
            taps.append(weights.vector(f"{p}{s}.conv", (n, m.conv), init="normal"))
        else:                                                        # one tap and none stored: the projection as it is
            taps.append(torch.ones((n, 1), dtype=torch.float32, device=weights.device))
    ra, rg = _rank(weights, p + "a1", m.a_rank, d), _rank(weights, p + "g1", m.g_rank, d)
    low = _up8(ra + rg)
    beta = weights.matrix(p + "b", (H, W))
    a_log = weights.vector(p + "A_log", (H,), init="normal")
    norm = weights.vector(p + "norm", (dv,))
    a1, a2 = weights.matrix(p + "a1", (ra, W)), weights.matrix(p + "a2", (H * d, ra))
    dt_bias = weights.vector(p + "dt_bias", (H * d,), init="normal")
    g1, g2 = weights.matrix(p + "g1", (rg, W)), weights.matrix(p + "g2", (H * dv, rg))
    out = weights.matrix(p + "o", (W, H * dv))
    rows += [_padded([a1, g1], low), beta]
    up = _placed([(a2, 0, 0), (g2, H * d, ra)], H * (d + dv), low)
    return ChannelDelta(proj=Linear(_padded(rows, delta_columns(G, H, d, dv, low)[-1]), p + "q|k|v|a1|g1|b"),
                        up=Linear(up, p + "a2|g2"), out=Linear(out, p + "o"), conv_weight=torch.cat(taps, dim=0).t().contiguous(),
                        dt_bias=dt_bias, a_log=a_log, norm_weight=norm, heads=H, kv_heads=G, dim=d, value_dim=dv, low=low,
                        eps=c.eps, act_dtype=act)


def _feed_forward(c: SufopelConfig, layer: SufopelLayer, p: str, weights: WeightSource, act):
    m, W = layer.mlp, c.width
    if m is None:
        return None
    if m.kind == "dense":
        gate_up = _cat([weights.matrix(p + "gate", (m.ff, W)), weights.matrix(p + "up", (m.ff, W))])
        return DenseSwiGLU(gate_up=Linear(gate_up, p + "gate|up"), down=Linear(weights.matrix(p + "down", (W, m.ff)), p + "down"),
                           act_dtype=act)
    gate_up, down = [], []
    for e in range(m.experts):                 # file order: e0.gate, e0.up, e0.down, e1.gate, ...
        gate_up.append(_cat([weights.matrix(f"{p}e{e}.gate", (m.ff, W)), weights.matrix(f"{p}e{e}.up", (m.ff, W))]))
        down.append(weights.matrix(f"{p}e{e}.down", (W, m.ff)))
    router = weights.vector(p + "router", (m.experts, W), init="normal")
    correction = weights.vector(p + "correction", (m.experts,), init="normal")
    return MoESigmoidGroups(router=router, correction=correction,
                            experts_gate_up=GroupedLinear(torch.stack(gate_up).contiguous(), p + "experts.gate|up"),
                            experts_down=GroupedLinear(torch.stack(down).contiguous(), p + "experts.down"),
                            top_k=m.top, groups=m.groups, keep=m.keep, limit=m.limit, act_dtype=act)


def _side(c: SufopelConfig, i: int, table: Optional[torch.Tensor], p: str, weights: WeightSource, act) -> Optional[TokenSide]:
    if table is None:
        return None
    W, dim, padded = c.width, c.side_dim, _up8(c.side_dim)
    gate, proj = weights.matrix(p + "gate", (dim, W)), weights.matrix(p + "proj", (W, dim))
    return TokenSide(table=table, column=i * dim, dim=dim, gate=Linear(_placed([(gate, 0, 0)], padded, W), p + "gate"),
                     proj=Linear(_placed([(proj, 0, 0)], W, padded), p + "proj"),
                     norm_weight=weights.vector(p + "norm", (W,)), eps=c.eps, act_dtype=act)


def build_sufopel(config: SufopelConfig, weights: WeightSource) -> DecoderModel:
    c, act, W = config, weights.compute_dtype, config.width
    embedding = weights.matrix("embed", (c.vocab, W))
    pos = weights.matrix("pos", (c.max_positions, W))
    side = weights.matrix("side.embed", (c.vocab, len(c.layers) * c.side_dim)) if c.side_dim else None
    blocks, schedule = [], []
    for i, layer in enumerate(c.layers):
        p = f"l{i}."
        norm1, norm1b = RMSNorm(weights.vector(p + "norm1", (W,)), c.eps), RMSNorm(weights.vector(p + "norm1b", (W,)), c.eps)
        ls1 = weights.vector(p + "ls1", (W,))
        norm2 = norm2b = ls2 = None
        if layer.mlp is not None:
            norm2, norm2b = RMSNorm(weights.vector(p + "norm2", (W,)), c.eps), RMSNorm(weights.vector(p + "norm2b", (W,)), c.eps)
            ls2 = weights.vector(p + "ls2", (W,))
        else:                                   # a folder may keep the vectors of a feed-forward that is not there:
            for name in ("norm2", "norm2b", "ls2"):     # asked for so that the folder checks clean, and not used
                if weights.stored(p + name):
                    weights.vector(p + name, (W,))
        make = _latent if isinstance(layer.mixer, SufopelLatent) else _delta
        blocks.append(SandwichBlock(mixer_norm=norm1, mixer=make(c, layer.mixer, p + "mix.", weights, act), mixer_post=norm1b,
                                    mixer_scale=ls1, ffn_norm=norm2, ffn=_feed_forward(c, layer, p + "mlp.", weights, act),
                                    ffn_post=norm2b, ffn_scale=ls2, side=_side(c, i, side, p + "side.", weights, act),
                                    act_dtype=act))
        schedule.append(ScheduleEntry(i, cache_from=getattr(layer.mixer, "kv_from", None)))     # layers run once, in order
    final_norm = RMSNorm(weights.vector("final.norm", (W,)), c.eps)
    head = Linear(weights.matrix("head", (c.vocab, W)), "head")
    return DecoderModel(embedding=embedding, blocks=blocks, final_norm=final_norm, head=head, act_dtype=act, config=c,
                        schedule=schedule, embedder=TableWithPositions(embed=embedding, pos=pos, scale=c.embedding_scale),
                        logit_scale=c.logit_scale)


register_architecture("Sufopel", SufopelConfig, build_sufopel)
