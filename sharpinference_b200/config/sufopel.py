"""``SufopelConfig``: the typed configuration of the Sufopel architecture.

A Sufopel ``config.json`` gives

* ``vocab``, ``width``, ``max_positions`` (rows of the learned position table), ``norm.eps``, ``embedding.scale``,
  ``logit_scale``, ``token_side.dim`` (numbers per token and layer);
* ``layers``: a list of ``{"type", "mixer", "mlp"}``.  ``type`` is ``latent_attention`` (``heads``, ``dim``, ``vdim``,
  ``q_rank``, ``kv_rank``, ``scale``, and ``kv_from`` where the layer reads the latents that an earlier one caches) or
  ``channel_delta`` (``heads``, ``kv_heads``, ``dim``, ``vdim``, ``conv`` taps).  ``mlp`` is null, ``{"kind": "dense", "ff"}``
  or ``{"kind": "moe", "expert": {"ff", "limit"}, "router": {"experts", "top", "groups": {"count", "keep"}}}``.

No size stands in code; every layer has sizes of its own.  The inner sizes of the delta layers' two low-rank maps come from
the stored tensors (``a_rank`` and ``g_rank`` in the mixer give them where there is no file; without either the key size is
taken).  Defaults for what a file may leave out: ``kv_heads`` = ``heads``, ``vdim`` = ``dim``, ``scale`` = ``dim^(-1/2)``,
``conv`` = 1 tap, no ``groups`` = one group, ``embedding.scale`` = ``logit_scale`` = 1, no ``token_side`` = none.
"""
from __future__ import annotations

from dataclasses import dataclass
from typing import Optional, Tuple

from .base import ConfigReader
from .notedra import _merge


@dataclass(frozen=True)
class SufopelLatent:
    heads: int
    dim: int
    vdim: int
    q_rank: int
    kv_rank: int
    scale: float
    kv_from: Optional[int] = None

    type = "latent_attention"

    def to_dict(self) -> dict:
        out = {"heads": self.heads, "dim": self.dim, "vdim": self.vdim, "q_rank": self.q_rank, "kv_rank": self.kv_rank,
               "scale": self.scale}
        if self.kv_from is not None:
            out["kv_from"] = self.kv_from
        return out


@dataclass(frozen=True)
class SufopelDelta:
    heads: int
    kv_heads: int
    dim: int
    vdim: int
    conv: int = 1
    a_rank: int = 0              # 0: the stored tensor's
    g_rank: int = 0

    type = "channel_delta"

    def to_dict(self) -> dict:
        out = {"heads": self.heads, "kv_heads": self.kv_heads, "dim": self.dim, "vdim": self.vdim, "conv": self.conv}
        if self.a_rank:
            out["a_rank"] = self.a_rank
        if self.g_rank:
            out["g_rank"] = self.g_rank
        return out


@dataclass(frozen=True)
class SufopelMLP:
    kind: str                    # "dense" | "moe"
    ff: int
    limit: float = 0.0
    experts: int = 0
    top: int = 0
    groups: int = 1
    keep: int = 1

    def to_dict(self) -> dict:
        if self.kind == "dense":
            return {"kind": "dense", "ff": self.ff}
        router = {"experts": self.experts, "top": self.top}
        if self.groups > 1:
            router["groups"] = {"count": self.groups, "keep": self.keep}
        return {"kind": "moe", "expert": {"ff": self.ff, "limit": self.limit}, "router": router}


@dataclass(frozen=True)
class SufopelLayer:
    mixer: object                # SufopelLatent | SufopelDelta
    mlp: Optional[SufopelMLP]

    def to_dict(self) -> dict:
        return {"type": self.mixer.type, "mixer": self.mixer.to_dict(), "mlp": None if self.mlp is None else self.mlp.to_dict()}


@dataclass(frozen=True)
class SufopelConfig:
    vocab: int
    width: int
    max_positions: int
    eps: float
    embedding_scale: float
    logit_scale: float
    side_dim: int                # 0: no side input
    layers: Tuple[SufopelLayer, ...]

    architecture = "Sufopel"

    @classmethod
    def from_dict(cls, obj: dict, where: str = "config.json") -> "SufopelConfig":
        r = ConfigReader(obj, where)
        vocab, width, max_positions = r.int("vocab"), r.int("width"), r.int("max_positions")
        logit_scale = r.float("logit_scale", 1.0)
        eps, embedding_scale, side_dim = None, 1.0, 0
        norm = r.object("norm")
        if norm is not None:
            nr = ConfigReader(norm, f"{where}[norm]")
            eps = nr.float("eps")
            _merge(r, nr)
        emb = r.object("embedding", None)
        if emb is not None:
            er = ConfigReader(emb, f"{where}[embedding]")
            embedding_scale = er.float("scale", 1.0)
            _merge(r, er)
        side = r.object("token_side", None)
        if side is not None:
            sr = ConfigReader(side, f"{where}[token_side]")
            side_dim = sr.int("dim")
            _merge(r, sr)
        raw_layers = obj.get("layers")
        if not isinstance(raw_layers, list) or not raw_layers:
            r.problem("key 'layers': expected a non-empty list of layer descriptions")
            raw_layers = []
        layers = []
        for i, entry in enumerate(raw_layers):
            layer = _read_layer(entry, f"{where}[layers][{i}]", r)
            if layer is not None:
                layers.append(layer)
        if r.ok:
            r.require(vocab > 0 and width > 0, f"vocab ({vocab}) and width ({width}) must be positive")
            r.require(max_positions > 0, f"max_positions ({max_positions}) must be positive")
            r.require(eps >= 0, f"norm.eps must not be negative, found {eps}")
            r.require(side is None or side_dim > 0, f"token_side.dim ({side_dim}) must be positive")
            for i, layer in enumerate(layers):
                j = getattr(layer.mixer, "kv_from", None)
                if j is None:
                    continue
                src = layers[j].mixer if 0 <= j < i else None
                r.require(isinstance(src, SufopelLatent) and src.kv_from is None and src.kv_rank == layer.mixer.kv_rank,
                          f"layers[{i}].mixer.kv_from ({j}) must name an earlier latent_attention layer with a latent of its "
                          f"own and the same kv_rank")
        r.finish()
        return cls(vocab=vocab, width=width, max_positions=max_positions, eps=eps, embedding_scale=embedding_scale,
                   logit_scale=logit_scale, side_dim=side_dim, layers=tuple(layers))

    def to_dict(self) -> dict:
        out = {"architecture": self.architecture, "vocab": self.vocab, "width": self.width, "max_positions": self.max_positions,
               "norm": {"eps": self.eps}, "embedding": {"scale": self.embedding_scale}, "logit_scale": self.logit_scale,
               "layers": [layer.to_dict() for layer in self.layers]}
        if self.side_dim:
            out["token_side"] = {"dim": self.side_dim}
        return out


def _read_layer(entry, where: str, top: ConfigReader) -> Optional[SufopelLayer]:
    if not isinstance(entry, dict):
        top.problem(f"{where}: expected an object, found {type(entry).__name__}")
        return None
    r = ConfigReader(entry, where)
    kind, mixer = r.str("type"), r.object("mixer")
    mlp = _read_mlp(entry.get("mlp"), f"{where}[mlp]", r)
    m = None
    if kind is not None and mixer is not None:
        if kind == "latent_attention":
            m = _read_latent(mixer, f"{where}[mixer]", r)
        elif kind == "channel_delta":
            m = _read_delta(mixer, f"{where}[mixer]", r)
        else:
            r.problem(f"key 'type': expected 'latent_attention' or 'channel_delta', found {kind!r}")
    _merge(top, r)
    return SufopelLayer(m, mlp) if r.ok and m is not None else None


def _read_latent(obj: dict, where: str, top: ConfigReader) -> Optional[SufopelLatent]:
    m = ConfigReader(obj, where)
    heads, dim, q_rank, kv_rank = m.int("heads"), m.int("dim"), m.int("q_rank"), m.int("kv_rank")
    vdim, scale, kv_from = m.int("vdim", dim), m.float("scale", None), m.int("kv_from", None)
    out = None
    if m.ok:
        m.require(min(heads, dim, vdim, q_rank, kv_rank) > 0,
                  f"heads ({heads}), dim ({dim}), vdim ({vdim}), q_rank ({q_rank}) and kv_rank ({kv_rank}) must be positive")
        if m.ok:
            out = SufopelLatent(heads, dim, vdim, q_rank, kv_rank, float(dim) ** -0.5 if scale is None else scale, kv_from)
    _merge(top, m)
    return out


def _read_delta(obj: dict, where: str, top: ConfigReader) -> Optional[SufopelDelta]:
    m = ConfigReader(obj, where)
    heads, dim = m.int("heads"), m.int("dim")
    kv_heads, vdim, conv = m.int("kv_heads", heads), m.int("vdim", dim), m.int("conv", 1)
    a_rank, g_rank = m.int("a_rank", 0), m.int("g_rank", 0)
    out = None
    if m.ok:
        m.require(min(heads, dim, vdim) > 0, f"heads ({heads}), dim ({dim}) and vdim ({vdim}) must be positive")
        m.require(kv_heads > 0 and heads % max(kv_heads, 1) == 0, f"heads ({heads}) must be a multiple of kv_heads ({kv_heads})")
        m.require(conv >= 1, f"conv ({conv}) must be at least one tap")
        m.require(min(a_rank, g_rank) >= 0, f"a_rank ({a_rank}) and g_rank ({g_rank}) must not be negative")
        if m.ok:
            out = SufopelDelta(heads, kv_heads, dim, vdim, conv, a_rank, g_rank)
    _merge(top, m)
    return out


def _read_mlp(entry, where: str, top: ConfigReader) -> Optional[SufopelMLP]:
    if entry is None:
        return None
    if not isinstance(entry, dict):
        top.problem(f"{where}: expected an object or null, found {type(entry).__name__}")
        return None
    r = ConfigReader(entry, where)
    kind = r.str("kind")
    mlp = None
    if kind == "dense":
        ff = r.int("ff")
        if r.ok:
            r.require(ff > 0, f"ff must be positive, found {ff}")
            mlp = SufopelMLP("dense", ff)
    elif kind == "moe":
        expert, router = r.object("expert"), r.object("router")
        if expert is not None and router is not None:
            er, rr = ConfigReader(expert, f"{where}[expert]"), ConfigReader(router, f"{where}[router]")
            ff, limit, experts, top_k = er.int("ff"), er.float("limit"), rr.int("experts"), rr.int("top")
            groups = rr.object("groups", None)
            count = keep = 1
            if groups is not None:
                gr = ConfigReader(groups, f"{where}[router][groups]")
                count, keep = gr.int("count"), gr.int("keep")
                _merge(rr, gr)
            if er.ok and rr.ok:
                er.require(ff > 0 and limit > 0, f"ff ({ff}) and limit ({limit}) must be positive")
                rr.require(experts > 0 and count >= 1 and experts % max(count, 1) == 0 and 1 <= keep <= count,
                           f"groups.count ({count}) must divide experts ({experts}) and groups.keep ({keep}) be 1 .. count")
                if rr.ok:
                    rr.require(1 <= top_k <= keep * (experts // count),
                               f"top ({top_k}) must be 1 .. the experts of the kept groups ({keep * (experts // count)})")
            _merge(r, er)
            _merge(r, rr)
            if r.ok:
                mlp = SufopelMLP("moe", ff, limit, experts, top_k, count, keep)
    elif kind is not None:
        r.problem(f"key 'kind': expected 'dense' or 'moe', found {kind!r}")
    _merge(top, r)
    return mlp if r.ok else None
