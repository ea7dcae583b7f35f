"""``RadupelConfig``: the typed configuration of the Radupel architecture.

A Radupel ``config.json`` gives

* ``vocab``, ``width``, ``norm.eps``, ``logit_softcap`` (0 or absent: logits as they are);
* ``loop`` (optional): layers ``start`` .. ``stop - 1`` run ``times`` times in a row;
* ``layers``: a list of ``{"type": "parallel", "mixer", "mlp"}``.  ``mixer.left`` is attention over convolved projections:
  ``heads``, ``kv_heads``, ``dim``, ``vdim``, ``scale``, ``conv`` (taps), ``rot.dims`` / ``rot.base``; ``mixer.right`` is
  linear attention with a constant decay: ``heads``, ``dim``, ``vdim``, ``decay`` (one number a head);
  ``mixer.left_scale`` and ``mixer.right_scale`` weight the two outputs.  ``mlp`` is null, ``{"kind": "dense", "ff"}`` or
  ``{"kind": "moe", "expert": {"ff", "limit"}, "router": {"experts", "top", "scale", "identity", "groups": {"count",
  "keep"}}, "shared": {"ff", "limit"} or null}``.

No size stands in code; every layer has sizes of its own.  Defaults for what a file may leave out: ``kv_heads`` =
``heads``, ``vdim`` = ``dim``, ``scale`` = ``dim^(-1/2)``, ``conv`` = 1 tap, no ``rot`` = no rotation, ``rot.base`` =
10000, scales of 1, no ``groups`` = one group, ``identity`` = 0.
"""
from __future__ import annotations

from dataclasses import dataclass
from typing import Optional, Tuple

from .base import ConfigReader
from .notedra import _merge


@dataclass(frozen=True)
class RadupelAttention:
    heads: int
    kv_heads: int
    dim: int
    vdim: int
    scale: float
    conv: int = 1
    rot_dims: int = 0
    rot_base: float = 10000.0

    def to_dict(self) -> dict:
        out = {"heads": self.heads, "kv_heads": self.kv_heads, "dim": self.dim, "vdim": self.vdim, "scale": self.scale,
               "conv": self.conv}
        if self.rot_dims:
            out["rot"] = {"dims": self.rot_dims, "base": self.rot_base}
        return out


@dataclass(frozen=True)
class RadupelLinear:
    heads: int
    dim: int
    vdim: int
    decay: Tuple[float, ...]

    def to_dict(self) -> dict:
        return {"heads": self.heads, "dim": self.dim, "vdim": self.vdim, "decay": list(self.decay)}


@dataclass(frozen=True)
class RadupelMLP:
    kind: str                    # "dense" | "moe"
    ff: int
    limit: float = 0.0
    experts: int = 0
    top: int = 0
    identity: int = 0
    groups: int = 1
    keep: int = 1
    scale: float = 1.0
    shared_ff: int = 0           # 0: no shared expert
    shared_limit: float = 0.0

    def to_dict(self) -> dict:
        if self.kind == "dense":
            return {"kind": "dense", "ff": self.ff}
        router = {"experts": self.experts, "top": self.top, "scale": self.scale, "identity": self.identity}
        if self.groups > 1:
            router["groups"] = {"count": self.groups, "keep": self.keep}
        return {"kind": "moe", "expert": {"ff": self.ff, "limit": self.limit}, "router": router,
                "shared": {"ff": self.shared_ff, "limit": self.shared_limit} if self.shared_ff else None}


@dataclass(frozen=True)
class RadupelLayer:
    left: RadupelAttention
    right: RadupelLinear
    left_scale: float
    right_scale: float
    mlp: Optional[RadupelMLP]

    def to_dict(self) -> dict:
        return {"type": "parallel",
                "mixer": {"left": self.left.to_dict(), "right": self.right.to_dict(), "left_scale": self.left_scale,
                          "right_scale": self.right_scale},
                "mlp": None if self.mlp is None else self.mlp.to_dict()}


@dataclass(frozen=True)
class RadupelConfig:
    vocab: int
    width: int
    eps: float
    logit_softcap: float
    layers: Tuple[RadupelLayer, ...]
    loop_start: int = 0
    loop_stop: int = 0
    loop_times: int = 0          # 0: no loop

    architecture = "Radupel"

    def layer_runs(self):
        """The order in which layers run: ``(layer, whether the embedding output is added right before it)``."""
        runs = []
        for i in range(len(self.layers)):
            if not self.loop_times or not self.loop_start <= i < self.loop_stop:
                runs.append((i, False))
            elif i == self.loop_start:
                for t in range(self.loop_times):
                    runs += [(j, t > 0 and j == i) for j in range(self.loop_start, self.loop_stop)]
        return runs

    @classmethod
    def from_dict(cls, obj: dict, where: str = "config.json") -> "RadupelConfig":
        r = ConfigReader(obj, where)
        vocab, width, softcap = r.int("vocab"), r.int("width"), r.float("logit_softcap", 0.0)
        eps = None
        norm = r.object("norm")
        if norm is not None:
            nr = ConfigReader(norm, f"{where}[norm]")
            eps = nr.float("eps")
            _merge(r, nr)
        raw_layers = obj.get("layers")
        if not isinstance(raw_layers, list) or not raw_layers:
            r.problem("key 'layers': expected a non-empty list of layer descriptions")
            raw_layers = []
        layers = []
        for i, entry in enumerate(raw_layers):
            layer = _read_layer(entry, f"{where}[layers][{i}]", r)
            if layer is not None:
                layers.append(layer)
        start = stop = times = 0
        loop = r.object("loop", None)
        if loop is not None:
            lr = ConfigReader(loop, f"{where}[loop]")
            start, stop, times = lr.int("start"), lr.int("stop"), lr.int("times")
            if lr.ok:
                lr.require(0 <= start < stop <= len(raw_layers),
                           f"start ({start}) and stop ({stop}) must satisfy 0 <= start < stop <= layers ({len(raw_layers)})")
                lr.require(times >= 1, f"times must be at least 1, found {times}")
            _merge(r, lr)
        if r.ok:
            r.require(vocab > 0 and width > 0, f"vocab ({vocab}) and width ({width}) must be positive")
            r.require(eps >= 0, f"norm.eps must not be negative, found {eps}")
            r.require(softcap >= 0, f"logit_softcap must not be negative, found {softcap}")
        r.finish()
        return cls(vocab=vocab, width=width, eps=eps, logit_softcap=softcap, layers=tuple(layers), loop_start=start,
                   loop_stop=stop, loop_times=times)

    def to_dict(self) -> dict:
        out = {"architecture": self.architecture, "vocab": self.vocab, "width": self.width, "norm": {"eps": self.eps},
               "logit_softcap": self.logit_softcap, "layers": [layer.to_dict() for layer in self.layers]}
        if self.loop_times:
            out["loop"] = {"start": self.loop_start, "stop": self.loop_stop, "times": self.loop_times}
        return out


def _read_layer(entry, where: str, top: ConfigReader) -> Optional[RadupelLayer]:
    if not isinstance(entry, dict):
        top.problem(f"{where}: expected an object, found {type(entry).__name__}")
        return None
    r = ConfigReader(entry, where)
    kind, mixer = r.str("type"), r.object("mixer")
    mlp = _read_mlp(entry.get("mlp"), f"{where}[mlp]", r)
    layer = None
    if kind is not None and kind != "parallel":
        r.problem(f"key 'type': expected 'parallel', found {kind!r}")
    elif mixer is not None:
        m = ConfigReader(mixer, f"{where}[mixer]")
        left, right = m.object("left"), m.object("right")
        left_scale, right_scale = m.float("left_scale", 1.0), m.float("right_scale", 1.0)
        att = None if left is None else _read_attention(left, f"{where}[mixer][left]", m)
        lin = None if right is None else _read_linear(right, f"{where}[mixer][right]", m)
        _merge(r, m)
        if r.ok and att is not None and lin is not None:
            layer = RadupelLayer(att, lin, left_scale, right_scale, mlp)
    _merge(top, r)
    return layer if r.ok else None


def _read_attention(obj: dict, where: str, top: ConfigReader) -> Optional[RadupelAttention]:
    m = ConfigReader(obj, where)
    heads, dim = m.int("heads"), m.int("dim")
    kv_heads, vdim, scale, conv = m.int("kv_heads", heads), m.int("vdim", dim), m.float("scale", None), m.int("conv", 1)
    rot = m.object("rot", None)
    rot_dims, rot_base = 0, 10000.0
    if rot is not None:
        rr = ConfigReader(rot, f"{where}[rot]")
        rot_dims, rot_base = rr.int("dims"), rr.float("base", 10000.0)
        _merge(m, rr)
    out = None
    if m.ok:
        m.require(heads > 0 and dim > 0 and vdim > 0, f"heads ({heads}), dim ({dim}) and vdim ({vdim}) must be positive")
        m.require(kv_heads > 0 and heads % max(kv_heads, 1) == 0, f"heads ({heads}) must be a multiple of kv_heads ({kv_heads})")
        m.require(conv >= 1, f"conv ({conv}) must be at least one tap")
        m.require(rot_dims % 2 == 0 and 0 <= rot_dims <= dim, f"rot.dims ({rot_dims}) must be even and at most dim ({dim})")
        m.require(rot_base > 0, f"rot.base ({rot_base}) must be positive")
        if m.ok:
            out = RadupelAttention(heads, kv_heads, dim, vdim, float(dim) ** -0.5 if scale is None else scale, conv,
                                   rot_dims, rot_base)
    _merge(top, m)
    return out


def _read_linear(obj: dict, where: str, top: ConfigReader) -> Optional[RadupelLinear]:
    m = ConfigReader(obj, where)
    heads, dim = m.int("heads"), m.int("dim")
    vdim, decay = m.int("vdim", dim), obj.get("decay")
    numbers = isinstance(decay, list) and all(isinstance(a, (int, float)) and not isinstance(a, bool) for a in decay)
    if not numbers:
        m.problem(f"key 'decay': expected a list of numbers, found {decay!r}")
    out = None
    if m.ok:
        m.require(heads > 0 and dim > 0 and vdim > 0, f"heads ({heads}), dim ({dim}) and vdim ({vdim}) must be positive")
        m.require(len(decay) == heads, f"decay has {len(decay)} numbers for {heads} heads")
        if m.ok:
            out = RadupelLinear(heads, dim, vdim, tuple(float(a) for a in decay))
    _merge(top, m)
    return out


def _read_mlp(entry, where: str, top: ConfigReader) -> Optional[RadupelMLP]:
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
            mlp = RadupelMLP("dense", ff)
    elif kind == "moe":
        expert, router, shared = r.object("expert"), r.object("router"), r.object("shared", None)
        if expert is not None and router is not None:
            er, rr = ConfigReader(expert, f"{where}[expert]"), ConfigReader(router, f"{where}[router]")
            ff, limit = er.int("ff"), er.float("limit")
            experts, top_k = rr.int("experts"), rr.int("top")
            scale, identity, groups = rr.float("scale", 1.0), rr.int("identity", 0), rr.object("groups", None)
            count = keep = 1
            if groups is not None:
                gr = ConfigReader(groups, f"{where}[router][groups]")
                count, keep = gr.int("count"), gr.int("keep")
                _merge(rr, gr)
            shared_ff, shared_limit = 0, 0.0
            if shared is not None:
                sr = ConfigReader(shared, f"{where}[shared]")
                shared_ff, shared_limit = sr.int("ff"), sr.float("limit", limit)
                if sr.ok:
                    sr.require(shared_ff > 0 and shared_limit > 0, f"ff ({shared_ff}) and limit ({shared_limit}) must be positive")
                _merge(er, sr)
            if er.ok and rr.ok:
                er.require(ff > 0 and limit > 0, f"ff ({ff}) and limit ({limit}) must be positive")
                rr.require(experts > 0 and identity >= 0, f"experts ({experts}) must be positive, identity ({identity}) not negative")
                n = experts + identity
                rr.require(count >= 1 and n % max(count, 1) == 0 and 1 <= keep <= count,
                           f"groups.count ({count}) must divide experts + identity ({n}) and groups.keep ({keep}) be 1 .. count")
                if rr.ok:
                    rr.require(1 <= top_k <= keep * (n // count),
                               f"top ({top_k}) must be 1 .. the experts of the kept groups ({keep * (n // count)})")
            _merge(r, er)
            _merge(r, rr)
            if r.ok:
                mlp = RadupelMLP("moe", ff, limit, experts, top_k, identity, count, keep, scale, shared_ff, shared_limit)
    elif kind is not None:
        r.problem(f"key 'kind': expected 'dense' or 'moe', found {kind!r}")
    _merge(top, r)
    return mlp if r.ok else None
