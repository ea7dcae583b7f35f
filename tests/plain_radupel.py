"""A plain, slow statement of the Radupel design in float64, one function per mechanism.

Nothing here is shared with the engine: the tests compare the engine's logits with these functions on small random
models.  A model is a configuration dictionary (the keys of ``config.json``) and a dictionary of tensors by file name.

Notation: ``x`` is the residual stream ``[n, W]`` of one sequence whose first row is position 0; matrices are stored
``[out, in]`` and applied as ``x @ W.T``.  A layer is ``x += mixer(rms(x) w1) + ff(rms(x) w2)``, both norms of the same
``x``.  ``round_to`` (a torch dtype or None) rounds the operands of matrix products, so that what rounding alone does
can be measured; None keeps everything in float64.
"""
from __future__ import annotations

import math
from typing import Dict, List, Optional

import torch

F64 = torch.float64


def _r(t: torch.Tensor, round_to) -> torch.Tensor:
    return t if round_to is None else t.to(round_to).to(F64)


def rms(x, w, eps):
    return x / torch.sqrt((x * x).mean(dim=-1, keepdim=True) + eps) * w


def silu(z):
    return z * torch.sigmoid(z)


# ---------------------------------------------------------------------------------------------------------------
# the left branch: attention over convolved projections
# ---------------------------------------------------------------------------------------------------------------
def causal_conv(u, w):
    """``y_t = sum_j w[:, j] u_(t - taps + 1 + j)``, zeros before the start; u [n, C], w [C, taps]."""
    n, C = u.shape
    taps = w.shape[1]
    padded = torch.cat([torch.zeros(taps - 1, C, dtype=u.dtype), u], dim=0)
    y = torch.zeros_like(u)
    for j in range(taps):
        y = y + w[:, j] * padded[j: j + n]
    return y


def rotate_halves(v, dims, base):
    """v [n, heads, d]: row p is position p; elements i and i + dims/2 turn by p * base^(-2i/dims)."""
    n, half = v.shape[0], dims // 2
    out = v.clone()
    for i in range(half):
        a = torch.arange(n, dtype=F64) * base ** (-2.0 * i / dims)
        c, s = torch.cos(a).view(n, 1), torch.sin(a).view(n, 1)
        u, w = v[:, :, i], v[:, :, i + half]
        out[:, :, i] = u * c - w * s
        out[:, :, i + half] = w * c + u * s
    return out


def causal_softmax(scores):
    """scores [heads, n, n]: softmax of every row over the columns up to its own."""
    n = scores.shape[-1]
    visible = torch.arange(n).view(1, n) <= torch.arange(n).view(n, 1)
    s = scores.masked_fill(~visible, -math.inf)
    e = torch.exp(s - s.max(dim=-1, keepdim=True).values)
    return e / e.sum(dim=-1, keepdim=True)


def attention(h, m, t, p, round_to=None):
    """Causal grouped-query attention with a short convolution on every channel of q, k and v, a rotation of the heads'
    leading elements and a sigmoid gate per head; h [n, W] -> [n, W]."""
    n = h.shape[0]
    H, G, d, dv = m["heads"], m.get("kv_heads", m["heads"]), m["dim"], m.get("vdim", m["dim"])
    h = _r(h, round_to)
    proj = {}
    for s in "qkv":
        proj[s] = h @ t[p + s].T
        if (p + s + ".conv") in t:
            proj[s] = causal_conv(proj[s], t[p + s + ".conv"])
    q, k, v = proj["q"].view(n, H, d), proj["k"].view(n, G, d), proj["v"].view(n, G, dv)
    rot = m.get("rot")
    if rot and rot["dims"]:
        q, k = rotate_halves(q, rot["dims"], rot["base"]), rotate_halves(k, rot["dims"], rot["base"])
    q, k, v = _r(q, round_to), _r(k, round_to), _r(v, round_to)
    rep = H // G
    s = torch.einsum("ihd,jhd->hij", q, k.repeat_interleave(rep, dim=1)) * m.get("scale", d ** -0.5)
    o = torch.einsum("hij,jhd->ihd", causal_softmax(s), v.repeat_interleave(rep, dim=1))
    o = o * torch.sigmoid(h @ t[p + "g"].T).view(n, H, 1)
    return _r(o.reshape(n, H * dv), round_to) @ t[p + "o"].T


# ---------------------------------------------------------------------------------------------------------------
# the right branch: linear attention with a constant decay per head
# ---------------------------------------------------------------------------------------------------------------
def decayed_sums(q, k, v, decay, state=None):
    """Per head ``S <- decay S + k v^T``, ``o = S^T q``, row by row; q, k [n, H, d], v [n, H, dv] -> [n, H, dv] and S."""
    n, H, d = q.shape
    S = torch.zeros(H, d, v.shape[-1], dtype=q.dtype) if state is None else state.clone()
    a = torch.as_tensor(decay, dtype=q.dtype).view(H, 1, 1)
    out = []
    for i in range(n):
        S = a * S + k[i].unsqueeze(-1) * v[i].unsqueeze(-2)
        out.append(torch.einsum("hdv,hd->hv", S, q[i]))
    return torch.stack(out), S


def lightning(h, m, t, p, eps, round_to=None):
    n = h.shape[0]
    H, d, dv = m["heads"], m["dim"], m.get("vdim", m["dim"])
    h = _r(h, round_to)
    q, k, v = (silu(h @ t[p + s].T).view(n, H, -1) for s in "qkv")
    assert q.shape[-1] == d and k.shape[-1] == d and v.shape[-1] == dv
    o, _ = decayed_sums(q, k, v, m["decay"])
    o = rms(o.reshape(n, H * dv), t[p + "norm"], eps) * torch.sigmoid(h @ t[p + "g"].T)
    return _r(o, round_to) @ t[p + "o"].T


def side_by_side(h, m, t, p, eps, round_to=None):
    left = attention(h, m["left"], t, p + "left.", round_to)
    right = lightning(h, m["right"], t, p + "right.", eps, round_to)
    return m.get("left_scale", 1.0) * left + m.get("right_scale", 1.0) * right


# ---------------------------------------------------------------------------------------------------------------
# feed-forwards
# ---------------------------------------------------------------------------------------------------------------
def dense(h, t, p, round_to=None):
    h = _r(h, round_to)
    g, u = h @ t[p + "gate"].T + t[p + "gate.b"], h @ t[p + "up"].T + t[p + "up.b"]
    return _r(silu(g) * u, round_to) @ t[p + "down"].T + t[p + "down.b"]


def expert(h, t, p, limit, round_to=None):
    """``g = min(Wg h, limit)``, ``u = clamp(Wu h, -limit, limit)``, ``Wd (g sigmoid(1.702 g) (u + 1))``."""
    g = torch.clamp(h @ t[p + "gate"].T, max=limit)
    u = torch.clamp(h @ t[p + "up"].T, min=-limit, max=limit)
    return _r(g * torch.sigmoid(1.702 * g) * (u + 1.0), round_to) @ t[p + "down"].T


def allowed_experts(choice, count, keep):
    """Which experts may be chosen: those of the ``keep`` groups whose largest choice score is largest.
    choice [n, N] -> bool [n, N]."""
    n, N = choice.shape
    best = choice.view(n, count, N // count).max(dim=-1).values
    kept = torch.topk(best, keep, dim=-1).indices
    ok = torch.zeros(n, count, dtype=torch.bool)
    ok[torch.arange(n).view(n, 1), kept] = True
    return ok.repeat_interleave(N // count, dim=1)


def router_scores(h, t, p):
    """(softmax scores [n, N], choice scores [n, N])."""
    s = torch.softmax(h @ t[p + "router"].T, dim=-1)
    return s, s + t[p + "correction"]


def choose(choice, router):
    """The ``top`` experts with the largest choice scores among those of the kept groups: [n, top]."""
    groups = router.get("groups")
    if groups:
        choice = choice.masked_fill(~allowed_experts(choice, groups["count"], groups["keep"]), -math.inf)
    return torch.topk(choice, router["top"], dim=-1).indices


def mixture(h, mlp, t, p, round_to=None, choices=None):
    """``choices`` [n, top]: experts to use instead of the router's own (their weights still come from the scores).
    Returns (output, chosen [n, top], choice scores [n, N])."""
    router = mlp["router"]
    E, ident, limit = router["experts"], router.get("identity", 0), mlp["expert"]["limit"]
    s, choice = router_scores(h, t, p)
    assert s.shape[1] == E + ident
    idx = choose(choice, router) if choices is None else choices.to(torch.long)
    w = torch.gather(s, 1, idx)
    w = w / (w.sum(dim=-1, keepdim=True) + 1e-20) * router.get("scale", 1.0)
    hr = _r(h, round_to)
    out = torch.zeros_like(h)
    for e in range(E + ident):
        rows, slot = (idx == e).nonzero(as_tuple=True)
        if rows.numel():
            y = expert(hr[rows], t, f"{p}e{e}.", limit, round_to) if e < E else h[rows]
            out[rows] += w[rows, slot].view(-1, 1) * y
    if mlp.get("shared"):
        y = expert(hr, t, p + "shared.", mlp["shared"]["limit"], round_to)
        out = out + torch.sigmoid(h @ t[p + "shared.sg"].T) * y
    return out, idx, choice


def feed_forward(h, mlp, t, p, round_to=None, choices=None):
    if mlp["kind"] == "dense":
        return dense(h, t, p, round_to), None, None
    return mixture(h, mlp, t, p, round_to, choices)


# ---------------------------------------------------------------------------------------------------------------
# the model
# ---------------------------------------------------------------------------------------------------------------
def layer_order(config):
    """(layer, whether the embedding output is added right before it) per layer run."""
    n, loop = len(config["layers"]), config.get("loop")
    if not loop:
        return [(i, False) for i in range(n)]
    a, b, times = loop["start"], loop["stop"], loop["times"]
    runs = [(i, False) for i in range(a)]
    for k in range(times):
        runs += [(i, k > 0 and i == a) for i in range(a, b)]
    return runs + [(i, False) for i in range(b, n)]


def forward(config: dict, tensors: Dict[str, torch.Tensor], tokens: List[int], round_to=None, layers_out=None,
            choices: Optional[List[torch.Tensor]] = None, choices_out: Optional[list] = None) -> torch.Tensor:
    """Logits [n, vocab] of one sequence from position 0.  ``layers_out``: a list that receives the residual stream
    after every layer run.  ``choices``: per mixture run (in order) the experts to follow.  ``choices_out``: a list
    that receives, per mixture run, (choice scores [n, N], chosen experts [n, top])."""
    t = {k: (v.to(F64) if v.is_floating_point() else v) for k, v in tensors.items()}
    eps = config["norm"]["eps"]
    x0 = t["embed"][torch.tensor(tokens, dtype=torch.long)]
    x = x0.clone()
    routed = 0
    for i, again in layer_order(config):
        layer, p = config["layers"][i], f"l{i}."
        if again:
            x = x + x0
        y = side_by_side(rms(x, t[p + "norm1"], eps), layer["mixer"], t, p + "mix.", eps, round_to)
        if layer.get("mlp"):
            follow = None
            if layer["mlp"]["kind"] == "moe":
                follow = choices[routed] if choices is not None else None
                routed += 1
            f, idx, score = feed_forward(rms(x, t[p + "norm2"], eps), layer["mlp"], t, p + "mlp.", round_to, follow)
            if idx is not None and choices_out is not None:
                choices_out.append((score, idx))
            y = y + f
        x = x + y
        if layers_out is not None:
            layers_out.append(x.clone())
    logits = _r(rms(x, t["final.norm"], eps), round_to) @ t["embed"].T
    cap = config.get("logit_softcap")
    return cap * torch.tanh(logits / cap) if cap else logits


def load_folder(model_dir):
    import json
    import os

    from safetensors.torch import load_file
    with open(os.path.join(model_dir, "config.json")) as fh:
        cfg = json.load(fh)
    w = {k: (v.to(F64) if v.is_floating_point() else v) for k, v in
         load_file(os.path.join(model_dir, "model.safetensors")).items()}
    return cfg, w


def generate_greedy(config, W, prompt, n):
    toks, out = list(prompt), []
    for _ in range(n):
        nxt = int(torch.argmax(forward(config, W, toks)[-1]))
        out.append(nxt)
        toks.append(nxt)
    return out
