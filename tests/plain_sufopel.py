"""A plain, slow statement of the Sufopel design in float64, one function per mechanism.

Nothing here is shared with the engine: the tests compare the engine's logits with these functions on small random
models.  A model is a configuration dictionary (the keys of ``config.json``) and a dictionary of tensors by file name.

Notation: ``x`` is the residual stream ``[n, W]`` of one sequence whose first row is position 0; matrices are stored
``[out, in]`` and applied as ``x @ W.T``.  A layer is

    x += ls1 * rms(mixer(rms(x) w1)) w1b ;   x += ls2 * rms(ff(rms(x) w2)) w2b ;   x += rms(P (gelu(G x) * e)) ws

with ``e`` the layer's slice of a per-token table.  ``round_to`` (a torch dtype or None) rounds the operands of matrix
products, so that what rounding alone does can be measured; None keeps everything in float64.
"""
from __future__ import annotations

import math
from typing import Dict, List, Optional

import torch

F64 = torch.float64


def _r(t: torch.Tensor, round_to) -> torch.Tensor:
    return t if round_to is None else t.to(round_to).to(F64)


def unit_rms(x, eps):
    return x / torch.sqrt((x * x).mean(dim=-1, keepdim=True) + eps)


def rms(x, w, eps):
    return unit_rms(x, eps) * w


def silu(z):
    return z * torch.sigmoid(z)


def gelu_tanh(z):
    return 0.5 * z * (1.0 + torch.tanh(math.sqrt(2.0 / math.pi) * (z + 0.044715 * z ** 3)))


# ---------------------------------------------------------------------------------------------------------------
# embedding and the per-token input of a layer
# ---------------------------------------------------------------------------------------------------------------
def embedding(config, t, tokens):
    ids = torch.tensor(tokens, dtype=torch.long)
    return t["embed"][ids] * config["embedding"]["scale"] + t["pos"][: len(tokens)]


def token_side(x, tokens, layer, config, t, round_to=None):
    """What layer ``layer`` adds to the stream from its slice of the token's side vector."""
    dim, p = config["token_side"]["dim"], f"l{layer}.side."
    e = t["side.embed"][torch.tensor(tokens, dtype=torch.long)][:, layer * dim: (layer + 1) * dim]
    g = gelu_tanh(_r(x, round_to) @ t[p + "gate"].T) * e
    return rms(_r(g, round_to) @ t[p + "proj"].T, t[p + "norm"], config["norm"]["eps"])


# ---------------------------------------------------------------------------------------------------------------
# latent attention
# ---------------------------------------------------------------------------------------------------------------
def causal_softmax(scores):
    """scores [heads, n, n]: softmax of every row over the columns up to its own."""
    n = scores.shape[-1]
    visible = torch.arange(n).view(1, n) <= torch.arange(n).view(n, 1)
    s = scores.masked_fill(~visible, -math.inf)
    e = torch.exp(s - s.max(dim=-1, keepdim=True).values)
    return e / e.sum(dim=-1, keepdim=True)


def latent(h, t, p, eps, round_to=None):
    """The one vector per token from which keys and values are made: [n, kv_rank]."""
    return rms(_r(h, round_to) @ t[p + "dkv"].T, t[p + "dkv.norm"], eps)


def latent_attention(h, c, m, t, p, eps, round_to=None):
    """Queries from ``h`` [n, W], keys and values from the latents ``c`` [n, kv_rank]."""
    n, H, d, dv = h.shape[0], m["heads"], m["dim"], m["vdim"]
    h, c = _r(h, round_to), _r(c, round_to)
    cq = rms(h @ t[p + "dq"].T, t[p + "dq.norm"], eps)
    q = (_r(cq, round_to) @ t[p + "uq"].T).view(n, H, d)
    k, v = (c @ t[p + "uk"].T).view(n, H, d), (c @ t[p + "uv"].T).view(n, H, dv)
    q, k, v = _r(q, round_to), _r(k, round_to), _r(v, round_to)
    w = causal_softmax(torch.einsum("ihd,jhd->hij", q, k) * m["scale"])
    o = torch.einsum("hij,jhd->ihd", w, v).reshape(n, H * dv)
    o = o * torch.sigmoid(h @ t[p + "g"].T)
    return _r(o, round_to) @ t[p + "o"].T


# ---------------------------------------------------------------------------------------------------------------
# the delta rule with a decay per key channel
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


def unit(x):
    return x / torch.sqrt((x * x).sum(dim=-1, keepdim=True) + 1e-6)


def delta_rule(q, k, v, g, beta, state=None):
    """Row by row, per head: ``S <- g * S`` (g scales the rows of S), ``u = beta (v - S^T k)``, ``S <- S + k u^T``,
    ``o = S^T q``.  q, k, g [n, H, d], v [n, H, dv], beta [n, H] -> o [n, H, dv] and S [H, d, dv]."""
    n, H, d = q.shape
    S = torch.zeros(H, d, v.shape[-1], dtype=q.dtype) if state is None else state.clone()
    out = []
    for i in range(n):
        S = g[i].unsqueeze(-1) * S
        u = beta[i].unsqueeze(-1) * (v[i] - torch.einsum("hdv,hd->hv", S, k[i]))
        S = S + k[i].unsqueeze(-1) * u.unsqueeze(-2)
        out.append(torch.einsum("hdv,hd->hv", S, q[i]))
    return torch.stack(out), S


def channel_decay(h, m, t, p, round_to=None):
    """``exp(-exp(A_log) softplus(W_a2 W_a1 h + dt_bias))``: [n, heads, dim], every number in (0, 1)."""
    z = _r(_r(h, round_to) @ t[p + "a1"].T, round_to) @ t[p + "a2"].T + t[p + "dt_bias"]
    z = torch.log1p(torch.exp(-z.abs())) + z.clamp(min=0)
    return torch.exp(-torch.exp(t[p + "A_log"]).view(1, -1, 1) * z.view(h.shape[0], m["heads"], m["dim"]))


def delta_inputs(h, m, t, p, round_to=None):
    """q, k, g [n, H, d], v [n, H, dv], beta [n, H] of every row of ``h`` [n, W]."""
    n, H, G, d, dv = h.shape[0], m["heads"], m["kv_heads"], m["dim"], m["vdim"]
    hr = _r(h, round_to)
    q, k, v = (silu(causal_conv(hr @ t[p + s].T, t[p + s + ".conv"])) for s in "qkv")
    q = unit(q.view(n, G, d)).repeat_interleave(H // G, dim=1) * d ** -0.5
    k = unit(k.view(n, G, d)).repeat_interleave(H // G, dim=1)
    return q, k, v.view(n, H, dv), channel_decay(h, m, t, p, round_to), torch.sigmoid(hr @ t[p + "b"].T)


def channel_delta(h, m, t, p, eps, round_to=None):
    n, H, dv = h.shape[0], m["heads"], m["vdim"]
    q, k, v, g, beta = delta_inputs(h, m, t, p, round_to)
    o, _ = delta_rule(q, k, v, g, beta)
    gate = torch.sigmoid(_r(_r(h, round_to) @ t[p + "g1"].T, round_to) @ t[p + "g2"].T)
    o = rms(o, t[p + "norm"], eps).reshape(n, H * dv) * gate
    return _r(o, round_to) @ t[p + "o"].T


# ---------------------------------------------------------------------------------------------------------------
# feed-forwards
# ---------------------------------------------------------------------------------------------------------------
def dense(h, t, p, round_to=None):
    h = _r(h, round_to)
    return _r(silu(h @ t[p + "gate"].T) * (h @ t[p + "up"].T), round_to) @ t[p + "down"].T


def expert(h, t, p, limit, round_to=None):
    """``g = min(Wg h, limit)``, ``u = clamp(Wu h, -limit, limit)``, ``Wd (g sigmoid(1.702 g) (u + 1))``."""
    g = torch.clamp(h @ t[p + "gate"].T, max=limit)
    u = torch.clamp(h @ t[p + "up"].T, min=-limit, max=limit)
    return _r(g * torch.sigmoid(1.702 * g) * (u + 1.0), round_to) @ t[p + "down"].T


def group_scores(choice, count):
    """A group's score: the sum of its two largest choice scores (of its only one in a group of one).  [n, count]."""
    per = choice.shape[1] // count
    return torch.topk(choice.view(-1, count, per), min(2, per), dim=-1).values.sum(-1)


def allowed_experts(choice, count, keep):
    """Which experts may be chosen: those of the ``keep`` groups with the largest scores.  bool [n, E]."""
    n, E = choice.shape
    kept = torch.topk(group_scores(choice, count), keep, dim=-1).indices
    ok = torch.zeros(n, count, dtype=torch.bool)
    ok[torch.arange(n).view(n, 1), kept] = True
    return ok.repeat_interleave(E // count, dim=1)


def choose(choice, router):
    """The ``top`` experts with the largest choice scores among those of the kept groups: [n, top]."""
    groups = router.get("groups")
    if groups:
        choice = choice.masked_fill(~allowed_experts(choice, groups["count"], groups["keep"]), -math.inf)
    return torch.topk(choice, router["top"], dim=-1).indices


def mixture(h, mlp, t, p, round_to=None, choices=None):
    """``choices`` [n, top]: experts to use instead of the router's own (their weights still come from the scores).
    Returns (output, chosen [n, top], choice scores [n, E])."""
    router, limit = mlp["router"], mlp["expert"]["limit"]
    s = torch.sigmoid(h @ t[p + "router"].T)
    choice = s + t[p + "correction"]
    idx = choose(choice, router) if choices is None else choices.to(torch.long)
    w = torch.gather(s, 1, idx)
    hr = _r(h, round_to)
    out = torch.zeros_like(h)
    for e in range(router["experts"]):
        rows, slot = (idx == e).nonzero(as_tuple=True)
        if rows.numel():
            out[rows] += w[rows, slot].view(-1, 1) * expert(hr[rows], t, f"{p}e{e}.", limit, round_to)
    return out, idx, choice


def feed_forward(h, mlp, t, p, round_to=None, choices=None):
    if mlp["kind"] == "dense":
        return dense(h, t, p, round_to), None, None
    return mixture(h, mlp, t, p, round_to, choices)


# ---------------------------------------------------------------------------------------------------------------
# the model
# ---------------------------------------------------------------------------------------------------------------
def forward(config: dict, tensors: Dict[str, torch.Tensor], tokens: List[int], round_to=None, layers_out=None,
            choices: Optional[List[torch.Tensor]] = None, choices_out: Optional[list] = None) -> torch.Tensor:
    """Logits [n, vocab] of one sequence from position 0.  ``layers_out``: a list that receives the residual stream
    after every layer.  ``choices``: per mixture layer (in order) the experts to follow.  ``choices_out``: a list that
    receives, per mixture layer, (choice scores [n, E], chosen experts [n, top])."""
    t = {k: (v.to(F64) if v.is_floating_point() else v) for k, v in tensors.items()}
    eps = config["norm"]["eps"]
    x = embedding(config, t, tokens)
    routed, latents = 0, {}
    for i, layer in enumerate(config["layers"]):
        p, m = f"l{i}.", layer["mixer"]
        h = rms(x, t[p + "norm1"], eps)
        if layer["type"] == "channel_delta":
            y = channel_delta(h, m, t, p + "mix.", eps, round_to)
        else:
            j = m.get("kv_from")
            if j is None:
                latents[i] = latent(h, t, p + "mix.", eps, round_to)
            y = latent_attention(h, latents[i if j is None else j], m, t, p + "mix.", eps, round_to)
        x = x + t[p + "ls1"] * rms(y, t[p + "norm1b"], eps)
        if layer.get("mlp"):
            follow = None
            if layer["mlp"]["kind"] == "moe":
                follow = choices[routed] if choices is not None else None
                routed += 1
            f, idx, score = feed_forward(rms(x, t[p + "norm2"], eps), layer["mlp"], t, p + "mlp.", round_to, follow)
            if idx is not None and choices_out is not None:
                choices_out.append((score, idx))
            x = x + t[p + "ls2"] * rms(f, t[p + "norm2b"], eps)
        x = x + token_side(x, tokens, i, config, t, round_to)
        if layers_out is not None:
            layers_out.append(x.clone())
    return _r(rms(x, t["final.norm"], eps), round_to) @ t["head"].T * config["logit_scale"]


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
