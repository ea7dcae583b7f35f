"""Small Sufopel configurations for the tests, and folders with random weights for them.

The configurations differ from each other in every size; between them they cover: latent attention with few and many heads,
values wider and narrower than keys, cached rows that the tensor-core kernels take (up to 512), that they do not, and of odd
sizes; layers that borrow latents, several from one, with other heads and sizes than the lender; the delta rule with one key
head for several heads and one each, key sizes of 1 to 300 (beyond what is cut into chunks), values wider and narrower than
keys, convolutions of 1 to 7 taps, low-rank maps of unequal sizes; layers without a feed-forward, dense ones, mixtures of one
to sixteen experts in groups of one to four, of which one to all are kept; widths that are no multiple of 8; sizes of one and
two everywhere; embedding and logit scales that differ.

Random weights alone would hide some faults, so ``write`` edits a few tensors afterwards: the taps of the convolutions are all
of one size (a lost input shows), the decays are spread from channels that forget at once to ones that keep hundreds of
tokens, the steps over (0, 1), router corrections over both signs (they decide choices, and a choice score below zero must
still beat one that is not allowed), router rows are large.  The score factors are large (single keys carry a row's output)
and the limits of the clamped gates lie inside the range of the products.
"""
from __future__ import annotations

import os

import torch


def dense(ff):
    return {"kind": "dense", "ff": ff}


def moe(experts, top, ff, limit, groups=None):
    """``groups`` = (count, keep)."""
    router = {"experts": experts, "top": top}
    if groups:
        router["groups"] = {"count": groups[0], "keep": groups[1]}
    return {"kind": "moe", "expert": {"ff": ff, "limit": limit}, "router": router}


def latent(heads, dim, vdim, q_rank, kv_rank, scale, mlp, kv_from=None):
    m = {"heads": heads, "dim": dim, "vdim": vdim, "q_rank": q_rank, "kv_rank": kv_rank, "scale": scale}
    if kv_from is not None:
        m["kv_from"] = kv_from
    return {"type": "latent_attention", "mixer": m, "mlp": mlp}


def delta(heads, kv_heads, dim, vdim, conv, ranks, mlp):
    m = {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "conv": conv, "a_rank": ranks[0], "g_rank": ranks[1]}
    return {"type": "channel_delta", "mixer": m, "mlp": mlp}


def top(vocab, width, positions, eps, scales, side, layers):
    """``scales`` = (embedding, logits)."""
    return {"architecture": "Sufopel", "vocab": vocab, "width": width, "max_positions": positions, "norm": {"eps": eps},
            "embedding": {"scale": scales[0]}, "logit_scale": scales[1], "token_side": {"dim": side}, "layers": layers}


# A: two heads to a key head, a borrowing layer with other heads and sizes than the lender, a layer without a feed-forward.
CASE_A = top(97, 64, 420, 1e-5, (1.7, 0.4), 12, [
    delta(4, 2, 16, 24, 3, (8, 12), dense(40)),
    latent(4, 16, 24, 24, 40, 0.5, moe(8, 3, 24, 1.0, (4, 2))),
    delta(6, 2, 24, 8, 4, (16, 8), None),
    latent(2, 24, 16, 16, 40, 0.4, dense(24), kv_from=1),
    delta(2, 2, 8, 32, 2, (4, 20), moe(6, 2, 16, 0.7)),
])

# B: a width that is no multiple of 8 (no library product, no tensor-core expert product) and odd sizes; the longest
# convolution and one of a single tap; groups of one expert; the lender last but one.
CASE_B = top(61, 52, 300, 1e-4, (0.8, 1.3), 5, [
    delta(3, 1, 5, 7, 7, (3, 5), moe(3, 2, 12, 1.4, (3, 2))),
    delta(2, 1, 9, 3, 1, (7, 2), dense(19)),
    latent(3, 7, 5, 11, 9, 0.9, moe(6, 4, 10, 0.7, (2, 2))),
    latent(1, 10, 12, 5, 9, 0.7, None, kv_from=2),
])

# C: sizes that the tensor-core kernels take; key sizes of 128 and 64; sixteen experts in four groups; a single expert.
CASE_C = top(131, 128, 512, 1e-6, (1.2, 0.6), 32, [
    delta(2, 1, 128, 64, 4, (32, 16), moe(16, 4, 32, 1.3, (4, 2))),
    latent(4, 64, 32, 64, 256, 0.3, dense(96)),
    delta(3, 3, 64, 128, 4, (24, 40), moe(1, 1, 32, 2.0)),
    latent(8, 32, 64, 32, 128, 0.35, moe(8, 3, 48, 1.1, (4, 3))),
    latent(2, 64, 64, 48, 256, 0.3, moe(12, 2, 24, 1.0, (3, 1)), kv_from=1),
    delta(1, 1, 96, 96, 3, (8, 8), dense(64)),
])

# D: ones and twos wherever a size can be one or two (a norm over a single element is its sign, which no rounding leaves
# alone: what is normed has two, and a large eps).
CASE_D = top(23, 16, 128, 3e-2, (1.0, 1.0), 1, [
    delta(1, 1, 2, 2, 2, (1, 1), moe(1, 1, 1, 1.0)),
    latent(1, 1, 2, 2, 2, 1.2, dense(1)),
    delta(2, 1, 2, 2, 1, (1, 2), moe(2, 2, 1, 0.8, (2, 2))),
    latent(2, 2, 1, 2, 2, 1.5, moe(2, 1, 2, 1.0, (2, 1)), kv_from=1),
    delta(2, 2, 3, 2, 3, (2, 1), None),
])

# E: the largest sizes: keys of 300 (walked whatever the portion) and of 256, cached rows of 560 (the general attention
# kernel); two layers that borrow from one.
CASE_E = top(50, 96, 256, 1e-5, (2.0, 0.7), 20, [
    delta(2, 1, 300, 24, 4, (16, 8), dense(72)),
    latent(2, 48, 40, 40, 560, 0.3, moe(4, 2, 16, 1.0, (2, 1))),
    delta(1, 1, 256, 40, 3, (8, 24), moe(10, 3, 16, 0.9, (2, 2))),
    latent(3, 24, 32, 24, 560, 0.4, None, kv_from=1),
    latent(1, 32, 24, 56, 560, 0.35, dense(40), kv_from=1),
])

# config, std of the weights, seed
CASES = {"A": (CASE_A, 0.12, 71), "B": (CASE_B, 0.15, 72), "C": (CASE_C, 0.1, 73), "D": (CASE_D, 0.5, 81), "E": (CASE_E, 0.1, 75)}


def drawn_config(seed: int) -> dict:
    """A configuration drawn from a seeded generator: two to six layers, widths of 64 to 320, any grouping of heads, key sizes
    of 8 to 160, cached rows of 24 to 256, one to five taps, every kind of feed-forward, some layers that borrow."""
    import random
    r = random.Random(seed)
    W = r.choice([64, 96, 128, 192, 256, 320])

    def mlp():
        k = r.random()
        if k < 0.15:
            return None
        if k < 0.5:
            return dense(r.choice([48, 72, 128, 200]))
        N = r.choice([4, 6, 8, 12, 18])
        count = r.choice([c for c in (1, 2, 3, 4) if N % c == 0])
        keep = r.randint(1, count)
        return moe(N, r.randint(1, min(keep * (N // count), 4)), r.choice([16, 24, 40, 64]), r.choice([0.7, 1.2, 3.0]),
                   groups=(count, keep) if count > 1 else None)

    layers = []
    for _ in range(r.randint(2, 6)):
        if r.random() < 0.6:
            G = r.choice([1, 2, 3])
            layers.append(delta(G * r.choice([1, 2, 3]), G, r.choice([8, 32, 40, 64, 128, 160]), r.choice([8, 32, 64, 128]),
                                r.randint(1, 5), (r.choice([4, 24, 32]), r.choice([8, 12, 40])), mlp()))
            continue
        lenders = [i for i, l in enumerate(layers) if l["type"] == "latent_attention" and "kv_from" not in l["mixer"]]
        j = r.choice(lenders) if lenders and r.random() < 0.5 else None
        rank = layers[j]["mixer"]["kv_rank"] if j is not None else r.choice([24, 48, 128, 200, 256])
        layers.append(latent(r.choice([1, 2, 4, 6]), r.choice([16, 32, 40, 64]), r.choice([16, 32, 64]), r.choice([16, 40, 96]), rank,
                             r.choice([0.15, 0.2, 0.3]), mlp(), kv_from=j))
    return top(r.choice([100, 333, 1000]), W, 1024, r.choice([1e-6, 1e-5]), (r.choice([0.5, 1.0, 3.0]), r.choice([0.3, 1.0])),
               r.choice([8, 12, 40]), layers)


def one_layer(name: str, index: int, mlp="same") -> dict:
    """A case's configuration cut down to one of its layers (with the lender in front where it borrows); ``mlp``: the layer's
    own, or a replacement."""
    cfg = dict(CASES[name][0])
    one = {**cfg["layers"][index], "mixer": dict(cfg["layers"][index]["mixer"])}
    if mlp != "same":
        one["mlp"] = mlp
    cfg["layers"] = [one]
    if one["mixer"].get("kv_from") is not None:
        cfg["layers"] = [{**CASES[name][0]["layers"][one["mixer"]["kv_from"]], "mlp": None}, one]
        one["mixer"]["kv_from"] = 0
    return cfg


def write(name: str, out_dir: str) -> str:
    """``config.json`` and ``model.safetensors`` for a case: seeded random weights, then the edits named above."""
    cfg, std, seed = CASES[name]
    return write_config(cfg, std, seed, out_dir)


def write_config(cfg: dict, std: float, seed: int, out_dir: str) -> str:
    from safetensors.torch import load_file

    from sharpinference_b200.weights import safetensors_io, write_random_model
    write_random_model(dict(cfg), out_dir, seed, std=std, norm_std=0.1)
    path = os.path.join(out_dir, "model.safetensors")
    tensors = load_file(path)
    g = torch.Generator().manual_seed(seed + 1000)
    for key in sorted(tensors):
        t = tensors[key]
        rnd = torch.rand(t.shape, generator=g)
        if key.endswith(".conv"):
            new = (0.4 + 0.6 * rnd) * torch.where(torch.rand(t.shape, generator=g) < 0.5, -1.0, 1.0)
        elif key.endswith(".A_log"):
            new = 2.0 * rnd - 1.0
        elif key.endswith(".dt_bias"):                   # slow channels, quick ones, and some that keep nothing at all
            new = torch.where(rnd < 0.1, torch.full_like(rnd, 30.0), -9.0 + 11.0 * rnd)
        elif key.endswith(".mix.b"):
            new = t.float() * 3.0
        elif key.endswith(".correction"):
            new = 0.8 * (rnd - 0.9)                      # mostly negative choice scores
        elif key.endswith(".router"):
            new = t.float() * 3.0
        else:
            continue
        tensors[key] = new.to(t.dtype)
    safetensors_io.save_file(sorted(tensors.items()), path, metadata={"format": "pt"})
    return out_dir
