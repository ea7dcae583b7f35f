"""Small Radupel configurations for the tests, and folders with random weights for them.

The configurations differ from each other in every size; between them they cover: attention with one key head, one per
query head and groups, values wider and narrower than keys, head sizes that the tensor-core kernels take (64, 128) and
that they do not (odd ones, 144), rotations of part of a head, of all of it and none, convolutions of 1 to 6 taps; linear
attention with decays from 0 to 1, key sizes of 1 to 300, values wider and narrower than keys; branch factors of either
sign; layers without a feed-forward, dense ones, mixtures of one to sixteen experts with zero to four identity experts, in
one to four groups of which one to all are kept, one to four experts a row, with and without a shared expert; loops from
the first layer, in the middle, over all layers, of one pass and none; widths that are no multiple of 8; logits with and
without a cap; sizes of one and two everywhere.

Random weights alone would hide some faults, so ``write`` edits a few tensors afterwards: the taps of the convolutions are
all of one size (a lost input shows), router corrections are spread over both signs (they decide choices, and a choice
score below zero must still beat one that is not allowed), router rows are large (a peaked softmax), biases are visible.
The score factors in the configurations are large (single keys carry a row's output), the limits of the clamped gates
lie inside the range of the products, and slow decays keep hundreds of tokens.
"""
from __future__ import annotations

import os

import torch


def dense(ff):
    return {"kind": "dense", "ff": ff}


def moe(experts, top, ff, limit, identity=0, groups=None, scale=1.0, shared=None):
    """``groups`` = (count, keep), ``shared`` = (ff, limit)."""
    router = {"experts": experts, "top": top, "scale": scale, "identity": identity}
    if groups:
        router["groups"] = {"count": groups[0], "keep": groups[1]}
    return {"kind": "moe", "expert": {"ff": ff, "limit": limit}, "router": router,
            "shared": {"ff": shared[0], "limit": shared[1]} if shared else None}


def left(heads, kv, dim, vdim, scale, conv, rot=None):
    m = {"heads": heads, "kv_heads": kv, "dim": dim, "vdim": vdim, "scale": scale, "conv": conv}
    if rot:
        m["rot"] = {"dims": rot[0], "base": rot[1]}
    return m


def right(heads, dim, vdim, decay):
    return {"heads": heads, "dim": dim, "vdim": vdim, "decay": list(decay)}


def layer(lft, rgt, scales, mlp):
    return {"type": "parallel", "mixer": {"left": lft, "right": rgt, "left_scale": scales[0], "right_scale": scales[1]},
            "mlp": mlp}


def top(vocab, width, eps, cap, layers, loop=None):
    out = {"architecture": "Radupel", "vocab": vocab, "width": width, "norm": {"eps": eps}, "logit_softcap": cap,
           "layers": layers}
    if loop:
        out["loop"] = dict(zip(("start", "stop", "times"), loop))
    return out


# A: values wider than keys, a short rotation; a loop in the middle, over a layer without a feed-forward and a mixture with
# identity experts of which the groups of three keep two; a dense layer before and behind.
CASE_A = top(97, 64, 1e-5, 3.0, [
    layer(left(4, 2, 16, 24, 0.5, 3, (8, 100.0)), right(3, 8, 12, (0.5, 0.97, 0.999)), (0.8, 1.3), dense(40)),
    layer(left(2, 1, 24, 16, 0.35, 4, (24, 1000.0)), right(2, 16, 8, (0.9, 0.995)), (1.1, -0.6), None),
    layer(left(4, 4, 16, 16, 0.5, 2, None), right(1, 24, 20, (0.998,)), (-0.7, 0.9),
          moe(7, 3, 24, 1.0, identity=2, groups=(3, 2), scale=1.7, shared=(40, 0.8))),
    layer(left(3, 1, 16, 8, 0.5, 3, (4, 50.0)), right(2, 8, 8, (0.0, 0.99)), (1.0, 0.5), dense(24)),
], loop=(1, 3, 2))

# B: a width that is no multiple of 8 (no library product, no tensor-core expert product); odd head sizes, rotations of
# pairs that fit no vector; the longest convolution; one tap; a loop of a single pass; a mixture without groups, identity or
# shared expert, and one whose experts are half identity; no cap.
CASE_B = top(61, 52, 1e-4, 0.0, [
    layer(left(3, 3, 10, 7, 0.6, 6, (6, 30.0)), right(2, 5, 7, (0.7, 0.999)), (1.2, 0.7),
          moe(3, 3, 12, 1.4, scale=0.6)),
    layer(left(2, 1, 9, 11, 0.8, 2, (2, 10.0)), right(3, 7, 3, (0.9, 0.99, 1.0)), (0.9, 1.1), dense(19)),
    layer(left(1, 1, 12, 12, 1.1, 1, None), right(1, 3, 10, (0.6,)), (0.6, -1.2),
          moe(4, 2, 10, 0.7, identity=4, groups=(4, 2), scale=2.0, shared=(9, 1.2))),
], loop=(0, 2, 1))

# C: sizes that the tensor-core kernels take: heads of 64 (one key head for four) and of 128 (two for two), linear attention
# of 64 x 128, 128 x 64 and 96 x 96; sixteen experts in four groups of which two are kept, identity experts in the last
# group; a single expert; no loop.
CASE_C = top(131, 128, 1e-6, 6.0, [
    layer(left(4, 1, 64, 64, 0.3, 4, (32, 30000.0)), right(2, 64, 128, (0.9, 0.998)), (0.7, 0.8),
          moe(13, 4, 32, 1.3, identity=3, groups=(4, 2), scale=1.5, shared=(48, 1.1))),
    layer(left(2, 2, 128, 128, 0.2, 3, (128, 10000.0)), right(1, 128, 64, (0.997,)), (1.1, 0.4), dense(96)),
    layer(left(4, 2, 64, 32, 0.35, 5, (16, 500.0)), right(3, 96, 96, (0.3, 0.98, 0.9995)), (0.5, 1.0),
          moe(1, 1, 32, 2.0, shared=(32, 0.9))),
])

# D: ones and twos wherever a size can be one or two; a loop of one layer four times from the first layer on.
CASE_D = top(23, 16, 1e-5, 2.5, [
    layer(left(1, 1, 2, 1, 1.2, 2, (2, 10.0)), right(1, 1, 1, (0.9,)), (1.0, 1.0), moe(1, 1, 1, 1.0, identity=1)),
    layer(left(2, 1, 1, 2, 1.3, 1, None), right(2, 2, 1, (0.5, 0.95)), (0.7, 0.9), dense(1)),
    layer(left(2, 2, 2, 2, 1.1, 3, (2, 3.0)), right(1, 1, 2, (0.99,)), (0.9, -0.8),
          moe(2, 2, 1, 0.8, identity=2, groups=(2, 1), scale=1.3, shared=(2, 1.0))),
    layer(left(1, 1, 1, 1, 1.0, 2, None), right(1, 2, 2, (0.97,)), (1.0, 1.0), None),
], loop=(0, 1, 4))

# E: the largest sizes: heads of 144 (no tensor-core attention) and of 128 with values of 64; linear attention of 160 x 40 and
# 300 x 24; a loop over all layers.
CASE_E = top(50, 96, 1e-5, 4.0, [
    layer(left(2, 1, 144, 96, 0.15, 4, (48, 5000.0)), right(2, 160, 40, (0.99, 0.9)), (0.9, 0.6), dense(72)),
    layer(left(3, 1, 128, 64, 0.2, 2, (64, 100.0)), right(1, 300, 24, (0.996,)), (0.8, 0.7),
          moe(5, 2, 16, 1.0, identity=1, groups=(2, 1), scale=2.2, shared=(8, 1.5))),
], loop=(0, 2, 2))

# config, std of the weights, seed
CASES = {"A": (CASE_A, 0.12, 61), "B": (CASE_B, 0.15, 62), "C": (CASE_C, 0.1, 63), "D": (CASE_D, 0.5, 64),
         "E": (CASE_E, 0.1, 65)}


def drawn_config(seed: int) -> dict:
    """A configuration drawn from a seeded generator: two to six layers, widths of 64 to 320, any grouping, head sizes of 16
    to 128 for attention and 8 to 160 for linear attention, one to five taps, every kind of feed-forward, loops or none."""
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
        ident = r.choice([0, 0, 1, 2])
        count = r.choice([c for c in (1, 2, 3, 4) if N % c == 0])
        keep = r.randint(1, count)
        return moe(N - ident, r.randint(1, min(keep * (N // count), 4)), r.choice([16, 24, 40, 64]),
                   r.choice([0.7, 1.2, 3.0]), identity=ident, groups=(count, keep) if count > 1 else None,
                   scale=r.choice([1.0, 1.8]), shared=r.choice([None, (32, 1.0), (64, 2.0)]))

    layers = []
    for _ in range(r.randint(2, 6)):
        G, d = r.choice([1, 2, 4]), r.choice([16, 32, 64, 64, 128, 40])
        H = r.choice([1, 2, 3, 4])
        rot = r.choice([None, (d, 10000.0), (d // 2, 500.0), (8, 100000.0)])
        layers.append(layer(left(G * r.choice([1, 2, 3]), G, d, r.choice([d, d, 64, 32]), r.choice([0.1, 0.15, 0.2]),
                                 r.randint(1, 5), rot),
                            right(H, r.choice([8, 32, 64, 128, 160]), r.choice([8, 32, 64, 128]),
                                  [r.choice([0.2, 0.7, 0.95, 0.99, 0.999]) for _ in range(H)]),
                            (r.choice([0.5, 1.0, 1.4]), r.choice([0.5, 1.0, -0.8])), mlp()))
    loop = None
    if r.random() < 0.7:
        a = r.randrange(len(layers))
        loop = (a, r.randint(a + 1, len(layers)), r.choice([1, 2, 3]))
    return top(r.choice([100, 333, 1000]), W, r.choice([1e-6, 1e-5]), r.choice([0.0, 5.0, 15.0]), layers, loop)


def one_layer(name: str, index: int, mlp="same") -> dict:
    """A case's configuration cut down to one of its layers (``mlp``: the layer's own, or a replacement)."""
    cfg = {k: v for k, v in CASES[name][0].items() if k != "loop"}
    one = dict(cfg["layers"][index])
    if mlp != "same":
        one["mlp"] = mlp
    cfg["layers"] = [one]
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
        elif key.endswith(".correction"):
            new = 0.8 * (rnd - 0.6)                      # mostly negative choice scores
        elif key.endswith(".router"):
            new = t.float() * 3.0
        elif key.endswith(".b"):
            new = 0.8 * (rnd - 0.5)
        else:
            continue
        tensors[key] = new.to(t.dtype)
    safetensors_io.save_file(sorted(tensors.items()), path, metadata={"format": "pt"})
    return out_dir
