"""``bench.py --preset radupel``: prefill and decode throughput of the Radupel architecture at layer sizes that resemble a
real model's, beside Notedra (the framework's closest architecture: parallel layers, a linear memory per head, attention
with a partial rotation, a mixture with a choice correction, a looped span of layers) at equal width and depth, both with
random bfloat16 weights on one B200.

Per width W, Radupel has five layers that all run twice (ten layer runs), each with both branches: attention with W / 128
heads of 128 (a quarter as many key/value heads), four taps and a rotation of 64 elements, and linear attention with
W / 256 heads of 128 x 128.  The second layer has a dense feed-forward of 4 W; the others 16 experts of W / 2 and two
identity experts in two groups, two a row, and a shared expert of W / 2.  Notedra (``--preset notedra``) has one mixer a
layer, a window of 1024 positions, the same experts and no shared one.

Timing as in ``bench_notedra.py``: CUDA events after warm-up, a step's weights, state and cache exceed the L2 cache.
"""
from __future__ import annotations

import json
import time

from bench_notedra import _measure, notedra_config


def radupel_config(W: int, vocab: int = 32768) -> dict:
    ah, lh = max(1, W // 128), max(1, W // 256)
    mixer = {"left": {"heads": ah, "kv_heads": max(1, ah // 4), "dim": 128, "vdim": 128, "scale": 128 ** -0.5, "conv": 4,
                      "rot": {"dims": 64, "base": 500000.0}},
             "right": {"heads": lh, "dim": 128, "vdim": 128, "decay": [1.0 - 2.0 ** (-4 - i % 8) for i in range(lh)]},
             "left_scale": 1.0, "right_scale": 0.5}
    moe = {"kind": "moe", "expert": {"ff": W // 2, "limit": 7.0},
           "router": {"experts": 16, "top": 2, "scale": 2.0, "identity": 2, "groups": {"count": 2, "keep": 1}},
           "shared": {"ff": W // 2, "limit": 7.0}}
    layers = [{"type": "parallel", "mixer": dict(mixer), "mlp": {"kind": "dense", "ff": 4 * W} if i == 1 else dict(moe)}
              for i in range(5)]
    return {"architecture": "Radupel", "vocab": vocab, "width": W, "norm": {"eps": 1e-6}, "logit_softcap": 30.0,
            "layers": layers, "loop": {"start": 0, "stop": 5, "times": 2}}


def run(ns, pk, pk_kind) -> int:
    widths = [int(w) for w in ns.widths.split(",") if w.strip()]
    batches = [int(b) for b in ns.points.split(",") if b.strip()] or [8]
    t0 = time.time()
    sizes = {}
    for W in widths:
        sizes[str(W)] = {
            "radupel": _measure("radupel", radupel_config(W), ns.prefill_tokens, batches, ns.context, ns.steps, max(ns.warmup, 3)),
            "notedra": _measure("notedra", notedra_config(W), ns.prefill_tokens, batches, ns.context, ns.steps, max(ns.warmup, 3)),
        }
    first = sizes[str(widths[0])]["radupel"]["decode"][str(batches[0])]
    print(json.dumps({
        "metric": "decode tokens/s, Radupel layer sizes beside Notedra at equal width (random bf16 weights)",
        "value": first["tokens_per_s"], "unit": "tokens/s", "n_gpus": 1, "steps": ns.steps, "warmup": max(ns.warmup, 3),
        "ms_per_step": first["ms_per_step"], "higher_is_better": True, "dtype": "bf16", "data": "synthetic",
        "config": {"preset": "radupel", "widths": widths, "prefill_tokens": ns.prefill_tokens, "context": ns.context,
                   "batches": batches, "l2": "weights, state and cache of a step exceed the L2 cache"},
        "peaks": dict(pk, kind=pk_kind), "sizes": sizes, "seconds": round(time.time() - t0, 1)}))
    return 0
