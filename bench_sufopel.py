"""``bench.py --preset sufopel``: prefill and decode throughput of the Sufopel architecture at layer sizes that resemble a
real model's, beside Latinex (the framework's closest architecture: latent attention beside a recurrent mixer with a
matrix state behind a short convolution, one mixer a layer, a routed mixture) at equal width and depth, both with random
bfloat16 weights on one B200.

Per width W, Sufopel has ten layers: two of latent attention (the fourth, and the eighth, which reads the fourth's latents)
with W / 128 heads of 128, a query latent of 3 W / 8 and a cached row of 256, and eight of the delta rule with W / 128 heads of
128 x 128, four taps and low-rank maps of 128.  The first layer has a dense feed-forward of 4 W; the others 16 experts of W / 2
in four groups of which two are kept, two a row.  A token brings W / 16 numbers for every layer.  Latinex is the configuration
of ``--preset latinex``: four layers of latent attention, three of windowed attention, three of state-space duality, the same
experts and a shared one.

Timing as in ``bench_notedra.py``: CUDA events after warm-up, a step's weights, state and cache exceed the L2 cache.
"""
from __future__ import annotations

import json
import time

from bench_latinex import latinex_config
from bench_notedra import _measure


def sufopel_config(W: int, vocab: int = 32768, positions: int = 16384) -> dict:
    heads = max(1, W // 128)
    latent = {"heads": heads, "dim": 128, "vdim": 128, "q_rank": 3 * W // 8, "kv_rank": 256, "scale": 128 ** -0.5}
    delta = {"heads": heads, "kv_heads": heads, "dim": 128, "vdim": 128, "conv": 4}
    moe = {"kind": "moe", "expert": {"ff": W // 2, "limit": 7.0},
           "router": {"experts": 16, "top": 2, "groups": {"count": 4, "keep": 2}}}
    layers = []
    for i in range(10):
        mixer = dict(latent) if i in (3, 7) else dict(delta)
        if i == 7:
            mixer["kv_from"] = 3
        layers.append({"type": "latent_attention" if i in (3, 7) else "channel_delta", "mixer": mixer,
                       "mlp": {"kind": "dense", "ff": 4 * W} if i == 0 else dict(moe)})
    return {"architecture": "Sufopel", "vocab": vocab, "width": W, "max_positions": positions, "norm": {"eps": 1e-6},
            "embedding": {"scale": 1.0}, "logit_scale": 1.0, "token_side": {"dim": W // 16}, "layers": layers}


def run(ns, pk, pk_kind) -> int:
    widths = [int(w) for w in ns.widths.split(",") if w.strip()]
    batches = [int(b) for b in ns.points.split(",") if b.strip()] or [8]
    t0 = time.time()
    sizes = {}
    for W in widths:
        cfg = sufopel_config(W, positions=max(16384, ns.context + ns.steps + 64, ns.prefill_tokens))
        sizes[str(W)] = {
            "sufopel": _measure("sufopel", cfg, ns.prefill_tokens, batches, ns.context, ns.steps, max(ns.warmup, 3)),
            "latinex": _measure("latinex", latinex_config(W), ns.prefill_tokens, batches, ns.context, ns.steps, max(ns.warmup, 3)),
        }
    first = sizes[str(widths[0])]["sufopel"]["decode"][str(batches[0])]
    print(json.dumps({
        "metric": "decode tokens/s, Sufopel layer sizes beside Latinex at equal width (random bf16 weights)",
        "value": first["tokens_per_s"], "unit": "tokens/s", "n_gpus": 1, "steps": ns.steps, "warmup": max(ns.warmup, 3),
        "ms_per_step": first["ms_per_step"], "higher_is_better": True, "dtype": "bf16", "data": "synthetic",
        "config": {"preset": "sufopel", "widths": widths, "prefill_tokens": ns.prefill_tokens, "context": ns.context,
                   "batches": batches, "l2": "weights, state and cache of a step exceed the L2 cache"},
        "peaks": dict(pk, kind=pk_kind), "sizes": sizes, "seconds": round(time.time() - t0, 1)}))
    return 0
