"""Single-kernel timing at model sizes, for profiling one kernel without the model around it.

    python bench_kernels.py tc_gemm --mode gate_up --rows 2048 --row-tile 128
    python bench_kernels.py tc_gemm --mode down --rows 8
    python bench_kernels.py attention_decode --batch 64 --context 8192
    python bench_kernels.py attention_prefill --tokens 2048
    python bench_kernels.py dense --rows 8 --n 7168 --k 5120 --impl grouped
    python bench_kernels.py mlstm --batch 64 --tokens 1            (decode: the state streams through once)
    python bench_kernels.py mlstm --batch 1 --tokens 2048          (a prompt portion: float32 FMA work)
    python bench_kernels.py router_topk --tokens 2048 --experts 16 --top 2
    python bench_kernels.py wkv --batch 64 --tokens 1              (decode; --batch 1 --tokens 2048: a prompt)
    python bench_kernels.py scan --batch 64 --tokens 1             (convolution and selective scan)
    python bench_kernels.py streams --tokens 2048                  (stream update + grouped norm, token shift)
    python bench_kernels.py mixture_glue --tokens 2048             (activation, pair rows, combine)
    python bench_kernels.py ssd --batch 64 --tokens 1              (state-space duality and its gated norm)
    python bench_kernels.py attention_keys_decode --batch 64 --context 8192     (keys-only pages)
    python bench_kernels.py attention_keys_prefill --tokens 2048 --mask window
    python bench_kernels.py attention_prefill --tokens 2048 --softcap 30 --sinks        (capped scores, sinks)
    python bench_kernels.py lightning --batch 64 --tokens 1        (linear attention and its gated norm; --batch 1 --tokens 2048)
    python bench_kernels.py qkv_conv --tokens 2048                 (convolution, rotation, cache write)
    python bench_kernels.py softmax_mixture --tokens 2048          (router with groups, combine with identity experts)
    python bench_kernels.py delta --batch 64 --tokens 1            (delta rule and its gated norm; --batch 1 --tokens 2048)
    python bench_kernels.py delta_prep --tokens 2048               (convolution, unit norms, steps, low-rank columns)
    python bench_kernels.py sandwich --tokens 2048                 (normed update and norm, side gate, element gate, router)
    python bench_kernels.py elementwise --op add_rmsnorm_pair --tokens 2048 --hidden 2048
    python bench_kernels.py elementwise --op add_layernorm --tokens 2048 --hidden 2048

Each run warms the kernel up, times ``--iters`` launches with CUDA events and prints one line with
the time per launch and the achieved bytes or flops per second.  The inputs are larger than the L2
cache at the default sizes.  Profiler captures name this file so that they run committed code only.  It is a measuring tool beside
``bench.py``, not part of the package.
"""
from __future__ import annotations

import argparse
import math
import os
import sys

import torch

sys.path.insert(0, os.path.dirname(os.path.abspath(__file__)))

from sharpinference_b200.kernels import ops  # noqa: E402

DEV = "cuda:0"


USE_GRAPH = False


def _time(fn, iters: int, warmup: int = 3) -> float:
    """Milliseconds per call.  With --graph the calls are captured once and replayed, which takes the
    host's launch cost out of the measurement (short kernels are otherwise timed by it)."""
    for _ in range(warmup):
        fn()
    torch.cuda.synchronize()
    a, b = torch.cuda.Event(enable_timing=True), torch.cuda.Event(enable_timing=True)
    if USE_GRAPH:
        graph = torch.cuda.CUDAGraph()
        with torch.cuda.graph(graph):
            for _ in range(iters):
                fn()
        graph.replay()
        torch.cuda.synchronize()
        a.record()
        graph.replay()
        b.record()
    else:
        a.record()
        for _ in range(iters):
            fn()
        b.record()
    torch.cuda.synchronize()
    ops.check_status(DEV)
    return a.elapsed_time(b) / iters


def tc_gemm(ns) -> None:
    E, I, H, T = ns.experts, ns.inter, ns.hidden, ns.rows
    g = torch.Generator(device=DEV).manual_seed(0)
    used = min(E, ns.active) if ns.active else E
    counts = torch.zeros(E, dtype=torch.int64)
    if ns.skew > 0:
        share = torch.tensor([(1.0 - ns.skew) ** e for e in range(used)], dtype=torch.float64)
        counts[:used] = torch.floor(share / share.sum() * T).to(torch.int64)
    else:
        counts[:used] = T // used
    counts[: T - int(counts.sum())] += 1
    offsets = torch.cat([torch.zeros(1, dtype=torch.int64), torch.cumsum(counts, 0)]).to(torch.int32).to(DEV)
    if ns.mode == "gate_up":
        w = torch.empty(E, 2 * I, H, dtype=torch.bfloat16, device=DEV).normal_(0, 0.02, generator=g)
        a = torch.empty(T, H, dtype=torch.bfloat16, device=DEV).normal_(0, 1, generator=g)
        scale = torch.rand(T, device=DEV, generator=g)
        fn = lambda: ops.tc_grouped_gemm(a, w, offsets, mode=ops.TC_MODE_SWIGLU, row_scale=scale, row_tile=ns.row_tile,
                                         k_split=ns.k_split, max_ctas=ns.max_ctas)
        weight_bytes, flops = used * 2 * I * H * 2, 2 * T * 2 * I * H
    else:
        w = torch.empty(E, H, I, dtype=torch.bfloat16, device=DEV).normal_(0, 0.02, generator=g)
        a = torch.empty(T, I, dtype=torch.bfloat16, device=DEV).normal_(0, 1, generator=g)
        out = torch.zeros(T, H, device=DEV)
        rows = torch.randperm(T, device=DEV).to(torch.int32)
        fn = lambda: ops.tc_grouped_gemm(a, w, offsets, mode=ops.TC_MODE_STORE, out=out, out_rows=rows, accumulate=True,
                                         row_tile=ns.row_tile, k_split=ns.k_split, max_ctas=ns.max_ctas)
        weight_bytes, flops = used * H * I * 2, 2 * T * H * I
    if ns.beside:
        # the library's dense product (rows x N x K, operands in L2 for the most part) on a second stream beside
        # every launch: what a mixture layer's shared expert does while the routed experts stream their weights
        M2, N2, K2 = (int(v) for v in ns.beside.split(","))
        a2 = torch.randn(M2, K2, device=DEV).to(torch.bfloat16)
        w2 = torch.randn(N2, K2, device=DEV).to(torch.bfloat16)
        o2 = torch.empty(M2, N2, device=DEV)
        side = torch.cuda.Stream()
        dense = lambda: torch.mm(a2, w2.t(), out_dtype=torch.float32, out=o2)
        alone_dense = _time(dense, ns.iters)
        alone = _time(fn, ns.iters)
        inner = fn

        def fn():
            main = torch.cuda.current_stream()
            side.wait_stream(main)
            with torch.cuda.stream(side):
                for _ in range(ns.beside_count):
                    dense()
            inner()
            main.wait_stream(side)
        print(f"alone: grouped {alone * 1e3:.1f} us, dense {M2}x{N2}x{K2} {alone_dense * 1e3:.1f} us x {ns.beside_count} "
              f"({2 * M2 * N2 * K2 / alone_dense / 1e9:.0f} TFLOP/s)")
    ms = _time(fn, ns.iters)
    print(f"tc_gemm {ns.mode} rows={T} experts={used}/{E} row_tile={ops.tc_row_tile(T, ops.TC_MODE_SWIGLU if ns.mode == "gate_up" else ops.TC_MODE_STORE, E) if ns.row_tile is None else ns.row_tile}: {ms * 1e3:.1f} us, "
          f"weights {weight_bytes / ms / 1e6:.0f} GB/s, {flops / ms / 1e9:.0f} TFLOP/s")


def dense(ns) -> None:
    """A dense product of a few rows: the grouped tensor-core kernel with one group, the weight-streaming kernel for up to 16 rows, or the library.  The weights rotate through enough copies to exceed the L2 cache, as in a model of many layers."""
    M, N, K = ns.rows, ns.n, ns.k
    copies = max(2, (300 << 20) // (N * K * 2) + 1)
    ws = [torch.empty(N, K, dtype=torch.bfloat16, device=DEV).normal_(0, 0.02) for _ in range(copies)]
    a = torch.randn(M, K, device=DEV).to(torch.bfloat16)
    out = torch.empty(M, N, device=DEV)
    state = {"i": 0}

    def fn():
        w = ws[state["i"] % copies]
        state["i"] += 1
        if ns.impl == "grouped":
            ops.tc_dense(a, w, out=out)
        elif ns.impl == "rows":
            ops.dense_rows(a, w, swiglu=ns.swiglu, out=None if ns.swiglu else out)
        else:
            y = torch.mm(a, w.t(), out_dtype=torch.float32, out=out)
            if ns.swiglu:
                ops.swiglu(y, torch.bfloat16)
    ms = _time(fn, max(ns.iters, copies))
    print(f"dense {ns.impl} rows={M} N={N} K={K}{' swiglu' if ns.swiglu else ''}: {ms * 1e3:.1f} us, "
          f"weights {N * K * 2 / ms / 1e6:.0f} GB/s")


def router(ns) -> None:
    """Router logits, sigmoid and top-1 for a prompt portion's tokens (fp32), each call on another copy of the
    activations so that they come from memory as after the norm kernel of a long step."""
    T, H, E = ns.tokens, ns.hidden, ns.experts
    copies = max(2, (300 << 20) // (T * H * 4) + 1)
    hs = [torch.randn(T, H, device=DEV) for _ in range(copies)]
    wr = torch.randn(E, H, device=DEV) * 0.05
    state = {"i": 0}

    def fn():
        ops.router_top1(hs[state["i"] % copies], wr)
        state["i"] += 1
    ms = _time(fn, max(ns.iters, copies))
    print(f"router_top1 tokens={T} hidden={H} experts={E}: {ms * 1e3:.1f} us, "
          f"{(T * H * 4 + E * H * 4) / ms / 1e6:.0f} GB/s of activations and router rows read once")


def mlstm(ns) -> None:
    """The matrix-memory recurrence (gates, scan, head norm) for `batch` requests of `tokens` rows each.  Decode
    (tokens = 1) is a stream of the state: read and written once.  A prompt portion is float32 FMA work: per row and
    head 4 d dv flops (the update of S and S^T q)."""
    from sharpinference_b200.parts.mlstm import fused_mlstm_columns
    B, n, heads, d, dv = ns.batch, ns.tokens, ns.heads, ns.key_dim, ns.value_dim
    cq, ck, cv, cg, ci, cf, width = fused_mlstm_columns(heads, d, dv)
    T = B * n
    proj = torch.randn(T, width, device=DEV)
    proj[:, cf:cf + heads] += 3.0
    bias = torch.zeros(heads, device=DEV)
    w = torch.ones(heads * dv, device=DEV)
    per_head, per_request = ops.mlstm_state_floats(heads, d, dv)
    copies = max(1, (300 << 20) // (B * per_request * 4) + 1) if n == 1 else 1
    state = torch.zeros(copies * B, per_request, device=DEV)
    offs = torch.arange(0, T + 1, n, dtype=torch.int32, device=DEV)
    slot_sets = [torch.arange(c * B, (c + 1) * B, dtype=torch.int32, device=DEV) for c in range(copies)]
    it = {"i": 0}

    def fn():
        slots = slot_sets[it["i"] % copies]
        it["i"] += 1
        num, nq, coef = ops.mlstm_recurrence(proj, col_q=cq, col_k=ck, col_v=cv, col_i=ci, col_f=cf, bias_i=bias, bias_f=bias,
                                 row_offsets=offs, state_slots=slots, state=state, heads=heads, d=d, dv=dv, cap=15.0,
                                 q_scale=d ** -0.5)
        ops.mlstm_out(num, nq, coef, proj, cg, w, 1e-5, heads, dv, torch.bfloat16)
    ms = _time(fn, max(ns.iters, copies))
    state_bytes = 2 * B * per_request * 4
    flops = 4.0 * T * heads * d * dv
    print(f"mlstm batch={B} tokens={n} heads={heads} d={d} dv={dv}: {ms * 1e3:.1f} us, state {state_bytes / ms / 1e6:.0f} GB/s "
          f"(read and written once), {flops / ms / 1e9:.2f} TFLOP/s float32")


def wkv(ns) -> None:
    """The WKV recurrence and its output kernel for `batch` requests of `tokens` rows each.  Decode (tokens = 1)
    streams the state once (read and written); a prompt portion is float32 FMA work, 4 d d flops a row and head."""
    B, n, heads, d = ns.batch, ns.tokens, ns.heads, ns.head_dim
    T, hd = B * n, heads * d
    r, k, v, wraw, g = (0.5 * torch.randn(T, hd, device=DEV) for _ in range(5))
    w0, u, nw = torch.full((hd,), -3.0, device=DEV), torch.randn(hd, device=DEV), torch.ones(hd, device=DEV)
    per_request = heads * d * d
    copies = max(1, (300 << 20) // (B * per_request * 4) + 1) if n == 1 else 1
    state = torch.zeros(copies * B, per_request, device=DEV)
    offs = torch.arange(0, T + 1, n, dtype=torch.int32, device=DEV)
    slot_sets = [torch.arange(c * B, (c + 1) * B, dtype=torch.int32, device=DEV) for c in range(copies)]
    it = {"i": 0}

    def fn():
        slots = slot_sets[it["i"] % copies]
        it["i"] += 1
        o = ops.wkv_recurrence(r, k, v, wraw, w0, u, row_offsets=offs, state_slots=slots, state=state, heads=heads, d=d)
        ops.wkv_out(o, g, nw, 1e-5, heads, d, torch.bfloat16)
    ms = _time(fn, max(ns.iters, copies))
    print(f"wkv batch={B} tokens={n} heads={heads} d={d}: {ms * 1e3:.1f} us, state {2 * B * per_request * 4 / ms / 1e6:.0f} GB/s "
          f"(read and written once), {4.0 * T * heads * d * d / ms / 1e9:.2f} TFLOP/s float32")


def scan(ns) -> None:
    """The causal convolution (with the gate's silu), the softplus of the step sizes and the selective scan for `batch`
    requests of `tokens` rows each: per row, channel and state one exponential and four flops; decode streams the
    state once."""
    B, n, C, N, R = ns.batch, ns.tokens, ns.channels, ns.states, ns.dt_rank
    T = B * n
    xz, dbc, dtraw = torch.randn(T, 2 * C, device=DEV), 0.5 * torch.randn(T, R + 2 * N, device=DEV), torch.randn(T, C, device=DEV)
    conv_w, conv_b = 0.5 * torch.randn(C, ns.taps, device=DEV), torch.zeros(C, device=DEV)
    dt_b, a_log, dsk = torch.zeros(C, device=DEV), torch.zeros(C, N, device=DEV), torch.ones(C, device=DEV)
    copies = max(1, (300 << 20) // (B * C * N * 4) + 1) if n == 1 else 1
    state = torch.zeros(copies * B, C * N, device=DEV)
    conv_state = torch.zeros(copies * B, max(ns.taps - 1, 1) * C, device=DEV)
    offs = torch.arange(0, T + 1, n, dtype=torch.int32, device=DEV)
    rr = torch.arange(T, dtype=torch.int32, device=DEV) // n
    slot_sets = [torch.arange(c * B, (c + 1) * B, dtype=torch.int32, device=DEV) for c in range(copies)]
    it = {"i": 0}
    dtwork = torch.empty_like(dtraw)

    def fn():
        slots = slot_sets[it["i"] % copies]
        it["i"] += 1
        x32, _ = ops.causal_conv(xz, C, conv_w, conv_b, conv_state, row_request=rr, row_offsets=offs, state_slots=slots,
                                 act_dtype=torch.bfloat16, gate_col=C)
        dt = ops.bias_act(dtraw, dt_b, ops.ACT_SOFTPLUS, torch.float32, out=dtwork)
        ops.selective_scan(x32, dt, dbc, R, R + N, a_log, dsk, xz, C, row_offsets=offs, state_slots=slots,
                           state=state, out_dtype=torch.bfloat16)
    ms = _time(fn, max(ns.iters, copies))
    print(f"scan batch={B} tokens={n} channels={C} states={N}: {ms * 1e3:.1f} us, state {2 * B * C * N * 4 / ms / 1e6:.0f} GB/s "
          f"(read and written once), {T * C * N / ms / 1e6:.1f} G state updates/s (an exponential and four flops each)")


def streams(ns) -> None:
    """The stream update fused with the grouped norm, and the token shift, over `tokens` rows of `streams` streams:
    the streams are read and written once (2 S H floats a row), the sublayer output read once."""
    T, H, S = ns.tokens, ns.hidden, ns.streams
    x, y = torch.randn(T, S * H, device=DEV), torch.randn(T, H, device=DEV)
    mix, outc, inc = torch.eye(S, device=DEV).contiguous(), torch.ones(S, device=DEV), torch.full((S,), 1.0 / S, device=DEV)
    w, mu = torch.ones(H, device=DEV), torch.rand(1, H, device=DEV)
    state = torch.zeros(1, H, device=DEV)
    rr = torch.zeros(T, dtype=torch.int32, device=DEV)
    offs = torch.tensor([0, T], dtype=torch.int32, device=DEV)
    slots = torch.zeros(1, dtype=torch.int32, device=DEV)
    ms = _time(lambda: ops.hc_mix_norm(x, (y, mix, outc), inc, w, streams=S, groups=ns.groups, eps=1e-6,
                                       out_dtype=torch.bfloat16), ns.iters)
    print(f"stream update + norm tokens={T} width={H} streams={S}: {ms * 1e3:.1f} us, "
          f"{T * H * (8 * S + 4 + 2) / ms / 1e6:.0f} GB/s")
    h = torch.randn(T, H, device=DEV)
    ms = _time(lambda: ops.token_shift(h, mu, state, row_request=rr, row_offsets=offs, state_slots=slots,
                                       out_dtype=torch.bfloat16), ns.iters)
    print(f"token shift tokens={T} width={H}: {ms * 1e3:.1f} us, {T * H * 6 / ms / 1e6:.0f} GB/s")


def router_topk(ns) -> None:
    T, H, E = ns.tokens, ns.hidden, ns.experts
    copies = max(2, (300 << 20) // (T * H * 4) + 1)
    hs = [torch.randn(T, H, device=DEV) for _ in range(copies)]
    wr = torch.randn(E, H, device=DEV) * 0.05
    corr = torch.randn(E, device=DEV) * 0.1
    it = {"i": 0}

    def fn():
        ops.router_topk(hs[it["i"] % copies], wr, ns.top, correction=corr, scale=2.5)
        it["i"] += 1
    ms = _time(fn, max(ns.iters, copies))
    print(f"router_topk tokens={T} hidden={H} experts={E} top={ns.top}: {ms * 1e3:.1f} us, "
          f"{(T * H * 4 + E * H * 4) / ms / 1e6:.0f} GB/s of activations and router rows read once")


def mixture_glue(ns) -> None:
    """What stands between the grouped products of a top-k mixture: the activation over the first product, the rows
    of the sorted pairs, and the sum of a row's pairs."""
    T, H, I, k, E = ns.tokens, ns.hidden, ns.inter, ns.top, ns.experts
    P = T * k
    copies = max(2, (300 << 20) // (P * max(I, H) * 4) + 1)
    ups = [torch.randn(P, I, device=DEV) for _ in range(copies)]
    ys = [torch.randn(P, H, device=DEV) for _ in range(copies)]
    add = torch.randn(T, H, device=DEV)
    expert = torch.randint(0, E, (P,), device=DEV, dtype=torch.int32)
    it = {"i": 0}

    def act():
        ops.bias_act(ups[it["i"] % copies], None, ops.ACT_RELU2, torch.bfloat16)
        it["i"] += 1

    def combine():
        ops.moe_combine(ys[it["i"] % copies], k, add=add, out=add)
        it["i"] += 1

    def sort():
        _, pairs = ops.moe_sort(expert, E)
        ops.moe_pair_tokens(pairs, k)
    for name, fn, nbytes in (("bias_act relu2", act, P * I * 6), ("moe_combine", combine, P * H * 4 + 2 * T * H * 4),
                             ("moe_sort + pair_tokens", sort, P * 12)):
        ms = _time(fn, max(ns.iters, copies))
        print(f"{name} tokens={T} top={k}: {ms * 1e3:.1f} us, {nbytes / ms / 1e6:.0f} GB/s")


def elementwise(ns) -> None:
    """The memory-bound kernels between the products of a prompt step, each call on another copy of its inputs
    (copies that exceed L2 together), with the bytes each has to move."""
    T, H, I = ns.tokens, ns.hidden, ns.inter
    nq, nkv, d, ps = ns.heads, ns.kv_heads, ns.head_dim, ns.page_size
    state = {"i": 0}

    def rotate(items):
        def pick():
            state["i"] += 1
            return items[state["i"] % len(items)]
        return pick

    if ns.op == "add_rmsnorm":
        copies = max(2, (300 << 20) // (T * H * 8) + 1)
        xs = rotate([(torch.randn(T, H, device=DEV), torch.randn(T, H, device=DEV)) for _ in range(copies)])
        w = torch.ones(H, device=DEV)
        nbytes = T * H * (4 + 4 + 4 + 2 + (4 if ns.fp32_copy else 0))

        def fn():
            x, delta = xs()
            ops.add_rmsnorm(x, delta, w, 1e-5, torch.bfloat16, want_fp32=ns.fp32_copy)
    elif ns.op == "add_rmsnorm_pair":
        copies = max(2, (300 << 20) // (T * H * 8) + 1)
        xs = rotate([(torch.randn(T, H, device=DEV), torch.randn(T, H, device=DEV)) for _ in range(copies)])
        w1, w2 = torch.ones(H, device=DEV), torch.ones(H, device=DEV)
        nbytes = T * H * (4 + 4 + 4 + 2 + 2 + (4 if ns.fp32_copy else 0))

        def fn():
            x, delta = xs()
            ops.add_rmsnorm_pair(x, delta, w1, w2, 1e-5, torch.bfloat16, want_fp32=ns.fp32_copy)
    elif ns.op in ("add_layernorm", "add_dyt"):
        copies = max(2, (300 << 20) // (T * H * 8) + 1)
        xs = rotate([(torch.randn(T, H, device=DEV), torch.randn(T, H, device=DEV)) for _ in range(copies)])
        w, b, alpha = torch.ones(H, device=DEV), torch.zeros(H, device=DEV), torch.full((1,), 0.5, device=DEV)
        nbytes = T * H * (4 + 4 + 4 + 2 + (4 if ns.fp32_copy else 0))

        def fn():
            x, delta = xs()
            if ns.op == "add_layernorm":
                ops.add_layernorm(x, delta, w, b, 1e-5, torch.bfloat16, want_fp32=ns.fp32_copy)
            else:
                ops.add_dyt(x, delta, w, b, alpha, torch.bfloat16, want_fp32=ns.fp32_copy)
    elif ns.op == "qkv_post_wide":      # norm over the whole q and k, query factor, q store, keys and values into pages
        width = (nq + 2 * nkv) * d
        copies = max(2, (300 << 20) // (T * width * 4) + 1)
        qkvs = rotate([torch.randn(T, width, device=DEV) for _ in range(copies)])
        pages = (T + ps - 1) // ps
        kv = torch.zeros(pages, 2, nkv, ps, d, dtype=torch.bfloat16, device=DEV)
        table = torch.arange(pages, dtype=torch.int32, device=DEV).view(1, pages)
        positions = torch.arange(T, dtype=torch.int32, device=DEV)
        row_req = torch.zeros(T, dtype=torch.int32, device=DEV)
        wq, wk = torch.ones(nq * d, device=DEV), torch.ones(nkv * d, device=DEV)
        q = torch.empty(T, nq, d, dtype=torch.bfloat16, device=DEV)
        nbytes = T * width * 4 + T * width * 2
        fn = lambda: ops.qkv_post_wide(qkvs(), positions, row_req, table, q, kv, nq=nq, nkv=nkv, d=d, page_size=ps,
                                       q_weight=wq, k_weight=wk, eps=1e-6, q_count=nq * d, k_count=nkv * d, temp_coef=0.1,
                                       temp_every=128.0, write_kv=True, has_kv=True)
    elif ns.op == "swiglu":
        copies = max(2, (300 << 20) // (T * 2 * I * 4) + 1)
        gus = rotate([torch.randn(T, 2 * I, device=DEV) for _ in range(copies)])
        nbytes = T * I * (8 + 2)
        fn = lambda: ops.swiglu(gus(), torch.bfloat16)
    elif ns.op == "gather":
        copies = max(2, (300 << 20) // (T * H * 2) + 1)
        hs = rotate([torch.randn(T, H, device=DEV).to(torch.bfloat16) for _ in range(copies)])
        rows = torch.randperm(T, device=DEV).to(torch.int32)
        nbytes = T * H * 4
        fn = lambda: ops.gather_rows_bf16(hs(), rows)
    else:   # qkv_post: rotation, L2 norm, q store, keys and values into pages
        width = (nq + 2 * nkv) * d
        copies = max(2, (300 << 20) // (T * width * 4) + 1)
        qkvs = rotate([torch.randn(T, width, device=DEV) for _ in range(copies)])
        pages = (T + ps - 1) // ps
        kv = torch.zeros(pages, 2, nkv, ps, d, dtype=torch.bfloat16, device=DEV)
        table = torch.arange(pages, dtype=torch.int32, device=DEV).view(1, pages)
        positions = torch.arange(T, dtype=torch.int32, device=DEV)
        row_req = torch.zeros(T, dtype=torch.int32, device=DEV)
        inv_freq = (500000.0 ** (-torch.arange(0, d, 2, device=DEV, dtype=torch.float32) / d)).contiguous()
        q = torch.empty(T, nq, d, dtype=torch.bfloat16, device=DEV)
        nbytes = T * width * 4 + T * width * 2
        fn = lambda: ops.qkv_post(qkvs(), positions, row_req, table, inv_freq, q, kv, nq=nq, nkv=nkv, d=d, page_size=ps,
                                  pairing=ops.ROPE_INTERLEAVED, l2_eps=1e-5, temp_attn_scale=0.0, temp_floor_scale=0.0,
                                  write_kv=True)
    ms = _time(fn, max(ns.iters, 8))
    print(f"{ns.op} tokens={T}: {ms * 1e3:.1f} us, {nbytes / 1e6:.0f} MB -> {nbytes / ms / 1e6:.0f} GB/s")


def _cache(batch: int, context: int, nkv: int, d: int, ps: int):
    blocks = (context + ps - 1) // ps
    pages = batch * blocks
    kv = torch.empty(pages, 2, nkv, ps, d, dtype=torch.bfloat16, device=DEV).normal_(0, 1)
    table = torch.randperm(pages, device=DEV).to(torch.int32).view(batch, blocks).contiguous()
    return kv, table


def attention_decode(ns) -> None:
    B, S, nq, nkv, d, ps = ns.batch, ns.context, ns.heads, ns.kv_heads, ns.head_dim, ns.page_size
    kv, table = _cache(B, S, nkv, d, ps)
    q = torch.randn(B, nq, d, device=DEV).to(torch.bfloat16)
    positions = torch.full((B,), S - 1, dtype=torch.int32, device=DEV)
    if ns.others_context:                       # one row at the full context, the others shorter
        positions[1:] = min(ns.others_context, S) - 1
    row_req = torch.arange(B, dtype=torch.int32, device=DEV)
    out = torch.empty(B, nq * d, dtype=torch.bfloat16, device=DEV)
    kind = {"full": ops.MASK_FULL, "chunk": ops.MASK_CHUNK, "window": ops.MASK_WINDOW}[ns.mask]
    keys = int((positions.long() + 1).sum())
    sinks = torch.zeros(nq, device=DEV) if ns.sinks else None
    fn = lambda: ops.attention_decode(q, kv, table, row_req, positions, out, rows=None, num_rows=B, nq=nq, nkv=nkv, d=d,
                                      page_size=ps, mask_kind=kind, mask_span=ns.span, scale=1 / math.sqrt(d),
                                      max_context=S, max_keys=keys, softcap=ns.softcap, sinks=sinks)
    ms = _time(fn, ns.iters)
    nbytes = keys * nkv * d * 2 * 2
    print(f"attention_decode batch={B} context={S}{'/' + str(ns.others_context) if ns.others_context else ''} heads={nq}/{nkv} d={d} "
          f"cap={ns.softcap} sinks={ns.sinks}: {ms * 1e3:.1f} us, {nbytes / ms / 1e6:.0f} GB/s")


def attention_prefill(ns) -> None:
    T, nq, nkv, d, ps = ns.tokens, ns.heads, ns.kv_heads, ns.head_dim, ns.page_size
    start = ns.start
    kv, table = _cache(1, start + T, nkv, d, ps)
    q = torch.randn(T, nq, d, device=DEV).to(torch.bfloat16)
    rows = 64 if ns.warp_mma else ops.TC_PREFILL_TILE
    tiles = torch.tensor([[t0, min(rows, T - t0), start + t0, 0] for t0 in range(0, T, rows)], dtype=torch.int32, device=DEV)
    out = torch.empty(T, nq * d, dtype=torch.bfloat16, device=DEV)
    kind = {"full": ops.MASK_FULL, "chunk": ops.MASK_CHUNK, "window": ops.MASK_WINDOW}[ns.mask]
    kernel = ops.attention_prefill if ns.warp_mma else ops.attention_prefill_tc
    sinks = torch.zeros(nq, device=DEV) if ns.sinks else None
    fn = lambda: kernel(q, kv, table, tiles, out, nq=nq, nkv=nkv, d=d, page_size=ps, mask_kind=kind,
                        mask_span=ns.span, scale=1 / math.sqrt(d), softcap=ns.softcap, sinks=sinks)
    ms = _time(fn, ns.iters)
    pairs = sum(min(start + t + 1, (start + t) % ns.span + 1 if kind == ops.MASK_CHUNK else start + t + 1) for t in range(T))
    flops = 4 * nq * d * pairs
    print(f"attention_prefill ({'m16n8k16' if ns.warp_mma else 'tcgen05'}) tokens={T} start={start} heads={nq}/{nkv} d={d} cap={ns.softcap} sinks={ns.sinks}: {ms * 1e3:.1f} us, {flops / ms / 1e9:.0f} TFLOP/s")


def ssd(ns) -> None:
    """The state-space-duality recurrence and the gated group norm behind it for `batch` requests of `tokens` rows
    each: per row and head 4 states x vdim flops (decay and update of S, S^T C); decode streams the state once."""
    B, n, heads, N, P = ns.batch, ns.tokens, ns.heads, ns.states, ns.value_dim
    T, inner = B * n, heads * P
    xbc = 0.5 * torch.randn(T, inner + 2 * N, device=DEV)
    proj = torch.randn(T, 2 * inner + 2 * N + heads, device=DEV)         # [x B C | z | dt], as the mixer lays it out
    col_z, col_dt = inner + 2 * N, 2 * inner + 2 * N
    dt_bias, a_log, dsk = torch.zeros(heads, device=DEV), torch.zeros(heads, device=DEV), torch.ones(heads, device=DEV)
    w = torch.ones(inner, device=DEV)
    per_request = heads * N * P
    copies = max(1, (300 << 20) // (B * per_request * 4) + 1) if n == 1 else 1
    state = torch.zeros(copies * B, per_request, device=DEV)
    offs = torch.arange(0, T + 1, n, dtype=torch.int32, device=DEV)
    slot_sets = [torch.arange(c * B, (c + 1) * B, dtype=torch.int32, device=DEV) for c in range(copies)]
    it = {"i": 0}

    def fn():
        slots = slot_sets[it["i"] % copies]
        it["i"] += 1
        y = ops.ssd_scan(xbc, proj, col_x=0, col_b=inner, col_c=inner + N, col_dt=col_dt, dt_bias=dt_bias, a_log=a_log,
                         dskip=dsk, row_offsets=offs, state_slots=slots, state=state, heads=heads, groups=1, states=N, vdim=P)
        ops.gated_group_norm(y, proj, col_z, w, 1e-5, 1, torch.bfloat16)
    ms = _time(fn, max(ns.iters, copies))
    print(f"ssd batch={B} tokens={n} heads={heads} states={N} vdim={P}: {ms * 1e3:.1f} us, state {2 * B * per_request * 4 / ms / 1e6:.0f} GB/s "
          f"(read and written once), {4.0 * T * per_request / ms / 1e9:.2f} TFLOP/s float32")


def lightning(ns) -> None:
    """Linear attention with a constant decay and the norm and gate behind it for `batch` requests of `tokens` rows each:
    per row and head 4 d dv flops (update of S, S^T q: what the recurrence asks for, whatever form runs it); decode streams
    the state once."""
    from sharpinference_b200.parts.lightning import LightningPlanner, lightning_columns
    B, n, heads, d, dv = ns.batch, ns.tokens, ns.heads, ns.key_dim, ns.value_dim
    cq, ck, cv, cg, width = lightning_columns(heads, d, dv)
    T = B * n
    proj = torch.randn(T, width, device=DEV)
    powers = ops.decay_powers([1.0 - 2.0 ** (-4 - i % 8) for i in range(heads)]).to(DEV)
    w = torch.ones(heads * dv, device=DEV)
    per_request = heads * d * dv
    copies = max(1, (300 << 20) // (B * per_request * 4) + 1) if n == 1 else 1
    state = torch.zeros(copies * B, per_request, device=DEV)
    offs = torch.arange(0, T + 1, n, dtype=torch.int32, device=DEV)
    slot_sets = [torch.arange(c * B, (c + 1) * B, dtype=torch.int32, device=DEV) for c in range(copies)]
    planner = LightningPlanner()
    if ns.walk:
        planner.WALK_ROWS_UP_TO = 1 << 30
    plan = planner.plan([0] * B, [n] * B)
    dev = {k: (torch.from_numpy(v).to(DEV) if v.size else None) for k, v in plan.arrays.items()}
    out = torch.empty(T, heads * dv, dtype=torch.bfloat16, device=DEV)
    it = {"i": 0}

    def fn():
        slots = slot_sets[it["i"] % copies]
        it["i"] += 1
        y = ops.lightning(proj, col_q=cq, col_k=ck, col_v=cv, powers=powers, row_offsets=offs, state_slots=slots, state=state,
                          heads=heads, d=d, dv=dv, num_requests=B, walk_requests=dev["walk"], num_walk=plan.values["num_walk"],
                          chunks=dev["chunks"], spans=dev["spans"], fast_activations=True)
        ops.norm_sigmoid_gate(y, proj[:, cg: cg + heads * dv], w, 1e-6, out)
    ms = _time(fn, max(ns.iters, copies))
    print(f"lightning batch={B} tokens={n} heads={heads} d={d} dv={dv}{' walked' if ns.walk else ''}: {ms * 1e3:.1f} us, state "
          f"{2 * B * per_request * 4 / ms / 1e6:.0f} GB/s (read and written once), {4.0 * T * per_request / ms / 1e9:.2f} TFLOP/s float32")


def delta(ns) -> None:
    """The gated delta rule with a decay per key channel and the norm and gate behind it for `batch` requests of `tokens` rows
    each: per row and head 7 d dv flops (decay, S^T k, update, S^T q: what the recurrence asks for, whatever form runs it);
    decode streams the state once."""
    from sharpinference_b200.parts.delta import DeltaPlanner
    B, n, heads, d, dv = ns.batch, ns.tokens, ns.heads, ns.key_dim, ns.value_dim
    G = ns.kv_heads or heads
    T, C = B * n, 2 * G * d + heads * dv
    qkv = torch.randn(T, C, device=DEV)
    qk = qkv[:, : 2 * G * d].view(T, 2 * G, d)
    qk /= qk.norm(dim=-1, keepdim=True)
    beta = torch.rand(T, heads, device=DEV)
    z = torch.randn(T, heads * (d + dv), device=DEV)
    dt_bias, a_log, w = torch.randn(heads * d, device=DEV) - 3, torch.zeros(heads, device=DEV), torch.ones(dv, device=DEV)
    per_request = ops.delta_state_floats(heads, d, dv)
    copies = max(1, (300 << 20) // (B * per_request * 4) + 1) if n == 1 else 1
    state = torch.zeros(copies * B, per_request, device=DEV)
    offs = torch.arange(0, T + 1, n, dtype=torch.int32, device=DEV)
    slot_sets = [torch.arange(c * B, (c + 1) * B, dtype=torch.int32, device=DEV) for c in range(copies)]
    planner = DeltaPlanner(4, True)
    if ns.walk:
        planner.WALK_ROWS_UP_TO = 1 << 30
    if ns.chunk:
        planner.WALK_ROWS_UP_TO = 0
    plan = planner.plan([0] * B, [n] * B)
    dev = {k: (torch.from_numpy(v).to(DEV) if v.size else None) for k, v in plan.arrays.items()}
    it = {"i": 0}

    def fn():
        slots = slot_sets[it["i"] % copies]
        it["i"] += 1
        y = ops.delta_rule(qkv, beta, z[:, : heads * d], dt_bias=dt_bias, a_log=a_log, row_offsets=offs, state_slots=slots, state=state,
                           kv_heads=G, heads=heads, d=d, dv=dv, num_requests=B, walk_requests=dev["walk"],
                           num_walk=plan.values["num_walk"], chunks=dev["chunks"], spans=dev["spans"], max_rows=n, split=not ns.exact)
        ops.head_norm_gate(y, z[:, heads * d:], w, 1e-6, heads, torch.bfloat16)
    ms = _time(fn, max(ns.iters, copies))
    print(f"delta batch={B} tokens={n} heads={heads}/{G} d={d} dv={dv}{' walked' if ns.walk else ''}: {ms * 1e3:.1f} us, state "
          f"{2 * B * per_request * 4 / ms / 1e6:.0f} GB/s (read and written once), {7.0 * T * heads * d * dv / ms / 1e9:.2f} TFLOP/s float32")


def delta_prep(ns) -> None:
    """Convolution, silu, unit norms, steps and low-rank columns behind the delta rule's fused projection."""
    from sharpinference_b200.parts.delta import DeltaPlanner, delta_columns
    B, n, heads, d, dv, low = ns.batch, ns.tokens, ns.heads, ns.key_dim, ns.value_dim, 2 * ns.key_dim
    G = ns.kv_heads or heads
    C, _, width = delta_columns(G, heads, d, dv, low)
    T = B * n
    copies = max(2, (300 << 20) // (T * width * 4) + 1) if T > 64 else 2
    projs = [torch.randn(T, width, device=DEV) for _ in range(copies)]
    conv, state = torch.randn(4, C, device=DEV), torch.zeros(B, 3 * C, device=DEV)
    offs = torch.arange(0, T + 1, n, dtype=torch.int32, device=DEV)
    slots = torch.arange(B, dtype=torch.int32, device=DEV)
    arr = DeltaPlanner(4, True).plan([0] * B, [n] * B).arrays["tiles"]
    tiles = torch.from_numpy(arr).to(DEV) if arr.size else None
    it = {"i": 0}

    def fn():
        ops.delta_prep(projs[it["i"] % copies], conv_weight=conv, conv_state=state, row_offsets=offs, state_slots=slots, tiles=tiles,
                       kv_heads=G, heads=heads, d=d, dv=dv, low=low, act_dtype=torch.bfloat16)
        it["i"] += 1
    ms = _time(fn, max(ns.iters, copies))
    print(f"delta_prep batch={B} tokens={n} heads={heads}/{G} d={d} dv={dv}: {ms * 1e3:.1f} us, "
          f"{T * (C * 8 + low * 6 + heads * 8) / ms / 1e6:.0f} GB/s")


def sandwich(ns) -> None:
    """A normed update and the norm behind it, the same with the bare stream, the side gate, the element gate of latent
    attention and the router with sigmoid scores in groups."""
    T, H, N, k = ns.tokens, ns.hidden, ns.experts, ns.top
    copies = max(2, (300 << 20) // (T * H * 8) + 1)
    xs = [(torch.randn(T, H, device=DEV), torch.randn(T, H, device=DEV)) for _ in range(copies)]
    w1, w2 = torch.ones(H, device=DEV), torch.ones(H, device=DEV)
    it = {"i": 0}

    def timed(name, fn, nbytes):
        def call():
            fn(it["i"] % copies)
            it["i"] += 1
        ms = _time(call, max(ns.iters, copies))
        print(f"{name} tokens={T} hidden={H}: {ms * 1e3:.1f} us, {nbytes / ms / 1e6:.0f} GB/s")
    timed("add_normed", lambda i: ops.add_normed(xs[i][0], xs[i][1], w1, w2, 1e-6, torch.bfloat16), T * H * 14)
    timed("add_normed, bare stream", lambda i: ops.add_normed(xs[i][0], xs[i][1], w1, None, 1e-6, torch.bfloat16), T * H * 14)
    timed("add_rmsnorm", lambda i: ops.add_rmsnorm(xs[i][0], xs[i][1], w1, 1e-6, torch.bfloat16), T * H * 14)
    n = max(8, H // 16)
    gate, table = torch.randn(T, n, device=DEV), torch.randn(32768, 10 * n, device=DEV).to(torch.bfloat16)
    ids = torch.randint(0, 32768, (T,), device=DEV, dtype=torch.int32)
    timed(f"side_gate n={n}", lambda i: ops.side_gate(gate, ids, table, 3 * n, n, torch.bfloat16), T * n * 8)
    heads = max(1, H // 128)
    v, wide = torch.randn(heads * T, 128, device=DEV), torch.randn(T, 2 * H, device=DEV)
    timed("head_minor, element gate", lambda i: ops.head_minor(v, heads=heads, out_dtype=torch.bfloat16, gate=wide[:, H:]), T * H * 10)
    timed("head_minor, head gate", lambda i: ops.head_minor(v, heads=heads, out_dtype=torch.bfloat16, gate=wide[:, :heads]), T * H * 6)
    wr, corr = torch.randn(N, H, device=DEV) * 0.05, torch.randn(N, device=DEV) * 0.1
    timed(f"router_groups, sigmoid, {N} experts", lambda i: ops.router_groups(
        xs[i][0], wr, k, correction=corr, renormalize=False, n_groups=4, keep=2, scoring="sigmoid", group_top=2), T * H * 4 + N * H * 4)
    timed(f"router_topk, {N} experts", lambda i: ops.router_topk(xs[i][0], wr, k, correction=corr), T * H * 4 + N * H * 4)


def qkv_conv(ns) -> None:
    """Short convolution of q, k and v, rotation, q store and cache write for `batch` requests of `tokens` rows each."""
    from sharpinference_b200.parts.position import leading_rotary_inv_freq_parts
    B, n, nq, nkv, d, ps = ns.batch, ns.tokens, ns.heads, ns.kv_heads, ns.head_dim, ns.page_size
    T, C = B * n, (nq + 2 * nkv) * d
    width = (C + nq + 7) // 8 * 8
    copies = max(2, (300 << 20) // (T * width * 4) + 1) if T > 64 else 2
    projs = [torch.randn(T, width, device=DEV) for _ in range(copies)]
    pages = (n + ps - 1) // ps
    kv = torch.zeros(B * pages, 2, nkv, ps, d, dtype=torch.bfloat16, device=DEV)
    table = torch.arange(B * pages, dtype=torch.int32, device=DEV).view(B, pages)
    positions = torch.arange(n, dtype=torch.int32, device=DEV).repeat(B)
    row_req = torch.arange(B, dtype=torch.int32, device=DEV).repeat_interleave(n)
    offs = torch.arange(0, T + 1, n, dtype=torch.int32, device=DEV)
    slots = torch.arange(B, dtype=torch.int32, device=DEV)
    state = torch.zeros(B, (ns.taps - 1) * C, device=DEV)
    w = torch.randn(ns.taps, C, device=DEV)
    inv, low = (t.to(DEV) for t in leading_rotary_inv_freq_parts(ns.rot, 500000.0))
    q = torch.empty(T, nq, d, dtype=torch.bfloat16, device=DEV)
    it = {"i": 0}

    def fn():
        ops.qkv_conv(projs[it["i"] % copies][:, :C], q, kv, weight=w, state=state, positions=positions, row_req=row_req, row_offsets=offs,
                     state_slots=slots, block_table=table, nq=nq, nkv=nkv, D=d, key_dim=d, value_dim=d, page_size=ps, inv_freq=inv,
                     inv_freq_low=low, rot_dims=ns.rot)
        it["i"] += 1
    ms = _time(fn, max(ns.iters, copies))
    print(f"qkv_conv batch={B} tokens={n} heads={nq}/{nkv} d={d} taps={ns.taps}: {ms * 1e3:.1f} us, {T * C * 6 / ms / 1e6:.0f} GB/s")


def softmax_mixture(ns) -> None:
    """The router of a softmax mixture in groups with a gate row, the sum of a row's pairs with identity experts, a gated
    shared expert and an add-in, and the head gate."""
    T, H, N, k = ns.tokens, ns.hidden, ns.experts, ns.top
    copies = max(2, (300 << 20) // (T * H * 4) + 1)
    hs = [torch.randn(T, H, device=DEV) for _ in range(copies)]
    wr, corr, gw = torch.randn(N, H, device=DEV) * 0.05, torch.randn(N, device=DEV) * 0.1, torch.randn(H, device=DEV)
    it = {"i": 0}

    def router():
        ops.router_groups(hs[it["i"] % copies], wr, k, correction=corr, scale=2.0, n_groups=2, keep=1, gate_weight=gw)
        it["i"] += 1
    ms = _time(router, max(ns.iters, copies))
    print(f"router_groups tokens={T} hidden={H} experts={N} top={k}: {ms * 1e3:.1f} us, {(T * H * 4 + N * H * 4) / ms / 1e6:.0f} GB/s")
    expert, weight, gate, _ = ops.router_groups(hs[0], wr, k, n_groups=2, keep=1, gate_weight=gw)
    ys = [torch.randn(T * k, H, device=DEV) for _ in range(2)]
    shared, add = torch.randn(T, H, device=DEV), torch.randn(T, H, device=DEV)

    def combine():
        ops.moe_combine_full(ys[it["i"] % 2], expert, weight, hs[it["i"] % copies], N - 2, shared=shared, gate=gate, add=add, out=add)
        it["i"] += 1
    ms = _time(combine, max(ns.iters, copies))
    print(f"moe_combine_full tokens={T} top={k}: {ms * 1e3:.1f} us, {(T * k + 4 * T) * H * 4 / ms / 1e6:.0f} GB/s")
    heads, D = max(1, H // 128), 128
    o, g = torch.randn(T, heads, D, device=DEV).to(torch.bfloat16), torch.randn(T, heads, device=DEV)
    out = torch.empty(T, heads * D, dtype=torch.bfloat16, device=DEV)
    ms = _time(lambda: ops.gate_heads(o, g, out, heads=heads, D=D, dv=D), max(ns.iters, 8))
    print(f"gate_heads tokens={T} heads={heads}: {ms * 1e3:.1f} us, {T * heads * D * 4 / ms / 1e6:.0f} GB/s")
    gu = [torch.randn(T, 8 * H, device=DEV) for _ in range(2)]
    bias, wide = torch.randn(8 * H, device=DEV), torch.empty(T, 4 * H + 8, dtype=torch.bfloat16, device=DEV)

    def gated():
        ops.gated_cols(gu[it["i"] % 2], wide, bias=bias, ones=3)
        it["i"] += 1
    ms = _time(gated, max(ns.iters, 8))
    print(f"gated_cols tokens={T} ff={4 * H}: {ms * 1e3:.1f} us, {T * 4 * H * 10 / ms / 1e6:.0f} GB/s")


def _keys_cache(batch: int, context: int, nkv: int, d: int, ps: int):
    blocks = (context + ps - 1) // ps
    pages = batch * blocks
    kv = torch.empty(pages, 1, nkv, ps, d, dtype=torch.bfloat16, device=DEV).normal_(0, 1)
    table = torch.randperm(pages, device=DEV).to(torch.int32).view(batch, blocks).contiguous()
    return kv, table


def _keys_mask(ns):
    kind = {"full": ops.MASK_FULL, "window": ops.MASK_WINDOW}[ns.mask]
    bias = 0.1 * torch.randn(ns.bias_far + 1, ns.heads, device=DEV) if ns.bias_far else None
    return kind, bias


def _visible(pos: int, kind: int, span: int, keep: int) -> int:
    return pos + 1 if kind == ops.MASK_FULL or pos < span else span + min(keep, pos + 1 - span)


def attention_keys_decode(ns) -> None:
    """Single query rows over keys-only pages (a key's leading elements are its value): the keys stream once."""
    B, S, nq, nkv, d, dv, ps = ns.batch, ns.context, ns.heads, ns.kv_heads, ns.head_dim, ns.value_dim or ns.head_dim, ns.page_size
    kv, table = _keys_cache(B, S, nkv, d, ps)
    q = torch.randn(B, nq, d, device=DEV).to(torch.bfloat16)
    positions = torch.full((B,), S - 1, dtype=torch.int32, device=DEV)
    row_req = torch.arange(B, dtype=torch.int32, device=DEV)
    out = torch.empty(B, nq * dv, dtype=torch.bfloat16, device=DEV)
    kind, bias = _keys_mask(ns)
    fn = lambda: ops.attention_keys_decode(q, kv, table, row_req, positions, out, rows=None, num_rows=B, nq=nq, nkv=nkv, d=d,
                                           dv=dv, page_size=ps, mask_kind=kind, mask_span=ns.span, scale=1 / math.sqrt(d),
                                           max_context=S, keep_first=ns.keep_first, dist_bias=bias)
    ms = _time(fn, ns.iters)
    nbytes = B * _visible(S - 1, kind, ns.span, ns.keep_first) * nkv * d * 2
    print(f"attention_keys_decode batch={B} context={S} heads={nq}/{nkv} d={d} dv={dv} mask={ns.mask}: {ms * 1e3:.1f} us, "
          f"{nbytes / ms / 1e6:.0f} GB/s of visible keys")


def attention_keys_prefill(ns) -> None:
    """One prompt of `tokens` rows over keys-only pages in tiles of 64 rows: 2 (d + dv) flops a (query, visible key)."""
    T, nq, nkv, d, dv, ps = ns.tokens, ns.heads, ns.kv_heads, ns.head_dim, ns.value_dim or ns.head_dim, ns.page_size
    kv, table = _keys_cache(1, T, nkv, d, ps)
    q = torch.randn(T, nq, d, device=DEV).to(torch.bfloat16)
    tiles = torch.tensor([[t0, min(64, T - t0), t0, 0] for t0 in range(0, T, 64)], dtype=torch.int32, device=DEV)
    out = torch.empty(T, nq * dv, dtype=torch.bfloat16, device=DEV)
    kind, bias = _keys_mask(ns)
    fn = lambda: ops.attention_keys_prefill(q, kv, table, tiles, out, nq=nq, nkv=nkv, d=d, dv=dv, page_size=ps, mask_kind=kind,
                                            mask_span=ns.span, scale=1 / math.sqrt(d), keep_first=ns.keep_first, dist_bias=bias)
    ms = _time(fn, ns.iters)
    pairs = sum(_visible(t, kind, ns.span, ns.keep_first) for t in range(T))
    print(f"attention_keys_prefill tokens={T} heads={nq}/{nkv} d={d} dv={dv} mask={ns.mask}: {ms * 1e3:.1f} us, "
          f"{2.0 * (d + dv) * nq * pairs / ms / 1e9:.0f} TFLOP/s")


def main(argv=None) -> int:
    ap = argparse.ArgumentParser(description=__doc__, formatter_class=argparse.RawDescriptionHelpFormatter)
    sub = ap.add_subparsers(dest="kernel", required=True)
    p = sub.add_parser("tc_gemm")
    p.add_argument("--mode", choices=["gate_up", "down"], default="gate_up")
    p.add_argument("--rows", type=int, default=2048)
    p.add_argument("--experts", type=int, default=16)
    p.add_argument("--active", type=int, default=0, help="experts that receive rows (0 = all)")
    p.add_argument("--hidden", type=int, default=5120)
    p.add_argument("--inter", type=int, default=8192)
    p.add_argument("--row-tile", type=int, default=None)
    p.add_argument("--k-split", type=int, default=None)
    p.add_argument("--max-ctas", type=int, default=0, help="persistent kernel: at most this many SMs (0 = all)")
    p.add_argument("--beside", default="", help="M,N,K of a library product launched on a second stream beside each call")
    p.add_argument("--beside-count", type=int, default=1)
    p.add_argument("--skew", type=float, default=0.0,
                   help="0: equal groups; else expert e gets rows in proportion to (1 - skew)^e")
    p.set_defaults(fn=tc_gemm)
    p = sub.add_parser("dense")
    p.add_argument("--rows", type=int, default=8)
    p.add_argument("--n", type=int, default=7168)
    p.add_argument("--k", type=int, default=5120)
    p.add_argument("--swiglu", action="store_true", help="SwiGLU after the product (rows: in its epilogue; library: a second kernel)")
    p.add_argument("--impl", choices=["grouped", "rows", "library"], default="grouped")
    p.set_defaults(fn=dense)
    p = sub.add_parser("elementwise")
    p.add_argument("--op", choices=["add_rmsnorm", "add_rmsnorm_pair", "swiglu", "gather", "qkv_post", "add_layernorm", "add_dyt", "qkv_post_wide"], default="add_rmsnorm")
    p.add_argument("--tokens", type=int, default=2048)
    p.add_argument("--hidden", type=int, default=5120)
    p.add_argument("--inter", type=int, default=8192)
    p.add_argument("--heads", type=int, default=40)
    p.add_argument("--kv-heads", type=int, default=8)
    p.add_argument("--head-dim", type=int, default=128)
    p.add_argument("--page-size", type=int, default=64)
    p.add_argument("--fp32-copy", action="store_true", help="add_rmsnorm: also write the unrounded copy (as before a router)")
    p.set_defaults(fn=elementwise)
    p = sub.add_parser("router")
    p.add_argument("--tokens", type=int, default=2048)
    p.add_argument("--hidden", type=int, default=5120)
    p.add_argument("--experts", type=int, default=16)
    p.set_defaults(fn=router)
    p = sub.add_parser("mlstm")
    p.add_argument("--batch", type=int, default=64)
    p.add_argument("--tokens", type=int, default=1)
    p.add_argument("--heads", type=int, default=8)
    p.add_argument("--key-dim", type=int, default=128)
    p.add_argument("--value-dim", type=int, default=256)
    p.set_defaults(fn=mlstm)
    p = sub.add_parser("wkv")
    p.add_argument("--batch", type=int, default=64)
    p.add_argument("--tokens", type=int, default=1)
    p.add_argument("--heads", type=int, default=32)
    p.add_argument("--head-dim", type=int, default=64)
    p.set_defaults(fn=wkv)
    p = sub.add_parser("scan")
    p.add_argument("--batch", type=int, default=64)
    p.add_argument("--tokens", type=int, default=1)
    p.add_argument("--channels", type=int, default=4096)
    p.add_argument("--states", type=int, default=16)
    p.add_argument("--dt-rank", type=int, default=128)
    p.add_argument("--taps", type=int, default=4)
    p.set_defaults(fn=scan)
    p = sub.add_parser("streams")
    p.add_argument("--tokens", type=int, default=2048)
    p.add_argument("--hidden", type=int, default=2048)
    p.add_argument("--streams", type=int, default=4)
    p.add_argument("--groups", type=int, default=4)
    p.set_defaults(fn=streams)
    for name, fn in (("router_topk", router_topk), ("mixture_glue", mixture_glue)):
        p = sub.add_parser(name)
        p.add_argument("--tokens", type=int, default=2048)
        p.add_argument("--hidden", type=int, default=2048)
        p.add_argument("--inter", type=int, default=1024)
        p.add_argument("--experts", type=int, default=16)
        p.add_argument("--top", type=int, default=2)
        p.set_defaults(fn=fn)
    for name, fn in (("attention_decode", attention_decode), ("attention_prefill", attention_prefill)):
        p = sub.add_parser(name)
        p.add_argument("--batch", type=int, default=8)
        p.add_argument("--context", type=int, default=8192)
        p.add_argument("--others-context", type=int, default=0,
                       help="attention_decode: rows after the first have this many keys (a batch of unequal lengths)")
        p.add_argument("--tokens", type=int, default=2048)
        p.add_argument("--start", type=int, default=0)
        p.add_argument("--heads", type=int, default=40)
        p.add_argument("--kv-heads", type=int, default=8)
        p.add_argument("--head-dim", type=int, default=128)
        p.add_argument("--page-size", type=int, default=64)
        p.add_argument("--mask", choices=["full", "chunk", "window"], default="full")
        p.add_argument("--span", type=int, default=8192)
        p.add_argument("--warp-mma", action="store_true", help="attention_prefill: the m16n8k16 kernel with 64-row tiles")
        p.add_argument("--softcap", type=float, default=0.0, help="scores become softcap * tanh(score / softcap) (0: no cap)")
        p.add_argument("--sinks", action="store_true", help="a sink per head in the softmax's denominator")
        p.set_defaults(fn=fn)
    p = sub.add_parser("ssd")
    p.add_argument("--batch", type=int, default=64)
    p.add_argument("--tokens", type=int, default=1)
    p.add_argument("--heads", type=int, default=64)
    p.add_argument("--states", type=int, default=128)
    p.add_argument("--value-dim", type=int, default=64)
    p.set_defaults(fn=ssd)
    for name, fn in (("attention_keys_decode", attention_keys_decode), ("attention_keys_prefill", attention_keys_prefill)):
        p = sub.add_parser(name)
        p.add_argument("--batch", type=int, default=8)
        p.add_argument("--context", type=int, default=8192)
        p.add_argument("--tokens", type=int, default=2048)
        p.add_argument("--heads", type=int, default=16)
        p.add_argument("--kv-heads", type=int, default=4)
        p.add_argument("--head-dim", type=int, default=128)
        p.add_argument("--value-dim", type=int, default=0, help="a value's size (the head size when 0)")
        p.add_argument("--page-size", type=int, default=64)
        p.add_argument("--mask", choices=["full", "window"], default="full")
        p.add_argument("--span", type=int, default=1024)
        p.add_argument("--keep-first", type=int, default=0)
        p.add_argument("--bias-far", type=int, default=0, help="rows of a distance-bias table minus one (0: no bias)")
        p.set_defaults(fn=fn)
    p = sub.add_parser("lightning")
    p.add_argument("--batch", type=int, default=64)
    p.add_argument("--tokens", type=int, default=1)
    p.add_argument("--heads", type=int, default=16)
    p.add_argument("--key-dim", type=int, default=128)
    p.add_argument("--value-dim", type=int, default=128)
    p.add_argument("--walk", action="store_true", help="walk the rows one by one whatever their number")
    p.set_defaults(fn=lightning)
    for name, fn in (("delta", delta), ("delta_prep", delta_prep)):
        p = sub.add_parser(name)
        p.add_argument("--batch", type=int, default=64 if name == "delta" else 1)
        p.add_argument("--tokens", type=int, default=1 if name == "delta" else 2048)
        p.add_argument("--heads", type=int, default=16)
        p.add_argument("--kv-heads", type=int, default=0, help="heads of q and k (0: as many as heads)")
        p.add_argument("--key-dim", type=int, default=128)
        p.add_argument("--value-dim", type=int, default=128)
        p.add_argument("--walk", action="store_true", help="walk the rows one by one whatever their number")
        p.add_argument("--exact", action="store_true", help="chunks in float32 FMAs")
        p.add_argument("--chunk", action="store_true", help="cut into chunks whatever the number of rows")
        p.set_defaults(fn=fn)
    p = sub.add_parser("sandwich")
    p.add_argument("--tokens", type=int, default=2048)
    p.add_argument("--hidden", type=int, default=2048)
    p.add_argument("--experts", type=int, default=16)
    p.add_argument("--top", type=int, default=2)
    p.set_defaults(fn=sandwich)
    p = sub.add_parser("qkv_conv")
    p.add_argument("--batch", type=int, default=1)
    p.add_argument("--tokens", type=int, default=2048)
    p.add_argument("--heads", type=int, default=16)
    p.add_argument("--kv-heads", type=int, default=4)
    p.add_argument("--head-dim", type=int, default=128)
    p.add_argument("--page-size", type=int, default=64)
    p.add_argument("--taps", type=int, default=4)
    p.add_argument("--rot", type=int, default=64)
    p.set_defaults(fn=qkv_conv)
    p = sub.add_parser("softmax_mixture")
    p.add_argument("--tokens", type=int, default=2048)
    p.add_argument("--hidden", type=int, default=2048)
    p.add_argument("--experts", type=int, default=18)
    p.add_argument("--top", type=int, default=2)
    p.set_defaults(fn=softmax_mixture)
    for sp in sub.choices.values():
        sp.add_argument("--iters", type=int, default=10)
        sp.add_argument("--graph", action="store_true", help="time replays of a CUDA graph of the calls")
    ns = ap.parse_args(argv)
    global USE_GRAPH
    USE_GRAPH = ns.graph
    if not torch.cuda.is_available():
        print("bench_kernels.py needs a CUDA device", file=sys.stderr)
        return 2
    ns.fn(ns)
    return 0


if __name__ == "__main__":
    sys.exit(main())
