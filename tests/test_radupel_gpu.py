"""Radupel on the GPU: each new kernel against the plain statement of its mechanism, each layer alone through a one-layer
model, and whole models through the engine (step function, cache manager, scheduler) under every way of cutting the work,
in 32-bit and in bfloat16."""
import copy
import json
import os

import pytest
import torch

import plain_radupel as plain
import traces
from radupel_models import CASES, write

pytestmark = pytest.mark.gpu
DEV = "cuda:0"
F64 = torch.float64

# Relative to the largest |logit| of a request.
TOL = {"float32": 5e-5, "bfloat16": 4e-2}
# A differing expert choice must be a near-tie of the choice scores (softmax scores plus corrections).
MARGIN = 6e-2
LENGTHS = {"A": [1, 9, 40, 83, 150, 2], "B": [150, 5, 67, 200, 31], "C": [3, 70, 140, 45, 210, 64, 65],
           "D": [1, 2, 30, 5, 100], "E": [140, 66, 3, 129, 230]}


def requests_for(name):
    vocab = CASES[name][0]["vocab"]
    return {f"r{i}": traces.random_tokens(vocab, n, seed=43 * i + n) for i, n in enumerate(LENGTHS[name])}


@pytest.fixture(scope="module")
def folders(tmp_path_factory):
    return {name: write(name, str(tmp_path_factory.mktemp(f"radupel_{name}"))) for name in CASES}


@pytest.fixture(scope="module")
def expected(folders):
    out = {}
    for name, folder in folders.items():
        cfg, w = plain.load_folder(folder)
        out[name] = {rid: plain.forward(cfg, w, toks) for rid, toks in requests_for(name).items()}
    return out


def engine_for(folder, dtype, max_tokens, max_batch=4, page_size=None):
    from sharpinference_b200 import Engine, EngineOptions
    opts = EngineOptions()
    if page_size:
        opts.page_size = page_size
    opts.max_cache_tokens = max(max_tokens, opts.page_size)
    opts.max_batch = max_batch
    return Engine(folder, dtype=dtype, device=DEV, options=opts)


def assert_near_ties(score, forced, router, rid, margin):
    """Every forced set of experts is the router's own up to ``MARGIN``: the groups it lies in are (nearly) the best, and its
    experts are (nearly) the largest within these groups."""
    groups = router.get("groups") or {"count": 1, "keep": 1}
    n, N = score.shape
    per = N // groups["count"]
    best = score.view(n, groups["count"], per).max(-1).values
    kth_group = best.topk(groups["keep"], dim=-1).values[:, -1]
    assert float((kth_group - best.gather(1, forced // per).min(-1).values).max()) < margin, f"request {rid}: a group beyond a near-tie"
    mine = torch.zeros(n, groups["count"], dtype=torch.bool)
    mine[torch.arange(n).view(n, 1), forced // per] = True
    own = score.masked_fill(~mine.repeat_interleave(per, dim=1), -1e9)
    kth = own.topk(forced.shape[1], dim=-1).values[:, -1]
    assert float((kth - score.gather(1, forced).min(-1).values).max()) < margin, f"request {rid}: an expert beyond a near-tie"


def reference_for(folder, reqs, routing, fallback, dtype, slack=None, margin=MARGIN):
    """float32 runs are held to the plain logits as they are; bfloat16 runs to the plain logits under the engine's own expert
    choices, each differing choice having to be a near-tie.  ``slack`` receives, per request, what rounding the operands of
    the matrix products alone does to every position's logits in the plain model: where that is more than the tolerance a
    bfloat16 run is held to three times it."""
    if dtype == "float32":
        return fallback
    cfg, w = plain.load_folder(folder)
    routers = [cfg["layers"][i]["mlp"]["router"] for i, _ in plain.layer_order(cfg)
               if cfg["layers"][i]["mlp"] and cfg["layers"][i]["mlp"]["kind"] == "moe"]
    ref = {}
    for rid, toks in reqs.items():
        choices = [torch.tensor(per_layer, dtype=torch.long).view(len(toks), -1) for per_layer in routing[rid]]
        seen = []
        logits = plain.forward(cfg, w, toks, choices=choices, choices_out=seen)
        assert len(seen) == len(routers)
        for (score, _), forced, router in zip(seen, choices, routers):
            assert_near_ties(score, forced, router, rid, margin)
        ref[rid] = logits
        if slack is not None:
            rounded = plain.forward(cfg, w, toks, choices=choices, round_to=torch.bfloat16)
            slack[rid] = (rounded - logits).abs().max(dim=-1).values / float(logits.abs().max())
    return ref


def worst_excess(got, ref, tol, slack):
    """The largest error over the wanted rows as a multiple of what the row is allowed."""
    worst, where = 0.0, None
    for (rid, pos), row in got.items():
        err = float((row.double() - ref[rid][pos]).abs().max()) / float(ref[rid].abs().max())
        allowed = max(tol, 3.0 * float(slack[rid][pos])) if slack else tol
        if not err / allowed <= worst:
            worst, where = err / allowed, (rid, pos, err)
    return worst, where


def run_and_compare(folder, name, dtype, steps, expected, page_size=None, max_batch=4):
    reqs = requests_for(name)
    eng = engine_for(folder, dtype, traces.max_tokens(steps, page_size or 64), max_batch=max_batch, page_size=page_size)
    routing = {} if dtype == "bfloat16" else None
    got = traces.replay(eng, steps, routing)
    eng.runner.flush_status()
    eng.cache.check_invariants()
    assert not eng.cache.requests and all(g.pages.held_count == 0 for g in eng.cache.groups)
    wanted = sum(len(e["want"]) for st in steps for e in st["entries"])
    assert len({rid for rid, _ in got}) == len(reqs) and len(got) == wanted
    slack = {} if dtype == "bfloat16" else None
    ref = reference_for(folder, reqs, routing, expected[name], dtype, slack)
    excess, where = worst_excess(got, ref, TOL[dtype], slack)
    assert excess < 1.0, f"{name} {dtype}: {excess} times the allowed error at {where}"
    return eng


f32 = lambda t: t.float().to(DEV).contiguous()
i32 = lambda v: torch.tensor(v, dtype=torch.int32, device=DEV)


def _rand(*shape, seed=0, scale=1.0):
    """Random float64 numbers that float32 holds exactly."""
    return (scale * torch.randn(*shape, generator=torch.Generator().manual_seed(seed), dtype=F64)).float().double()


def close(got, want, tol):
    err = float((got.double().cpu() - want).abs().max())
    assert err < tol * max(1.0, float(want.abs().max())), err


# ------------------------------------------------------------------------------------------
# kernels alone
# ------------------------------------------------------------------------------------------
@pytest.mark.parametrize("T,H", [(3, 1), (11, 52), (7, 257), (130, 1024), (200, 96), (5, 13000), (150, 9000)])
def test_two_norms_of_one_stream(T, H):
    from sharpinference_b200.kernels import ops
    x, delta, w1, w2 = 3 * _rand(T, H, seed=H), _rand(T, H, seed=H + 1), _rand(H, seed=H + 2), _rand(H, seed=H + 3)
    x = x.float().double()
    for d in (None, f32(delta)):
        xd = f32(x)
        a, b, b32 = ops.add_rmsnorm_pair(xd, d, f32(w1), f32(w2), 1e-5, torch.bfloat16, want_fp32=True)
        s = x + (0 if d is None else delta)
        close(b32, plain.rms(s, w2, 1e-5), 2e-6)
        assert torch.equal(b, b32.to(torch.bfloat16))
        close(a, plain.rms(s, w1, 1e-5), 5e-3)
        close(xd, s, 1e-6)
        one, _ = ops.add_rmsnorm(f32(x), d, f32(w1), 1e-5, torch.bfloat16)
        assert torch.equal(a, one)                                            # the bits of the norm by itself
    a, b, b32 = ops.add_rmsnorm_pair(f32(x), None, f32(w1), f32(w2), 1e-5, torch.float32, want_fp32=True)
    assert b32 is b
    close(a, plain.rms(x, w1, 1e-5), 2e-6)


@pytest.mark.parametrize("I,tail,ones,col", [(40, 8, 3, 16), (19, 5, 3, 8), (1, 7, 1, 0), (256, 0, 0, 24), (12, 4, 1, 3)])
@pytest.mark.parametrize("act,limit", [("silu", 0.0), ("gelu_tanh", 0.0), ("relu2", 0.0), ("silu", 0.9)])
def test_gated_activation_into_a_column_range(I, tail, ones, col, act, limit):
    from sharpinference_b200.kernels import ops
    T = 9
    gu, bias = 2 * _rand(T, 2 * I, seed=I), _rand(2 * I, seed=I + 1)
    wide = torch.full((T, col + I + tail + 5), 7.0, device=DEV)
    ops.gated_cols(f32(gu), wide[:, col: col + I + tail], bias=f32(bias), act=ops.ACTIVATIONS[act], limit=limit, ones=ones)
    z = gu.float().double() + bias
    g, u = z[:, :I], z[:, I:]
    if limit:
        g, u = g.clamp(max=limit), u.clamp(-limit, limit)
        y = g * torch.sigmoid(1.702 * g) * (u + 1)
    else:
        fn = {"silu": plain.silu, "relu2": lambda t: t.clamp(min=0) ** 2,
              "gelu_tanh": lambda t: torch.nn.functional.gelu(t, approximate="tanh")}[act]
        y = fn(g) * u
    want = torch.full(wide.shape, 7.0, dtype=F64)
    want[:, col: col + I] = y
    want[:, col + I: col + I + tail] = 0.0
    want[:, col + I: col + I + ones] = 1.0
    close(wide, want, 1e-5)
    out = torch.empty(T, I, dtype=torch.bfloat16, device=DEV)
    ops.gated_cols(f32(gu), out, act=ops.ACTIVATIONS[act], limit=limit)
    assert bool(torch.isfinite(out).all())


def test_head_gate_and_logit_cap():
    from sharpinference_b200.kernels import ops
    T, H, D, dv = 37, 3, 16, 10
    o, wide = _rand(T, H, D, seed=1), _rand(T, 20, seed=2, scale=2.0)
    g = f32(wide)[:, 5: 5 + H]
    out = torch.full((T, 50), 7.0, device=DEV)
    ops.gate_heads(f32(o), g, out[:, 8: 8 + H * dv], heads=H, D=D, dv=dv, scale=-1.5)
    want = torch.full((T, 50), 7.0, dtype=F64)
    want[:, 8: 8 + H * dv] = (o[..., :dv] * torch.sigmoid(wide[:, 5: 5 + H]).view(T, H, 1) * -1.5).reshape(T, -1)
    close(out, want, 1e-6)
    y = _rand(5, 33, seed=3, scale=20.0)
    got = ops.softcap_(f32(y), 7.5)
    close(got, 7.5 * torch.tanh(y.float().double() / 7.5), 1e-6)


@pytest.mark.parametrize("nq,nkv,dk,dv,taps,rot,layout,pad", [
    (4, 2, 16, 24, 4, 8, "halves", 8), (3, 3, 10, 7, 6, 6, "halves", 5), (2, 1, 128, 128, 3, 128, "halves", 4),
    (2, 2, 9, 11, 2, 2, "halves", 1), (1, 1, 12, 12, 1, 4, "interleaved", 0), (2, 1, 64, 64, 5, 16, "interleaved", 8),
    (2, 1, 144, 96, 4, 48, "halves", 8), (1, 1, 1, 2, 3, 0, "halves", 0)])
def test_convolution_rotation_and_cache_write(nq, nkv, dk, dv, taps, rot, layout, pad):
    """Two requests on two slots, in portions of one row, of fewer rows than the convolution keeps, and of more; the state
    left behind by a portion is what the next one starts from, and a third slot is untouched."""
    from sharpinference_b200.kernels import ops
    from sharpinference_b200.parts.position import leading_rotary_inv_freq_parts
    D = max(dk, dv)
    D = (D + 15) // 16 * 16 if D <= 128 else D + (D & 1)
    C = (nq + nkv) * dk + nkv * dv
    page, n = 8, 41
    w = _rand(C, taps, seed=C)
    us = [_rand(n, C, seed=1), _rand(n, C, seed=2)]
    slots = [2, 0]
    state = torch.full((3, max(taps - 1, 1) * C), 0.0, device=DEV)
    state[1] = 5.0
    kv = torch.full((14, 2, nkv, page, D), 7.0, device=DEV)
    table = i32([[3, 1, 12, 0, 7, 2], [5, 9, 11, 4, 13, 6]])
    inv, low = (t.to(DEV) for t in leading_rotary_inv_freq_parts(rot, 100.0)) if rot else (None, None)
    qs = [[], []]
    cuts = [[1, 2, 1, 1, 7, 3, 26], [5, 1, 20, 2, 1, 1, 11]]
    at = [0, 0]
    for m0, m1 in zip(*cuts):
        rows = torch.cat([us[0][at[0]: at[0] + m0], us[1][at[1]: at[1] + m1]])
        proj = torch.cat([rows, _rand(m0 + m1, pad, seed=9)], dim=1) if pad else rows
        pos = list(range(at[0], at[0] + m0)) + list(range(at[1], at[1] + m1))
        q = torch.full((m0 + m1, nq, D), 7.0, device=DEV)
        ops.qkv_conv(f32(proj)[:, :C], q, kv, weight=f32(w.T), state=state, positions=i32(pos), row_req=i32([0] * m0 + [1] * m1),
                     row_offsets=i32([0, m0, m0 + m1]), state_slots=i32(slots), block_table=table, nq=nq, nkv=nkv, D=D, key_dim=dk,
                     value_dim=dv, page_size=page, inv_freq=inv, inv_freq_low=low, rot_dims=rot,
                     pairing=ops.ROPE_HALVES if layout == "halves" else ops.ROPE_INTERLEAVED)
        qs[0].append(q[:m0].cpu())
        qs[1].append(q[m0:].cpu())
        at = [at[0] + m0, at[1] + m1]
    assert at == [n, n]

    def turn(v):
        if not rot:
            return v
        if layout == "halves":
            return plain.rotate_halves(v, rot, 100.0)
        order = [2 * i for i in range(rot // 2)] + [2 * i + 1 for i in range(rot // 2)]       # pairs side by side -> halves
        back = [order.index(i) for i in range(rot)]
        return torch.cat([plain.rotate_halves(v[..., order], rot, 100.0)[..., back], v[..., rot:]], dim=-1)
    for b in range(2):
        y = plain.causal_conv(us[b], w)
        q = turn(y[:, : nq * dk].reshape(n, nq, dk))
        k = turn(y[:, nq * dk: (nq + nkv) * dk].reshape(n, nkv, dk))
        v = y[:, (nq + nkv) * dk:].reshape(n, nkv, dv)
        got = torch.cat(qs[b])
        close(got[..., :dk], q, 1e-5)
        assert float(got[..., dk:].abs().sum()) == 0.0
        for t in range(n):
            pg = int(table[b, t // page])
            close(kv[pg, 0, :, t % page, :dk], k[t], 1e-5)
            close(kv[pg, 1, :, t % page, :dv], v[t], 1e-5)
            assert float(kv[pg, 0, :, t % page, dk:].abs().sum()) == 0.0 and float(kv[pg, 1, :, t % page, dv:].abs().sum()) == 0.0
        if taps > 1:
            close(state[slots[b]].view(taps - 1, C), us[b][n - taps + 1:], 1e-6)
    assert float((state[1] - 5.0).abs().max()) == 0.0


def test_angles_of_far_positions():
    """Positions up to a million: with the frequencies' low parts the turn is that of the exact angle; the product of float32
    numbers alone is off by hundredths of a radian there."""
    from sharpinference_b200.kernels import ops
    from sharpinference_b200.parts.position import leading_rotary_inv_freq_parts
    rot, base = 16, 30.0
    inv, low = leading_rotary_inv_freq_parts(rot, base)
    pos = [0, 5, 997, 40009, 999983]
    u = _rand(5, 3 * rot, seed=1)
    q = torch.empty(5, 1, rot, device=DEV)
    err = {}
    for name, lo in (("with", low.to(DEV)), ("without", None)):
        kv = torch.zeros(1, 2, 1, 1, rot, device=DEV)
        ops.qkv_conv(f32(u), q, kv, weight=torch.ones(1, 3 * rot, device=DEV), state=None, positions=i32(pos), row_req=i32([0] * 5),
                     row_offsets=i32([0, 5]), state_slots=i32([0]), block_table=torch.zeros(1, 1000000, dtype=torch.int32, device=DEV),
                     nq=1, nkv=1, D=rot, key_dim=rot, value_dim=rot, page_size=1, inv_freq=inv.to(DEV), inv_freq_low=lo, rot_dims=rot)
        a = torch.tensor(pos, dtype=F64).view(5, 1) * base ** (-2.0 * torch.arange(rot // 2, dtype=F64) / rot)
        x, y = u[:, : rot // 2], u[:, rot // 2: rot]
        want = torch.cat([x * torch.cos(a) - y * torch.sin(a), y * torch.cos(a) + x * torch.sin(a)], dim=1)
        err[name] = float((q[:, 0].double().cpu() - want).abs().max())
    assert err["with"] < 2e-6 and err["without"] > 1e-3, err


@pytest.mark.parametrize("fast", [False, True])
@pytest.mark.parametrize("H,d,dv,decay", [(2, 32, 32, (0.6, 0.999)), (3, 5, 7, (0.7, 0.0, 1.0)), (1, 128, 128, (0.995,)),
                                          (2, 64, 40, (0.9, 0.99)), (1, 160, 72, (0.98,)), (1, 300, 24, (0.97,)), (2, 1, 1, (0.5, 0.9)),
                                          (1, 96, 200, (0.9,)), (2, 128, 64, (0.3, 0.9999))])
def test_decayed_sums_walked_and_in_chunks(H, d, dv, decay, fast):
    """Three requests on slots of their own, in portions of one to 150 rows, walked and in chunks of 64 (also a last chunk of
    one row), against the sums row by row; the two forms continue one another's state."""
    from sharpinference_b200.kernels import ops
    from sharpinference_b200.parts import LightningPlanner
    cols = 2 * H * d + H * dv
    powers = ops.decay_powers(decay).to(DEV)
    sizes = [[150, 3, 65, 1], [1, 129, 2, 33], [40, 32, 1, 64]]
    n = [sum(s) for s in sizes]
    us = [_rand(m, cols, seed=70 + i) for i, m in enumerate(n)]
    slots = [3, 0, 2]
    state = torch.zeros(4, H * d * dv, device=DEV)
    state[1] = 5.0
    got = [[], [], []]
    at = [0, 0, 0]
    for step in range(4):
        lens = [sizes[b][step] for b in range(3)]
        proj = torch.cat([us[b][at[b]: at[b] + lens[b]] for b in range(3)])
        proj = torch.cat([_rand(sum(lens), 4, seed=1), proj, _rand(sum(lens), 3, seed=2)], dim=1)
        plan = LightningPlanner().plan(at, lens)
        off = [0, lens[0], lens[0] + lens[1], sum(lens)]
        dev = {k: (torch.from_numpy(v).to(DEV) if v.size else None) for k, v in plan.arrays.items()}
        y = ops.lightning(f32(proj), col_q=4, col_k=4 + H * d, col_v=4 + 2 * H * d, powers=powers, row_offsets=i32(off),
                          state_slots=i32(slots), state=state, heads=H, d=d, dv=dv, num_requests=3, walk_requests=dev["walk"],
                          num_walk=plan.values["num_walk"], chunks=dev["chunks"], spans=dev["spans"],
                          fast_activations=fast).cpu()
        for b in range(3):
            got[b].append(y[off[b]: off[b + 1]])
            at[b] += lens[b]
    for b in range(3):
        s = plain.silu(us[b])
        q, k, v = s[:, : H * d].reshape(-1, H, d), s[:, H * d: 2 * H * d].reshape(-1, H, d), s[:, 2 * H * d:].reshape(-1, H, dv)
        want, S = plain.decayed_sums(q, k, v, decay)
        close(torch.cat(got[b]), want.reshape(-1, H * dv), 3e-6)
        close(state[slots[b]].view(H, d, dv), S, 3e-6)
    assert float((state[1] - 5.0).abs().max()) == 0.0


@pytest.mark.parametrize("T,n", [(3, 1), (50, 36), (5, 2048), (7, 2100), (4, 9000)])
def test_norm_with_a_sigmoid_gate(T, n):
    from sharpinference_b200.kernels import ops
    y, g, w = _rand(T, n, seed=1, scale=4.0), _rand(T, n + 3, seed=2, scale=2.0), _rand(n, seed=3)
    wide = torch.full((T, n + 9), 7.0, device=DEV)
    ops.norm_sigmoid_gate(f32(y), f32(g)[:, 2: 2 + n], f32(w), 1e-4, wide[:, 4: 4 + n], scale=0.7)
    want = torch.full((T, n + 9), 7.0, dtype=F64)
    want[:, 4: 4 + n] = plain.rms(y, w, 1e-4) * torch.sigmoid(g[:, 2: 2 + n]) * 0.7
    close(wide, want, 2e-6)


@pytest.mark.parametrize("T,H,N,k,groups,keep", [(1, 64, 6, 2, 1, 1), (37, 52, 12, 3, 4, 2), (600, 128, 18, 4, 3, 1), (5, 16, 1, 1, 1, 1),
                                                 (9, 96, 80, 5, 40, 7), (700, 40, 16, 2, 2, 2), (20, 2048, 24, 3, 4, 3)])
def test_router_with_groups_and_a_gate_row(T, H, N, k, groups, keep):
    from sharpinference_b200.kernels import ops
    h, wr, corr, gw = _rand(T, H, seed=T), _rand(N, H, seed=N, scale=2.0 / H ** 0.5), _rand(N, seed=k) - 1.0, _rand(H, seed=9, scale=H ** -0.5)
    expert, weight, gate, scores = ops.router_groups(f32(h), f32(wr), k, correction=f32(corr), scale=1.6, n_groups=groups, keep=keep,
                                                     gate_weight=f32(gw), want_scores=True)
    s = torch.softmax(h @ wr.T, -1)
    close(scores, s, 2e-6)
    close(gate, torch.sigmoid(h @ gw), 2e-6)
    router = {"top": k, "groups": {"count": groups, "keep": keep}}
    idx = plain.choose(s + corr, router)
    same = (expert.cpu().long() == idx).all(-1)
    assert float(same.float().mean()) > 0.99                                    # only a tie within rounding may differ
    w = s.gather(1, idx)
    w = w / (w.sum(-1, keepdim=True) + 1e-20) * 1.6
    close(weight.cpu()[same], w[same], 3e-6)
    # no gate row, no correction, weights as they are
    e2, w2, g2, _ = ops.router_groups(f32(h), f32(wr), k, scale=2.0, renormalize=False)
    val, i2 = s.topk(k, -1)
    ok = (e2.cpu().long() == i2).all(-1)
    assert g2 is None and float(ok.float().mean()) > 0.99
    close(w2.cpu()[ok], 2.0 * val[ok], 2e-6)


def test_groups_that_are_not_kept_lose_to_negative_choice_scores():
    """Corrections far below zero: the kept group's second expert has a choice score of about -8, every expert of the other
    group about -1, and it is chosen all the same; equal groups: the first is kept."""
    from sharpinference_b200.kernels import ops
    h = torch.zeros(3, 8, device=DEV)
    wr = torch.zeros(4, 8, device=DEV)
    corr = torch.tensor([-0.5, -8.0, -1.0, -1.0], device=DEV)
    expert, weight, _, _ = ops.router_groups(h, wr, 2, correction=corr, n_groups=2, keep=1)
    assert expert.tolist() == [[0, 1]] * 3 and torch.allclose(weight, torch.full_like(weight, 0.5))
    expert, _, _, _ = ops.router_groups(h, wr, 2, n_groups=2, keep=1)
    assert expert.tolist() == [[0, 1]] * 3


@pytest.mark.parametrize("T,k,H,E,ident", [(1, 1, 8, 2, 1), (33, 3, 52, 4, 2), (70, 2, 64, 5, 0), (9, 4, 7, 1, 3)])
def test_combining_pairs_identity_shared_and_add_in(T, k, H, E, ident):
    from sharpinference_b200.kernels import ops
    y, h, shared, add, gate = _rand(T * k, H, seed=1), _rand(T, H, seed=2), _rand(T, H, seed=3), _rand(T, H, seed=4), _rand(T, seed=5)
    g = torch.Generator().manual_seed(T)
    expert = torch.randint(0, E + ident, (T, k), generator=g)
    weight = _rand(T, k, seed=6)
    base = torch.zeros(T, H, dtype=F64)
    for j in range(k):
        pick = (expert[:, j] < E).view(T, 1)
        base = base + torch.where(pick, y.view(T, k, H)[:, j], weight[:, j: j + 1] * h)
    for sh, ga, ad in ((shared, gate, add), (shared, None, None), (None, None, add), (None, None, None)):
        dev = lambda t: None if t is None else f32(t)
        a = dev(ad)
        yp = f32(y)
        yp.view(T, k, H)[(expert >= E).to(DEV)] = float("nan")                  # rows of identity pairs are never read
        got = ops.moe_combine_full(yp, expert.to(torch.int32).to(DEV), f32(weight), f32(h), E, shared=dev(sh), gate=dev(ga), add=a, out=a)
        want = base + (0 if sh is None else (1 if ga is None else ga.view(T, 1)) * sh) + (0 if ad is None else ad)
        close(got, want, 3e-6)


@pytest.mark.parametrize("rows,K,I,E", [(5, 64, 40, 3), (100, 128, 64, 4), (300, 96, 200, 2), (1500, 64, 136, 5), (2, 512, 256, 8)])
def test_grouped_product_with_the_clamped_gate(rows, K, I, E):
    """Every form of the grouped tcgen05 product (K split, row tiles, persistent), with rows behind the last group that
    belong to no expert."""
    from sharpinference_b200.kernels import ops
    extra = 7
    a = _rand(rows + extra, K, seed=rows).to(torch.bfloat16)
    w = _rand(E, 2 * I, K, seed=K, scale=K ** -0.5).to(torch.bfloat16)
    cuts = sorted(torch.randint(0, rows + 1, (E - 1,), generator=torch.Generator().manual_seed(rows)).tolist())
    off = [0] + cuts + [rows]
    limit = 0.8
    got = ops.tc_grouped_gemm_clamped(a.to(DEV), w.to(DEV), i32(off), limit)
    ops.check_status(DEV)
    want = torch.zeros(rows, I, dtype=F64)
    for e in range(E):
        z = a[off[e]: off[e + 1]].double() @ w[e].double().T
        g, u = z[:, :I].clamp(max=limit), z[:, I:].clamp(-limit, limit)
        want[off[e]: off[e + 1]] = g * torch.sigmoid(1.702 * g) * (u + 1)
    assert float((got[:rows].double().cpu() - want).abs().max()) < 8e-3 * float(want.abs().max())


# ------------------------------------------------------------------------------------------
# one layer at a time, through the engine
# ------------------------------------------------------------------------------------------
@pytest.mark.parametrize("name,index", [(n, i) for n in sorted(CASES) for i in range(len(CASES[n][0]["layers"]))])
def test_each_layer_alone(tmp_path, name, index):
    """A model of one layer: the residual stream behind it against the plain mixer's and feed-forward's outputs; a prompt of
    150 tokens in one step, then the same prompt with its last 40 tokens one by one."""
    from radupel_models import one_layer, write_config
    from sharpinference_b200 import StepEntry
    _, std, seed = CASES[name]
    for variant, mlp in (("bare", None), ("own", "same")):
        cfg = one_layer(name, index, mlp)
        if variant == "own" and cfg["layers"][0]["mlp"] is None:
            continue
        folder = write_config(cfg, std, seed + index, str(tmp_path / variant))
        cfg, w = plain.load_folder(folder)
        toks = traces.random_tokens(cfg["vocab"], 150, seed=index)
        after = []
        plain.forward(cfg, w, toks, layers_out=after)
        x, eps, one = w["embed"][torch.tensor(toks)], cfg["norm"]["eps"], cfg["layers"][0]
        want = x + plain.side_by_side(plain.rms(x, w["l0.norm1"], eps), one["mixer"], w, "l0.mix.", eps)
        if one["mlp"] is not None:
            want = want + plain.feed_forward(plain.rms(x, w["l0.norm2"], eps), one["mlp"], w, "l0.mlp.")[0]
        assert float((want - after[0]).abs().max()) < 1e-9
        eng = engine_for(folder, "float32", 256)
        eng.runner.trace_streams = True
        scale = float(want.abs().max())
        eng.open_request("a")
        eng.forward_step([StepEntry("a", toks, [])])
        got = eng.runner.last_layer_streams[0].double().cpu()
        assert float((got - want).abs().max()) < 3e-5 * scale, (variant, "prompt")
        eng.close_request("a")
        eng.open_request("b")
        eng.forward_step([StepEntry("b", toks[:110], [])])
        for t in range(110, 150):
            eng.forward_step([StepEntry("b", [toks[t]], [])])
            got = eng.runner.last_layer_streams[0].double().cpu()
            assert float((got[0] - want[t]).abs().max()) < 3e-5 * scale, (variant, "decoded", t)
        eng.close_request("b")


# ------------------------------------------------------------------------------------------
# whole models through the engine
# ------------------------------------------------------------------------------------------
@pytest.mark.parametrize("name", sorted(CASES))
def test_layers_one_after_the_other(folders, name):
    """The residual stream behind every layer run of a whole model against the plain model's."""
    from sharpinference_b200 import StepEntry
    cfg, w = plain.load_folder(folders[name])
    toks = traces.random_tokens(cfg["vocab"], 140, seed=8)
    after = []
    plain.forward(cfg, w, toks, layers_out=after)
    eng = engine_for(folders[name], "float32", 256)
    eng.runner.trace_streams = True
    eng.open_request("a")
    eng.forward_step([StepEntry("a", toks, [])])
    assert len(eng.runner.last_layer_streams) == len(after)
    for i, (got, want) in enumerate(zip(eng.runner.last_layer_streams, after)):
        assert float((got.double().cpu() - want).abs().max()) < 5e-5 * float(want.abs().max()), i
    eng.close_request("a")


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("name", sorted(CASES))
def test_whole_prompts(folders, expected, name, dtype):
    run_and_compare(folders[name], name, dtype, traces.whole(requests_for(name)), expected)


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("name", sorted(CASES))
def test_prompt_then_token_by_token(folders, expected, name, dtype):
    """The last 110 tokens one by one; the shorter requests from their first token on."""
    run_and_compare(folders[name], name, dtype, traces.tail_decode(requests_for(name), tail=110), expected)


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("name", sorted(CASES))
def test_portions_down_to_two_tokens(folders, expected, name, dtype):
    """Portions shorter and longer than the convolutions' memory, at and around the size from which the linear attention works
    in chunks, and across chunk borders."""
    run_and_compare(folders[name], name, dtype, traces.portions(requests_for(name)), expected)
    run_and_compare(folders[name], name, dtype, traces.portions(requests_for(name), sizes=(2, 17, 3, 64, 1, 32, 2, 65, 33, 2)),
                    expected, page_size=16)


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("name", sorted(CASES))
def test_mixed_batches_reuse_pages_and_slots(folders, expected, name, dtype):
    """Up to three live requests for three slots and a pool sized for the schedule's peak: every later request runs on pages
    and state slots that an earlier one left behind."""
    steps = traces.mixed(requests_for(name), max_live=3)
    eng = run_and_compare(folders[name], name, dtype, steps, expected, max_batch=3)
    assert eng.cache.state_slots.free_count == 3
    run_and_compare(folders[name], name, dtype, traces.drawn(requests_for(name), seed=5, max_live=4), expected)
    run_and_compare(folders[name], name, dtype, traces.drawn(requests_for(name), seed=6, max_live=4), expected, page_size=16)


@pytest.mark.parametrize("name", sorted(CASES))
def test_one_slot_for_all_requests_in_turn(folders, expected, name):
    """One request's worth of pages and one state slot, first decoded token by token, then whole: nothing of the request
    before is left in either."""
    reqs = requests_for(name)
    eng = engine_for(folders[name], "float32", 256, max_batch=1)
    for rid, toks in reqs.items():
        for steps in (traces.tail_decode({rid: toks}, tail=len(toks)), traces.whole({rid: toks})):
            got = traces.replay(eng, steps)
            err, where = traces.worst_error(got, expected[name])
            assert err < TOL["float32"], (rid, err, where)


def test_a_first_token_is_remembered_for_hundreds(folders):
    """The slow heads keep what they saw: exchanging a request's first token moves the plain logits 200 tokens later by many
    tolerances, and the engine's logits there are right, in a prompt's portion and decoded."""
    cfg, w = plain.load_folder(folders["C"])
    toks = traces.random_tokens(cfg["vocab"], 230, seed=21)
    want = plain.forward(cfg, w, toks)
    other = plain.forward(cfg, w, [(toks[0] + 7) % cfg["vocab"]] + toks[1:])
    moved = (other - want).abs().max(-1).values / float(want.abs().max())
    assert float(moved[200:].max()) > 20 * TOL["float32"]
    eng = engine_for(folders["C"], "float32", 256)
    got = traces.replay(eng, traces.tail_decode({"r": toks}, tail=15))
    assert traces.worst_error(got, {"r": want})[0] < TOL["float32"]


def _aim(w, cfg, marked, asking):
    """Edit layer 0 so that the query of token ``asking`` meets the key of token ``marked`` with a score far above every other:
    a rank-one term in the key projection along what sets the marked token's normed embedding apart from the average one, and
    one in the query's, in an element that is not rotated and whose convolution passes the current token alone."""
    m, p = cfg["layers"][0]["mixer"]["left"], "l0.mix.left."
    e = m["rot"]["dims"]
    h = plain.rms(w["embed"], w["l0.norm1"], cfg["norm"]["eps"])
    vk, vq = h[marked] - h.mean(0), h[asking] - h.mean(0)
    w[p + "k"][e] += 14.0 * vk / (vk @ vk)
    for hd in range(m["heads"]):
        w[p + "q"][hd * m["dim"] + e] += 14.0 * vq / (vq @ vq)
        w[p + "q.conv"][hd * m["dim"] + e] = torch.eye(m["conv"], dtype=F64)[-1]
    w[p + "k.conv"][e] = torch.eye(m["conv"], dtype=F64)[-1]
    return w


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_a_far_key_among_hundreds_carries_the_output(tmp_path, dtype):
    """The last token's query meets the key of one early token with a score far above all others: 400 positions back and
    across six pages, at both sides of a page's border, in a prompt's last row and in a decoded token.  Exchanging that early
    token then changes the layer's output at the end by a visible part of its size."""
    from radupel_models import layer, left, right, top, write_config
    from safetensors.torch import save_file
    from sharpinference_b200 import StepEntry
    cfg = top(40, 32, 1e-5, 0.0, [layer(left(2, 1, 16, 16, 0.6, 3, (8, 1000.0)), right(1, 8, 8, (0.5,)), (1.0, 0.3), None)])
    folder = write_config(cfg, 0.3, 5, str(tmp_path / "base"))
    cfg, w = plain.load_folder(folder)
    w = _aim(w, cfg, marked=37, asking=39)
    variant = str(tmp_path / "aimed")
    os.makedirs(variant)
    save_file({k: v.to(torch.bfloat16).contiguous() for k, v in w.items()}, os.path.join(variant, "model.safetensors"))
    with open(os.path.join(variant, "config.json"), "w") as fh:
        json.dump(cfg, fh)
    cfg, w = plain.load_folder(variant)
    n = 403
    eng = engine_for(variant, dtype, 512)
    for place in (0, 2, 63, 64, 320):
        toks = [t % 30 for t in traces.random_tokens(30, n, seed=3)]
        toks[place], toks[-2], toks[-1] = 37, 39, 39                 # the asking token as a prompt's last row and decoded
        after, other = [], []
        want = plain.forward(cfg, w, toks, layers_out=after)
        plain.forward(cfg, w, toks[:place] + [5] + toks[place + 1:], layers_out=other)
        for row in (n - 2, n - 1):
            assert float((after[-1][row] - other[-1][row]).abs().max()) / float(after[-1].abs().max()) > 0.03
        eng.open_request("a")
        lg = eng.forward_step([StepEntry("a", toks[:-1], [n - 2])]).double().cpu()
        assert float((lg[0] - want[n - 2]).abs().max()) < TOL[dtype] * float(want.abs().max()), place
        lg = eng.forward_step([StepEntry("a", toks[-1:], [0])]).double().cpu()
        assert float((lg[0] - want[n - 1]).abs().max()) < TOL[dtype] * float(want.abs().max()), place
        eng.close_request("a")


@pytest.mark.parametrize("seed", [3, 14, 15, 92, 65, 35])
def test_drawn_configurations(tmp_path, seed):
    """Configurations drawn at random with requests of 2 to 700 tokens: whole, with decoded tails, and in drawn mixed batches,
    in 32-bit; bfloat16 whole, held to what rounding does."""
    from radupel_models import drawn_config, write_config
    cfg = drawn_config(seed)
    folder = write_config(cfg, 0.1, seed, str(tmp_path))
    cfg, w = plain.load_folder(folder)
    reqs = {f"q{i}": traces.random_tokens(cfg["vocab"], n, seed=seed * 7 + i) for i, n in enumerate([330, 37, 150, 700, 2])}
    ref = {rid: plain.forward(cfg, w, toks) for rid, toks in reqs.items()}
    for steps in (traces.whole(reqs), traces.tail_decode(reqs, tail=40), traces.drawn(reqs, seed=seed, max_live=4)):
        eng = engine_for(folder, "float32", traces.max_tokens(steps))
        err, where = traces.worst_error(traces.replay(eng, steps), ref)
        eng.runner.flush_status()
        assert err < TOL["float32"], (err, where)
    steps = traces.whole(reqs)
    eng = engine_for(folder, "bfloat16", traces.max_tokens(steps))
    routing, slack = {}, {}
    got = traces.replay(eng, steps, routing)
    excess, where = worst_excess(got, reference_for(folder, reqs, routing, None, "bfloat16", slack, margin=0.15), TOL["bfloat16"], slack)
    assert excess < 2.0, (excess, where)


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("name", ["A", "C"])
def test_long_decoding_through_graphs(folders, name, dtype):
    """Three requests decode 260 tokens each side by side, over several pages; decode-only steps are replayed as CUDA graphs."""
    cfg, w = plain.load_folder(folders[name])
    reqs = {f"d{i}": traces.random_tokens(cfg["vocab"], 263 + i, seed=200 + i) for i in range(3)}
    steps = [{"step": 0, "entries": [{"id": rid, "tokens": toks[:3 + i], "want": [2 + i]}
                                     for i, (rid, toks) in enumerate(reqs.items())], "end": []}]
    for t in range(260):
        steps.append({"step": t + 1, "entries": [{"id": rid, "tokens": [toks[3 + i + t]], "want": [0]}
                                                 for i, (rid, toks) in enumerate(reqs.items())],
                      "end": list(reqs) if t == 259 else []})
    eng = engine_for(folders[name], dtype, traces.max_tokens(steps))
    routing = {} if dtype == "bfloat16" else None
    got = traces.replay(eng, steps, routing)
    slack = None
    if routing is None:
        assert eng.runner.graph_replays > 200
        ref = {rid: plain.forward(cfg, w, toks) for rid, toks in reqs.items()}
    else:
        slack = {}
        ref = reference_for(folders[name], reqs, routing, None, dtype, slack)
    excess, where = worst_excess(got, ref, TOL[dtype], slack)
    assert excess < 1.0, (excess, where)


@pytest.mark.parametrize("name", ["A", "C"])
def test_graphs_give_the_bits_of_eager_steps_in_bfloat16(folders, name):
    """Decode steps replayed as graphs against the same steps run eagerly (the branches and the feed-forward run on streams of
    their own; a missing join would show as a difference)."""
    from sharpinference_b200 import StepEntry
    cfg, _ = plain.load_folder(folders[name])
    toks = {f"d{i}": traces.random_tokens(cfg["vocab"], 60, seed=400 + i) for i in range(3)}
    rows = {}
    for graphs in (True, False):
        eng = engine_for(folders[name], "bfloat16", 3 * 64 + 64)
        eng.runner.use_graphs = eng.runner.use_graphs and graphs
        for rid, t in toks.items():
            eng.open_request(rid)
            eng.forward_step([StepEntry(rid, t[:20], [])])
        got = [eng.forward_step([StepEntry(rid, [t[at]], [0]) for rid, t in toks.items()]).cpu().clone() for at in range(20, 60)]
        assert (eng.runner.graph_replays > 30) == graphs
        rows[graphs] = torch.stack(got)
    assert torch.equal(rows[True], rows[False])


@pytest.mark.parametrize("name", sorted(CASES))
def test_greedy_generation_through_the_scheduler(folders, name):
    """``Engine.generate``: admission, portions under a small token budget, decoding in one batch, sampling (greedy) and the
    release of pages and slots, against the plain model generating token by token."""
    from sharpinference_b200 import Engine, EngineOptions, SamplingParams
    cfg, w = plain.load_folder(folders[name])
    prompts = [traces.random_tokens(cfg["vocab"], n, seed=300 + n) for n in (5, 41, 90, 17, 2)]
    opts = EngineOptions()
    opts.max_cache_tokens, opts.max_batch, opts.max_tokens_per_step = 1024, 3, 48
    eng = Engine(folders[name], dtype="float32", device=DEV, options=opts)
    outs = eng.generate(prompts, SamplingParams(temperature=0.0, max_new_tokens=12))
    for prompt, out in zip(prompts, outs):
        assert out == plain.generate_greedy(cfg, w, prompt, 12)
    m = eng.metrics()
    assert m["state_slots_free"] == 3 and all(g["held"] == 0 for g in m["cache_groups"].values())


def test_preempted_requests_start_over(folders):
    """A pool too small for all: the newest request is sent back, its pages and state slot are given up, and it is computed
    again from its first token."""
    from sharpinference_b200 import Engine, EngineOptions, SamplingParams
    cfg, w = plain.load_folder(folders["A"])
    prompts = [traces.random_tokens(cfg["vocab"], n, seed=500 + n) for n in (60, 50, 44)]
    opts = EngineOptions()
    opts.page_size, opts.max_cache_tokens, opts.max_batch, opts.max_tokens_per_step = 16, 176, 3, 64
    eng = Engine(folders["A"], dtype="float32", device=DEV, options=opts)
    outs = eng.generate(prompts, SamplingParams(temperature=0.0, max_new_tokens=20))
    for prompt, out in zip(prompts, outs):
        assert out == plain.generate_greedy(cfg, w, prompt, 20)


def test_command_line_and_trace_program(folders, capsys, tmp_path):
    """``sharpi-cli`` generates greedily on a Radupel folder, and ``bin/trace_run`` as a child process replays a mixed schedule
    from standard input and writes the logits the plain model gives."""
    import subprocess
    import sys

    import numpy as np

    from sharpinference_b200 import cli
    cfg, w = plain.load_folder(folders["C"])
    prompt = traces.random_tokens(cfg["vocab"], 21, seed=9)
    rc = cli.main(["-m", folders["C"], "--tokens", ",".join(map(str, prompt)), "-n", "6", "--temp", "0", "--dtype", "float32",
                   "--repeat-penalty", "1.0", "--json", "--max-cache-tokens", "256"])
    out = capsys.readouterr()
    assert rc == 0
    assert json.loads(out.out.strip().splitlines()[-1])["outputs"][0]["tokens"] == plain.generate_greedy(cfg, w, prompt, 6)

    reqs = {f"t{i}": traces.random_tokens(cfg["vocab"], n, seed=50 + i) for i, n in enumerate((40, 3, 77, 18, 166))}
    steps = traces.mixed(reqs, max_live=4)
    root = os.path.dirname(os.path.dirname(os.path.abspath(__file__)))
    res = subprocess.run([sys.executable, os.path.join(root, "bin", "trace_run"), "--model", folders["C"], "--dtype", "float32",
                          "--out", str(tmp_path), "--max-tokens", str(traces.max_tokens(steps))],
                         input="\n".join(json.dumps(s) for s in steps) + "\n", capture_output=True, text=True, timeout=900)
    assert res.returncode == 0, res.stderr[-2000:]
    assert [ln for ln in res.stdout.splitlines() if ln.startswith("done ")] == [f"done {s['step']}" for s in steps]
    ref = {rid: plain.forward(cfg, w, toks) for rid, toks in reqs.items()}
    at = {rid: 0 for rid in reqs}
    for st in steps:
        rows = np.fromfile(os.path.join(str(tmp_path), f"{st['step']}.f32"), dtype="<f4").reshape(-1, cfg["vocab"])
        r = 0
        for e in st["entries"]:
            for wpos in e["want"]:
                want = ref[e["id"]][at[e["id"]] + wpos]
                assert float((torch.from_numpy(rows[r]).double() - want).abs().max()) < TOL["float32"] * float(ref[e["id"]].abs().max())
                r += 1
            at[e["id"]] += len(e["tokens"])


def test_parts_are_registered():
    from sharpinference_b200.parts import part_kinds
    assert {"conv_attention", "lightning_attention", "scaled_branches"} <= set(part_kinds("mixer"))
    assert "parallel_pair" in part_kinds("block") and "add_input" in part_kinds("stream")
    assert "moe_softmax_groups" in part_kinds("feed_forward")


def test_a_branch_by_itself_is_a_mixer():
    """Linear attention outside a pair: its own two products around its inner columns, in portions of 50, 3 and 40 rows."""
    from types import SimpleNamespace

    from sharpinference_b200.parts import LayerSlot, LightningAttention, LightningPlanner, lightning_columns
    W, H, d, dv = 24, 3, 6, 10
    t = {"q": _rand(H * d, W, seed=1), "k": _rand(H * d, W, seed=2), "v": _rand(H * dv, W, seed=3), "g": _rand(H * dv, W, seed=4),
         "o": _rand(W, H * dv, seed=5), "norm": _rand(H * dv, seed=6)}
    m = {"heads": H, "dim": d, "vdim": dv, "decay": [0.5, 0.9, 0.99]}
    rows = torch.cat([t[s] for s in "qkvg"])
    proj = torch.zeros(lightning_columns(H, d, dv)[-1], W, dtype=F64)
    proj[: rows.shape[0]] = rows
    mixer = LightningAttention(proj=f32(proj), out=f32(t["o"]), norm_weight=f32(t["norm"]), decay=m["decay"], heads=H, dim=d,
                               value_dim=dv, eps=1e-5, act_dtype=torch.float32)
    state = torch.zeros(2, mixer.state_specs["S"].shape[0], device=DEV)
    slot = LayerSlot(index=0, layer=0, states={"S": state})
    h = _rand(93, W, seed=7, scale=0.3)
    got, at = [], 0
    for n in (50, 3, 40):
        data = LightningPlanner().plan([at], [n])
        arrays = {k: (torch.from_numpy(v).to(DEV) if v.size else None) for k, v in data.arrays.items()}
        ctx = SimpleNamespace(num_tokens=n, num_requests=1, row_offsets=i32([0, n]), state_slots=i32([1]),
                              plans={LightningPlanner.key: SimpleNamespace(**arrays, **data.values)})
        got.append(mixer.forward(ctx, slot, f32(h[at: at + n])).cpu())
        at += n
    close(torch.cat(got), plain.lightning(h, m, t, "", 1e-5), 1e-5)
    assert float(state[0].abs().max()) == 0.0
