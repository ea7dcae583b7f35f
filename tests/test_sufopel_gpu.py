"""Sufopel on the GPU: each new kernel against the plain statement of its mechanism, each layer alone through a model of one
layer, and whole models through the engine (step function, cache manager, scheduler) under every way of cutting the work, in
32-bit and in bfloat16."""
import json
import os

import pytest
import torch

import plain_sufopel as plain
import traces
from sufopel_models import CASES, write

pytestmark = pytest.mark.gpu
DEV = "cuda:0"
F64 = torch.float64

# Relative to the largest |logit| of a request.
TOL = {"float32": 5e-5, "bfloat16": 4e-2}
# A differing expert choice must be a near-tie of the choice scores.
MARGIN = 1e-1
LENGTHS = {"A": [1, 9, 40, 83, 150, 2], "B": [150, 5, 67, 200, 31], "C": [3, 70, 140, 45, 210, 64, 65],
           "D": [1, 2, 30, 5, 100], "E": [140, 66, 3, 129, 200]}


def requests_for(name):
    vocab = CASES[name][0]["vocab"]
    return {f"r{i}": traces.random_tokens(vocab, n, seed=47 * i + n) for i, n in enumerate(LENGTHS[name])}


@pytest.fixture(scope="module")
def folders(tmp_path_factory):
    return {name: write(name, str(tmp_path_factory.mktemp(f"sufopel_{name}"))) for name in CASES}


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
    """Every forced set of experts is the router's own up to ``margin``: the groups it lies in are (nearly) the best, and its
    experts are (nearly) the largest within these groups."""
    groups = router.get("groups") or {"count": 1, "keep": 1}
    n, E = score.shape
    per = E // groups["count"]
    best = plain.group_scores(score, groups["count"])
    kth_group = best.topk(groups["keep"], dim=-1).values[:, -1]
    assert float((kth_group - best.gather(1, forced // per).min(-1).values).max()) < 2 * margin, f"request {rid}: a group beyond a near-tie"
    mine = torch.zeros(n, groups["count"], dtype=torch.bool)
    mine[torch.arange(n).view(n, 1), forced // per] = True
    own = score.masked_fill(~mine.repeat_interleave(per, dim=1), -1e9)
    kth = own.topk(forced.shape[1], dim=-1).values[:, -1]
    assert float((kth - score.gather(1, forced).min(-1).values).max()) < margin, f"request {rid}: an expert beyond a near-tie"


def reference_for(folder, reqs, routing, fallback, dtype, slack=None, margin=MARGIN):
    """float32 runs are held to the plain logits as they are; bfloat16 runs to the plain logits under the engine's own expert
    choices, each differing choice having to be a near-tie.  ``slack`` receives, per request, what rounding the operands of
    the matrix products alone does to every position's logits in the plain model: where that is more than the tolerance a
    bfloat16 run is held to three times it (or one and a half times what it does at the request's worst position)."""
    if dtype == "float32":
        return fallback
    cfg, w = plain.load_folder(folder)
    routers = [layer["mlp"]["router"] for layer in cfg["layers"] if layer["mlp"] and layer["mlp"]["kind"] == "moe"]
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
        allowed = max(tol, 3.0 * float(slack[rid][pos]), 1.5 * float(slack[rid].max())) if slack else tol
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


def on_device(plan):
    return {k: (torch.from_numpy(v).to(DEV) if v.size else None) for k, v in plan.arrays.items()}


# ------------------------------------------------------------------------------------------
# kernels alone
# ------------------------------------------------------------------------------------------
@pytest.mark.parametrize("T,H", [(3, 1), (11, 52), (7, 257), (130, 1024), (200, 96), (5, 2048), (150, 4096), (9, 6144), (140, 8192),
                                 (4, 12000), (3, 20000)])
def test_normed_update_and_norm(T, H):
    from sharpinference_b200.kernels import ops
    x, y, wy, w = 3 * _rand(T, H, seed=H), 5 * _rand(T, H, seed=H + 1), _rand(H, seed=H + 2), _rand(H, seed=H + 3)
    x, y = x.float().double(), y.float().double()
    new = x + plain.rms(y, wy, 1e-5)
    xd = f32(x)
    h, h32 = ops.add_normed(xd, f32(y), f32(wy), f32(w), 1e-5, torch.bfloat16, want_fp32=True)
    close(xd, new, 1e-6)
    close(h32, plain.rms(new, w, 1e-5), 3e-6 if H > 1 else 1e-4)               # (one element: its sign, unless it is tiny)
    assert torch.equal(h, h32.to(torch.bfloat16))
    xd = f32(x)
    bare, b32 = ops.add_normed(xd, f32(y), f32(wy), None, 1e-5, torch.float32, want_fp32=True)
    assert b32 is bare and torch.equal(bare, xd)
    close(xd, new, 1e-6)
    rows = [T - 1, 0, T // 2]
    xd = f32(x)
    some, _ = ops.add_normed(xd, f32(y), f32(wy), f32(w), 1e-5, torch.float32, rows=i32(rows))
    assert torch.equal(xd, f32(x))                                              # the stream stays as it is
    assert torch.equal(some, h32[torch.tensor(rows, device=DEV)])               # and a row's bits do not depend on the others


@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
def test_embedding_with_positions_and_side_gate(dtype):
    from sharpinference_b200.kernels import ops
    V, P, H, L, n = 31, 17, 75, 3, 5
    table, pos, side = (_rand(*s, seed=i).to(dtype) for i, s in enumerate(((V, H), (P, H), (V, L * n))))
    ids, at = [3, 30, 0, 3], [16, 0, 5, 2]
    got = ops.embed_pos(i32(ids), i32(at), table.to(DEV), pos.to(DEV), 1.75)
    close(got, table.double()[ids] * 1.75 + pos.double()[at], 1e-6)
    wide = 2 * _rand(4, 12, seed=9)
    gate = f32(wide)[:, 2: 2 + 8]                                               # padded from five to eight
    out = ops.side_gate(gate, i32(ids), side.to(DEV), 2 * n, n, dtype)
    want = torch.zeros(4, 8, dtype=F64)
    want[:, :n] = plain.gelu_tanh(wide[:, 2: 2 + n]) * side.double()[ids][:, 2 * n: 3 * n]
    close(out, want, 1e-6 if dtype == torch.float32 else 8e-3)
    assert float(out[:, n:].abs().sum()) == 0.0


@pytest.mark.parametrize("T,heads,n", [(1, 1, 1), (37, 3, 10), (9, 4, 64)])
def test_gates_of_the_heads_side_by_side(T, heads, n):
    from sharpinference_b200.kernels import ops
    v, wide = _rand(heads * T, n, seed=1), 2 * _rand(T, heads * n + 7, seed=2)
    want = v.view(heads, T, n).transpose(0, 1).reshape(T, heads * n)
    got = ops.head_minor(f32(v), heads=heads, out_dtype=torch.float32, gate=f32(wide)[:, 3: 3 + heads * n])
    close(got, want * torch.sigmoid(wide[:, 3: 3 + heads * n]), 1e-6)
    got = ops.head_minor(f32(v), heads=heads, out_dtype=torch.float32, gate=f32(wide)[:, 3: 3 + heads])
    close(got, want * torch.sigmoid(wide[:, 3: 3 + heads]).repeat_interleave(n, dim=1), 1e-6)


@pytest.mark.parametrize("T,H,E,k,groups,keep", [(1, 64, 6, 2, 1, 1), (37, 52, 12, 3, 4, 2), (600, 128, 18, 4, 3, 1), (5, 16, 1, 1, 1, 1),
                                                 (9, 96, 80, 5, 40, 7), (700, 40, 16, 2, 2, 2), (20, 2048, 24, 3, 4, 3), (30, 32, 4, 2, 4, 2)])
def test_router_with_sigmoid_scores_in_groups(T, H, E, k, groups, keep):
    from sharpinference_b200.kernels import ops
    h, wr, corr = _rand(T, H, seed=T), _rand(E, H, seed=E, scale=2.0 / H ** 0.5), _rand(E, seed=k) - 1.0
    expert, weight, _, scores = ops.router_groups(f32(h), f32(wr), k, correction=f32(corr), renormalize=False, n_groups=groups, keep=keep,
                                                  scoring="sigmoid", group_top=2, want_scores=True)
    s = torch.sigmoid(h @ wr.T)
    close(scores, s, 2e-6)
    idx = plain.choose(s + corr, {"top": k, "groups": {"count": groups, "keep": keep}})
    same = (expert.cpu().long() == idx).all(-1)
    assert float(same.float().mean()) > 0.99                                    # only a tie within rounding may differ
    close(weight.cpu()[same], s.gather(1, idx)[same], 2e-6)


def test_a_groups_two_best_count_together_and_negative_scores_beat_other_groups():
    from sharpinference_b200.kernels import ops
    h, wr = torch.zeros(2, 8, device=DEV), torch.zeros(6, 8, device=DEV)        # every score is 1/2
    corr = torch.tensor([0.4, -1.3, -1.4, -0.2, -0.3, -1.2], device=DEV)        # choice scores 0.9 -0.8 -0.9 | 0.3 0.2 -0.7
    kw = dict(correction=corr, renormalize=False, n_groups=2, keep=1, scoring="sigmoid")
    expert, weight, _, _ = ops.router_groups(h, wr, 3, group_top=2, **kw)
    assert expert.tolist() == [[3, 4, 5]] * 2 and torch.allclose(weight, torch.full_like(weight, 0.5))
    assert ops.router_groups(h, wr, 3, group_top=1, **kw)[0].tolist() == [[0, 1, 2]] * 2


@pytest.mark.parametrize("G,H,d,dv,taps,low", [(2, 4, 16, 24, 4, 8), (1, 3, 5, 7, 7, 16), (2, 2, 128, 128, 4, 40), (1, 2, 9, 3, 1, 8),
                                               (1, 1, 1, 1, 2, 8), (1, 2, 300, 24, 3, 24), (3, 3, 40, 200, 5, 8), (2, 6, 64, 32, 2, 136),
                                               (1, 1, 256, 8, 12, 8)])
def test_delta_inputs(G, H, d, dv, taps, low):
    """Two requests on two slots, in portions of one row, of fewer rows than the convolution looks back, and of more; the state a
    portion leaves is what the next one starts from, and a third slot is untouched."""
    from sharpinference_b200.kernels import ops
    from sharpinference_b200.parts import DeltaPlanner
    C, n = 2 * G * d + H * dv, 46
    w = _rand(C, taps, seed=C)
    us = [_rand(n, C + low + H + 3, seed=1), _rand(n, C + low + H + 3, seed=2)]
    slots, planner = [2, 0], DeltaPlanner(taps, True)
    state = torch.zeros(3, max(taps - 1, 1) * C, device=DEV)
    state[1] = 5.0
    got = [[], []]
    cuts = [[1, 2, 1, 1, 7, 3, 31], [5, 1, 20, 2, 1, 1, 16]]
    at = [0, 0]
    for m0, m1 in zip(*cuts):
        proj = torch.cat([us[0][at[0]: at[0] + m0], us[1][at[1]: at[1] + m1]])
        tiles = on_device(planner.plan(at, [m0, m1]))["tiles"]
        out = ops.delta_prep(f32(proj), conv_weight=f32(w.T), conv_state=state if taps > 1 else None, row_offsets=i32([0, m0, m0 + m1]),
                             state_slots=i32(slots), tiles=tiles, kv_heads=G, heads=H, d=d, dv=dv, low=low, act_dtype=torch.float32)
        for b, rows in ((0, slice(0, m0)), (1, slice(m0, None))):
            got[b].append(torch.cat([t[rows].cpu() for t in out], dim=1))
        at = [at[0] + m0, at[1] + m1]
    assert at == [n, n]
    for b in range(2):
        y = plain.silu(plain.causal_conv(us[b][:, :C], w))
        q = plain.unit(y[:, : G * d].reshape(n, G, d)) * d ** -0.5
        k = plain.unit(y[:, G * d: 2 * G * d].reshape(n, G, d))
        want = torch.cat([q.reshape(n, -1), k.reshape(n, -1), y[:, 2 * G * d:], torch.sigmoid(us[b][:, C + low: C + low + H]),
                          us[b][:, C: C + low]], dim=1)
        close(torch.cat(got[b]), want, 3e-6)
        if taps > 1:
            close(state[slots[b]].view(taps - 1, C), us[b][n - taps + 1:, :C], 1e-6)
    assert float((state[1] - 5.0).abs().max()) == 0.0


def _delta_case(n, G, H, d, dv, seed, kind):
    """Operands of the delta rule: unit keys, some of them repeated (a correction then matters), decays of the named kind."""
    q, k = plain.unit(_rand(n, G, d, seed=seed)) * d ** -0.5, plain.unit(_rand(n, G, d, seed=seed + 1))
    k[n // 2:] = k[: n - n // 2].clone()
    v, b = _rand(n, H, dv, seed=seed + 2), torch.sigmoid(2 * _rand(n, H, seed=seed + 3))
    z = {"mixed": 4 * _rand(n, H * d, seed=seed + 4) - 4, "slow": _rand(n, H * d, seed=seed + 4) - 9,
         "strong": 30 * _rand(n, H * d, seed=seed + 4)}[kind].float().double()
    return q.float().double(), k.float().double(), v, b.float().double(), z


@pytest.mark.parametrize("kind", ["mixed", "slow", "strong"])
@pytest.mark.parametrize("G,H,d,dv,split", [(2, 2, 32, 32, False), (1, 3, 5, 7, False), (1, 2, 192, 33, False), (1, 2, 192, 33, True),
                                            (1, 1, 128, 128, False), (1, 1, 128, 128, True), (2, 4, 64, 40, False), (2, 4, 64, 40, True),
                                            (1, 1, 160, 72, False), (1, 2, 300, 24, False), (1, 2, 1, 1, False), (1, 1, 96, 200, False),
                                            (1, 2, 256, 16, False), (1, 2, 256, 17, True), (1, 1, 36, 17, False)])
def test_delta_rule_walked_and_in_chunks(G, H, d, dv, split, kind):
    """Three requests on slots of their own, in portions of one to 150 rows, walked and in chunks of 16 (also a last chunk of one
    row), against the rows one by one; the two forms continue one another's state.  Decays near 1 throughout, spread, and ones
    that are zero in 32-bit: a closed form that divides by a product of decays, or sums their logarithms, fails on the last."""
    from sharpinference_b200.kernels import ops
    from sharpinference_b200.parts import DeltaPlanner
    sizes = [[150, 3, 65, 1], [1, 129, 2, 33], [40, 32, 1, 64]]
    n = [sum(s) for s in sizes]
    cases = [_delta_case(m, G, H, d, dv, 70 + 10 * i, kind) for i, m in enumerate(n)]
    bias, a_log = _rand(H * d, seed=5), 0.5 * _rand(H, seed=6)
    slots, planner = [3, 0, 2], DeltaPlanner(4, d <= ops.DELTA_MAX_CHUNK_KEY)
    dp = (d + 3) // 4 * 4
    state = torch.zeros(4, H * dv * dp, device=DEV)
    state[1] = 5.0
    got, at = [[], [], []], [0, 0, 0]
    for step in range(4):
        lens = [sizes[b][step] for b in range(3)]
        cut = lambda i, w: torch.cat([cases[b][i][at[b]: at[b] + lens[b]].reshape(lens[b], -1) for b in range(3)])
        qkv = torch.cat([cut(0, 0), cut(1, 0), cut(2, 0)], dim=1)
        z = torch.cat([_rand(sum(lens), 3, seed=1), cut(4, 0), _rand(sum(lens), 2, seed=2)], dim=1)
        plan = planner.plan(at, lens)
        dev = on_device(plan)
        off = [0, lens[0], lens[0] + lens[1], sum(lens)]
        y = ops.delta_rule(f32(qkv), f32(cut(3, 0)), f32(z)[:, 3: 3 + H * d], dt_bias=f32(bias), a_log=f32(a_log), row_offsets=i32(off),
                           state_slots=i32(slots), state=state, kv_heads=G, heads=H, d=d, dv=dv, num_requests=3, walk_requests=dev["walk"],
                           num_walk=plan.values["num_walk"], chunks=dev["chunks"], spans=dev["spans"], max_rows=plan.values["walk_rows"], split=split).cpu()
        for b in range(3):
            got[b].append(y[off[b]: off[b + 1]])
            at[b] += lens[b]
    for b in range(3):
        q, k, v, beta, z = cases[b]
        g = torch.exp(-torch.exp(a_log).view(1, H, 1) * torch.nn.functional.softplus(z + bias, threshold=1e9).view(-1, H, d))
        want, S = plain.delta_rule(q.repeat_interleave(H // G, 1), k.repeat_interleave(H // G, 1), v, g, beta)
        close(torch.cat(got[b]), want.reshape(-1, H * dv), 3e-6)
        stored = state[slots[b]].view(H, dv, dp)
        close(stored[..., :d], S.transpose(1, 2), 3e-6)
        assert float(stored[..., d:].abs().sum()) == 0.0
    assert float((state[1] - 5.0).abs().max()) == 0.0


def test_a_key_written_once_is_read_back_hundreds_of_rows_later():
    """Slow decays, one key that stands out: its value comes back 400 rows later, from a portion in chunks and from walked rows, and
    a second value written under the same key replaces the first."""
    from sharpinference_b200.kernels import ops
    from sharpinference_b200.parts import DeltaPlanner
    n, d, dv = 440, 32, 16
    k = plain.unit(torch.cat([torch.zeros(n, 1, 1, dtype=F64), _rand(n, 1, d - 1, seed=1)], dim=-1))
    k[:, :, 1:16] = 0.0
    v, b = 0.1 * _rand(n, 1, dv, seed=2), torch.full((n, 1), 0.2, dtype=F64)
    for row, val in ((3, 4.0), (200, -7.0)):
        k[row] = 0.0
        k[row, 0, 0] = 1.0
        v[row], b[row] = val, 1.0
    q = torch.zeros(n, 1, d, dtype=F64)
    q[:, 0, 0] = 1.0
    z = torch.full((n, d), -11.0, dtype=F64)
    for cuts in ([n], [150] * 2 + [30] * 4 + [1] * 20):
        state = torch.zeros(1, dv * d, device=DEV)
        rows, at = [], 0
        for m in cuts:
            plan = DeltaPlanner(4, True).plan([at], [m])
            dev = on_device(plan)
            s = slice(at, at + m)
            qkv = torch.cat([q[s].reshape(m, -1), k[s].reshape(m, -1), v[s].reshape(m, -1)], dim=1)
            rows.append(ops.delta_rule(f32(qkv), f32(b[s]), f32(z[s]), dt_bias=torch.zeros(d, device=DEV), a_log=torch.zeros(1, device=DEV),
                                       row_offsets=i32([0, m]), state_slots=i32([0]), state=state, kv_heads=1, heads=1, d=d, dv=dv,
                                       num_requests=1, walk_requests=dev["walk"], num_walk=plan.values["num_walk"], chunks=dev["chunks"],
                                       spans=dev["spans"], max_rows=plan.values["walk_rows"]).cpu())
            at += m
        y = torch.cat(rows)
        assert at == n and float(y[:3].abs().max()) < 1e-6
        assert float((y[190] - 4.0).abs().max()) < 0.02 and float((y[439] + 7.0).abs().max()) < 0.05


@pytest.mark.parametrize("T,heads,dv", [(3, 1, 1), (50, 3, 36), (7, 2, 300), (9, 16, 128)])
def test_norm_per_head_with_a_gate(T, heads, dv):
    from sharpinference_b200.kernels import ops
    n = heads * dv
    y, g, w = _rand(T, n, seed=1, scale=4.0), _rand(T, n + 3, seed=2, scale=2.0), _rand(dv, seed=3)
    got = ops.head_norm_gate(f32(y), f32(g)[:, 2: 2 + n], f32(w), 1e-4, heads, torch.float32)
    close(got, plain.rms(y.view(T, heads, dv), w, 1e-4).reshape(T, n) * torch.sigmoid(g[:, 2: 2 + n]), 2e-6)


# ------------------------------------------------------------------------------------------
# one layer at a time, through the engine
# ------------------------------------------------------------------------------------------
@pytest.mark.parametrize("name,index", [(n, i) for n in sorted(CASES) for i in range(len(CASES[n][0]["layers"]))])
def test_each_layer_alone(tmp_path, name, index):
    """A model of one layer (a borrowing one behind its lender): the residual stream behind every layer against the plain
    model's; a prompt in one step, then the same prompt with its last 40 tokens one by one."""
    from sufopel_models import one_layer, write_config
    from sharpinference_b200 import StepEntry
    _, std, seed = CASES[name]
    n = min(150, CASES[name][0]["max_positions"])
    for variant, mlp in (("bare", None), ("own", "same")):
        cfg = one_layer(name, index, mlp)
        if variant == "own" and cfg["layers"][-1]["mlp"] is None:
            continue
        folder = write_config(cfg, std, seed + index, str(tmp_path / variant))
        cfg, w = plain.load_folder(folder)
        toks = traces.random_tokens(cfg["vocab"], n, seed=index)
        after = []
        plain.forward(cfg, w, toks, layers_out=after)
        eng = engine_for(folder, "float32", 256)
        eng.runner.trace_streams = True
        eng.open_request("a")
        eng.forward_step([StepEntry("a", toks, [])])
        for got, want in zip(eng.runner.last_layer_streams, after):
            assert float((got.double().cpu() - want).abs().max()) < 3e-5 * float(want.abs().max()), (variant, "prompt")
        eng.close_request("a")
        eng.open_request("b")
        eng.forward_step([StepEntry("b", toks[: n - 40], [])])
        for t in range(n - 40, n):
            eng.forward_step([StepEntry("b", [toks[t]], [])])
            got, want = eng.runner.last_layer_streams[-1].double().cpu(), after[-1]
            assert float((got[0] - want[t]).abs().max()) < 3e-5 * float(want.abs().max()), (variant, "decoded", t)
        eng.close_request("b")


# ------------------------------------------------------------------------------------------
# whole models through the engine
# ------------------------------------------------------------------------------------------
@pytest.mark.parametrize("name", sorted(CASES))
def test_layers_one_after_the_other(folders, name):
    """The residual stream behind every layer of a whole model against the plain model's."""
    from sharpinference_b200 import StepEntry
    cfg, w = plain.load_folder(folders[name])
    toks = traces.random_tokens(cfg["vocab"], 120, seed=8)
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
    """Portions shorter and longer than the convolutions' memory, at and around the size from which the delta rule works in
    chunks, and across chunk and page borders."""
    run_and_compare(folders[name], name, dtype, traces.portions(requests_for(name)), expected)
    run_and_compare(folders[name], name, dtype, traces.portions(requests_for(name), sizes=(2, 17, 3, 64, 1, 32, 2, 49, 33, 2)),
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


def test_a_first_token_is_remembered_for_hundreds(tmp_path):
    """Slow channels keep what they saw: in a model of delta layers alone, exchanging a request's first token moves the plain logits
    200 tokens later by many tolerances, and the engine's logits there are right, in a prompt's portion and decoded."""
    from sufopel_models import delta, dense, top, write_config
    from safetensors.torch import load_file, save_file
    cfg = top(60, 48, 400, 1e-5, (1.0, 1.0), 4, [delta(2, 1, 32, 24, 4, (4, 6), dense(32)), delta(3, 3, 24, 16, 3, (8, 4), None)])
    folder = write_config(cfg, 0.2, 11, str(tmp_path))
    path = os.path.join(folder, "model.safetensors")
    t = load_file(path)
    for key in t:
        if key.endswith(".dt_bias"):
            t[key] = torch.full_like(t[key], -9.0)
        if key.endswith(".mix.b"):
            t[key] = t[key] * 0.0                                     # every step is 1/2
    save_file(t, path)
    cfg, w = plain.load_folder(folder)
    toks = traces.random_tokens(cfg["vocab"], 230, seed=21)
    want = plain.forward(cfg, w, toks)
    other = plain.forward(cfg, w, [(toks[0] + 7) % cfg["vocab"]] + toks[1:])
    moved = (other - want).abs().max(-1).values / float(want.abs().max())
    assert float(moved[200:].max()) > 20 * TOL["float32"]
    eng = engine_for(folder, "float32", 256)
    got = traces.replay(eng, traces.tail_decode({"r": toks}, tail=15))
    assert traces.worst_error(got, {"r": want})[0] < TOL["float32"]


def _aim(w, cfg, layer, marked, asking):
    """Edit a lending (``layer`` 0) or borrowing (1) latent layer so that the query of token ``asking`` meets the key of token
    ``marked`` with a score far above every other: rank-one terms along what sets the tokens' normed embeddings apart."""
    m, p = cfg["layers"][layer]["mixer"], f"l{layer}.mix."
    eps = cfg["norm"]["eps"]
    h = plain.rms(w["embed"] * cfg["embedding"]["scale"], w["l0.norm1"], eps)
    if layer == 0:
        vk = h[marked] - h.mean(0)
        w["l0.mix.dkv"][0] += 30.0 * vk / (vk @ vk)                  # the latent's element 0 stands for the marked token
    vq = h[asking] - h.mean(0)
    w[p + "dq"][0] += 30.0 * vq / (vq @ vq)
    for hd in range(m["heads"]):
        w[p + "uk"][hd * m["dim"]] = 0.0
        w[p + "uk"][hd * m["dim"], 0] = 6.0
        w[p + "uq"][hd * m["dim"]] = 0.0
        w[p + "uq"][hd * m["dim"], 0] = 6.0
    return w


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_a_far_key_among_hundreds_carries_the_output(tmp_path, dtype):
    """The last token's query meets the key of one early token with a score far above all others: 400 positions back and across
    six pages, at both sides of a page's border, in a prompt's last row and in a decoded token; in a layer with a latent of its
    own and in the one that borrows it.  Exchanging that early token then changes the logits at the end by a visible part of
    their size."""
    from sufopel_models import latent, top, write_config
    from safetensors.torch import save_file
    from sharpinference_b200 import StepEntry
    cfg = top(40, 32, 512, 1e-5, (1.0, 1.0), 4, [latent(2, 16, 16, 16, 24, 1.5, None), latent(2, 16, 16, 16, 24, 1.5, None, kv_from=0)])
    folder = write_config(cfg, 0.3, 5, str(tmp_path / "base"))
    n = 403
    for layer in (0, 1):
        cfg, w = plain.load_folder(folder)
        w["pos"] *= 0.02                                             # positions hardly move the latents
        w["l0.ls1"] *= 1.0 if layer == 0 else 0.05                   # what the second layer reads is then the embedding
        w["side.embed"][:, :4] *= 1.0 if layer == 0 else 0.0
        w = _aim(w, cfg, 0, 37, 39)
        if layer == 1:
            w = _aim(w, cfg, 1, 37, 39)
            w["l1.norm1"] = w["l0.norm1"].clone()
        variant = str(tmp_path / f"aimed{layer}")
        os.makedirs(variant)
        save_file({k: v.to(torch.bfloat16).contiguous() for k, v in w.items()}, os.path.join(variant, "model.safetensors"))
        with open(os.path.join(variant, "config.json"), "w") as fh:
            json.dump(cfg, fh)
        cfg, w = plain.load_folder(variant)
        eng = engine_for(variant, dtype, 512)
        for place in (0, 2, 63, 64, 320):
            toks = [t % 30 for t in traces.random_tokens(30, n, seed=3)]
            toks[place], toks[-2], toks[-1] = 37, 39, 39              # the asking token as a prompt's last row and decoded
            want = plain.forward(cfg, w, toks)
            other = plain.forward(cfg, w, toks[:place] + [5] + toks[place + 1:])
            for row in (n - 2, n - 1):
                assert float((want[row] - other[row]).abs().max()) / float(want.abs().max()) > 0.08, (layer, place)
            slack = (plain.forward(cfg, w, toks, round_to=torch.bfloat16) - want).abs().max(-1).values
            for entry, row in ((StepEntry("a", toks[:-1], [n - 2]), n - 2), (StepEntry("a", toks[-1:], [0]), n - 1)):
                if row == n - 2:
                    eng.open_request("a")
                lg = eng.forward_step([entry]).double().cpu()
                allowed = TOL[dtype] * float(want.abs().max())
                if dtype == "bfloat16":
                    allowed = max(allowed, 3.0 * float(slack[row]))
                assert float((lg[0] - want[row]).abs().max()) < allowed, (layer, place, row)
            eng.close_request("a")


@pytest.mark.parametrize("seed", [3, 14, 15, 92, 65, 35])
def test_drawn_configurations(tmp_path, seed):
    """Configurations drawn at random with requests of 2 to 700 tokens: whole, with decoded tails, and in drawn mixed batches,
    in 32-bit; bfloat16 whole, held to what rounding does."""
    from sufopel_models import drawn_config, write_config
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


def test_positions_end_where_the_table_ends(folders):
    """A prompt longer than the position table is refused, a step beyond it too (before anything runs), and generation stops with
    ``length`` when the last position has been used."""
    from sharpinference_b200 import Engine, EngineOptions, SamplingParams, StepEntry
    from sharpinference_b200.engine.step import StepError
    cfg, w = plain.load_folder(folders["D"])
    P = cfg["max_positions"]
    eng = Engine(folders["D"], dtype="float32", device=DEV, options=EngineOptions(max_cache_tokens=512, max_batch=2))
    with pytest.raises(ValueError, match="positions"):
        eng.add_request([1] * (P + 1))
    eng.open_request("x")
    eng.forward_step([StepEntry("x", [1] * (P - 1), [])])
    with pytest.raises(StepError, match="positions"):
        eng.forward_step([StepEntry("x", [1, 2], [1])])
    toks = [1] * (P - 1) + [2]
    lg = eng.forward_step([StepEntry("x", [2], [0])]).double().cpu()[0]
    want = plain.forward(cfg, w, toks)
    assert float((lg - want[-1]).abs().max()) < TOL["float32"] * float(want.abs().max())
    eng.close_request("x")
    prompt = traces.random_tokens(cfg["vocab"], P - 3, seed=1)
    out = eng.generate([prompt, prompt[:4]], SamplingParams(temperature=0.0, max_new_tokens=9))
    assert out[0] == plain.generate_greedy(cfg, w, prompt, 4) and len(out[1]) == 9


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
    """``sharpi-cli`` generates greedily on a Sufopel folder, and ``bin/trace_run`` as a child process replays a mixed schedule
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
    assert {"channel_delta", "latent_attention"} <= set(part_kinds("mixer")) and "sandwich" in part_kinds("block")
    assert "moe_sigmoid_groups" in part_kinds("feed_forward")
