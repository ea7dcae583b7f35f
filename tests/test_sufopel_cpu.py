"""Sufopel without a GPU: the configuration reader, the tensor declaration, the schedule, the pages and state that the cache
manager hands to the layers, the step planner of the delta rule, how weights are laid together, the limit on positions, and
the plain implementation checked against each mechanism's defining property."""
import copy
import math

import pytest
import torch

import plain_sufopel as plain
import traces
from sufopel_models import CASE_A, CASE_B, CASE_C, CASE_D, CASE_E, CASES, drawn_config, write

from sharpinference_b200.config import ConfigError, SufopelConfig
from sharpinference_b200.registry import get_architecture, resolve
from sharpinference_b200.weights.loading import declared_tensors

F64 = torch.float64


def _rand(*shape, seed=0, scale=1.0):
    return scale * torch.randn(*shape, generator=torch.Generator().manual_seed(seed), dtype=F64)


# -- configuration -------------------------------------------------------------------------
@pytest.mark.parametrize("case", [CASE_A, CASE_B, CASE_C, CASE_D, CASE_E, drawn_config(3), drawn_config(4)])
def test_config_round_trip(case):
    arch, cfg = resolve(copy.deepcopy(case), "test")
    assert arch.name == "Sufopel" and isinstance(cfg, SufopelConfig)
    assert SufopelConfig.from_dict(cfg.to_dict()) == cfg
    assert cfg.to_dict() == case
    for got, raw in zip(cfg.layers, case["layers"]):
        assert got.mixer.type == raw["type"] and (got.mlp is None) == (raw["mlp"] is None)


def test_defaults_of_absent_keys():
    case = copy.deepcopy(CASE_A)
    del case["embedding"], case["logit_scale"], case["token_side"]
    m = case["layers"][0]["mixer"]
    for key in ("kv_heads", "vdim", "conv", "a_rank", "g_rank"):
        del m[key]
    m = case["layers"][1]["mixer"]
    for key in ("vdim", "scale"):
        del m[key]
    del case["layers"][1]["mlp"]["router"]["groups"]
    _, cfg = resolve(case, "test")
    a, b = cfg.layers[0].mixer, cfg.layers[1].mixer
    assert (a.kv_heads, a.vdim, a.conv, a.a_rank, a.g_rank) == (4, 16, 1, 0, 0)
    assert b.vdim == 16 and b.scale == pytest.approx(0.25) and b.kv_from is None
    assert (cfg.layers[1].mlp.groups, cfg.layers[1].mlp.keep) == (1, 1)
    assert (cfg.embedding_scale, cfg.logit_scale, cfg.side_dim) == (1.0, 1.0, 0)


def test_config_problems_are_listed_together():
    bad = copy.deepcopy(CASE_A)
    del bad["width"]
    bad["layers"][0]["mixer"]["kv_heads"] = 3                      # 4 heads are no multiple of 3
    bad["layers"][1]["mlp"]["router"]["groups"]["count"] = 3       # eight experts in three groups
    bad["layers"][1]["mixer"]["kv_rank"] = 0
    bad["layers"][4]["mlp"]["router"]["top"] = 7
    bad["layers"].append({"type": "serial", "mixer": {}, "mlp": None})
    with pytest.raises(ConfigError) as err:
        resolve(bad, "test")
    text = str(err.value)
    for piece in ("width", "kv_heads", "groups.count", "kv_rank", "top", "serial"):
        assert piece in text, (piece, text)


@pytest.mark.parametrize("source", [0, 3, 4, 9, -1])
def test_a_borrowing_layer_needs_an_earlier_lender_with_the_same_latent_size(source):
    bad = copy.deepcopy(CASE_A)
    bad["layers"][3]["mixer"]["kv_from"] = source                  # a delta layer, itself, a later one, nowhere
    with pytest.raises(ConfigError, match="kv_from"):
        resolve(bad, "test")
    bad["layers"][3]["mixer"].update(kv_from=1, kv_rank=32)
    with pytest.raises(ConfigError, match="kv_from"):
        resolve(bad, "test")


def test_declared_tensors_follow_the_configuration():
    arch = get_architecture("Sufopel")
    _, cfg = resolve(copy.deepcopy(CASE_A), "test")
    decls = {d.name: d.shape for d in declared_tensors(arch, cfg)}
    assert decls["embed"] == (97, 64) and decls["head"] == (97, 64) and decls["pos"] == (420, 64)
    assert decls["side.embed"] == (97, 5 * 12) and decls["l3.side.gate"] == (12, 64) and decls["l3.side.proj"] == (64, 12)
    assert decls["l0.mix.q"] == (32, 64) and decls["l0.mix.k"] == (32, 64) and decls["l0.mix.v"] == (96, 64)
    assert decls["l0.mix.k.conv"] == (32, 3) and decls["l0.mix.v.conv"] == (96, 3) and decls["l0.mix.b"] == (4, 64)
    assert decls["l0.mix.a1"] == (8, 64) and decls["l0.mix.a2"] == (64, 8) and decls["l0.mix.dt_bias"] == (64,)
    assert decls["l0.mix.g1"] == (12, 64) and decls["l0.mix.g2"] == (96, 12) and decls["l0.mix.norm"] == (24,)
    assert decls["l1.mix.dkv"] == (40, 64) and decls["l1.mix.uk"] == (64, 40) and decls["l1.mix.uv"] == (96, 40)
    assert decls["l1.mix.g"] == (96, 64) and decls["l1.mix.o"] == (64, 96)
    assert "l3.mix.dkv" not in decls and "l3.mix.dkv.norm" not in decls and decls["l3.mix.uk"] == (48, 40)
    assert "l2.norm2" not in decls and "l2.ls2" not in decls and decls["l2.norm1b"] == (64,)     # no feed-forward
    assert decls["l1.mlp.correction"] == (8,) and decls["l1.mlp.e7.down"] == (64, 24) and "l1.mlp.e8.down" not in decls


def test_low_rank_sizes_come_from_the_folder(tmp_path):
    """The configuration of a folder need not give them; and one that keeps the vectors of an absent feed-forward loads."""
    import json
    import os

    from safetensors.torch import load_file, save_file

    from sharpinference_b200.weights import FileWeights
    folder = write("A", str(tmp_path))
    with open(os.path.join(folder, "config.json")) as fh:
        raw = json.load(fh)
    for layer in raw["layers"]:
        layer["mixer"].pop("a_rank", None)
        layer["mixer"].pop("g_rank", None)
    path = os.path.join(folder, "model.safetensors")
    tensors = load_file(path)
    tensors.update({"l2.norm2": torch.ones(64), "l2.norm2b": torch.ones(64), "l2.ls2": torch.ones(64)})
    save_file(tensors, path)
    arch, cfg = resolve(raw, "test")
    source = FileWeights(folder, torch.float32, "cpu")
    decls = declared_tensors(arch, cfg, torch.float32, stored_names={n: tuple(e.shape) for n, e in source.entries.items()})
    source.check(decls)
    model = arch.build(cfg, source)
    assert model.blocks[0].mixer.low == 24 and model.blocks[4].mixer.low == 24            # 8 + 12 and 4 + 20, padded


def test_schedule_pages_and_state_in_the_cache_manager():
    """One page group per latent size; a borrowing entry sees its lender's pages and writes none; a delta layer has state and no
    pages, without a convolution's when it has one tap."""
    from sharpinference_b200.cache import CacheManager
    from sharpinference_b200.weights.source import DeclaringWeights
    arch = get_architecture("Sufopel")
    _, cfg = resolve(copy.deepcopy(CASE_C), "test")
    model = arch.build(cfg, DeclaringWeights(torch.float32))
    assert [(e.layer, e.cache_from) for e in model.schedule] == [(0, None), (1, None), (2, None), (3, None), (4, 1), (5, None)]
    assert model.max_positions == 512
    cache = CacheManager(model.schedule, model.blocks, page_size=4, num_pages=8, max_requests=3, dtype=torch.float32, device="cpu",
                         model_state_specs=model.state_specs)
    slots = cache.layer_slots()
    assert [g.spec.head_dim for g in cache.groups] == [256, 128] and all(g.spec.planes == 1 for g in cache.groups)
    assert slots[4].kv.data_ptr() == slots[1].kv.data_ptr() and slots[1].writes_cache and not slots[4].writes_cache
    assert slots[1].kv.shape == (8, 1, 1, 4, 256) and slots[3].group != slots[1].group
    assert slots[0].kv is None and slots[0].states["S"].shape == (3, 2 * 64 * 128)
    assert slots[0].states["conv"].shape == (3, 3 * (2 * 128 + 2 * 64))
    _, cfg = resolve(copy.deepcopy(CASE_B), "test")
    model = arch.build(cfg, DeclaringWeights(torch.float32))
    assert "conv" not in model.blocks[1].mixer.state_specs and "conv" in model.blocks[0].mixer.state_specs
    assert model.blocks[0].mixer.state_specs["S"].shape == (3 * 7 * 8,)                   # columns of 5 padded to 8


def test_planner_cuts_tiles_and_chunks():
    from sharpinference_b200.parts import DeltaPlanner
    p = DeltaPlanner(4, True)
    p.WALK_ROWS_UP_TO = 16
    d = p.plan([0, 5, 9, 0], [1, 40, 16, 17])
    assert d.arrays["walk"].tolist() == [0, 2] and d.values == {"num_walk": 2, "walk_rows": 16}
    assert d.arrays["chunks"].tolist() == [[1, 16, 1, 0], [17, 16, 1, 0], [33, 8, 1, 0], [57, 16, 3, 0], [73, 1, 3, 0]]
    assert d.arrays["spans"].tolist() == [[1, 0, 3, 0], [3, 3, 2, 0]]
    tiles = d.arrays["tiles"].tolist()
    assert tiles[0] == [0, 1, 0, 0] and tiles[1] == [1, 8, 1, 0] and tiles[-1] == [73, 1, 3, 0] and sum(t[1] for t in tiles) == 74
    d = p.plan([4, 5], [1, 1])                                  # nothing to list when every request is a piece and walked
    assert all(a.size == 0 for a in d.arrays.values()) and d.values["num_walk"] == 2
    long = DeltaPlanner(30, False)                              # a tile is never shorter than what a convolution looks back
    d = long.plan([0], [70])
    assert d.arrays["tiles"].tolist() == [[0, 29, 0, 0], [29, 29, 0, 0], [58, 12, 0, 0]] and d.values == {"num_walk": 1, "walk_rows": 70}
    assert long.key != p.key


def test_low_rank_maps_in_one_product(tmp_path):
    """The product that reads both low-rank parts side by side gives the two products; the norm behind a sublayer carries the
    layer's factor."""
    from sharpinference_b200.weights import FileWeights
    folder = write("A", str(tmp_path))
    cfg, w = plain.load_folder(folder)
    arch, typed = resolve(cfg, "test")
    model = arch.build(typed, FileWeights(folder, torch.float32, "cpu"))
    mixer, W = model.blocks[0].mixer, w["l0.mix.a1"].shape[1]
    h = _rand(5, W, seed=1)
    proj = h @ mixer.proj.weight.double().T
    low = proj[:, 32 + 32 + 96: 32 + 32 + 96 + mixer.low]
    z = low @ mixer.up.weight.double().T
    assert torch.allclose(z[:, :64], h @ w["l0.mix.a1"].T @ w["l0.mix.a2"].T, atol=1e-9)
    assert torch.allclose(z[:, 64:], h @ w["l0.mix.g1"].T @ w["l0.mix.g2"].T, atol=1e-9)
    assert torch.allclose(proj[:, 160 + mixer.low: 164 + mixer.low], h @ w["l0.mix.b"].T, atol=1e-9)
    assert torch.allclose(model.blocks[1].ffn_weight.double(), w["l1.norm2b"] * w["l1.ls2"], rtol=1e-6)


def test_requests_end_at_the_last_position():
    """A scheduler with a limit: a request that has filled the positions ends with ``length`` although it may go on generating;
    its last token is sampled and never run."""
    from sharpinference_b200 import SamplingParams
    from sharpinference_b200.cache import CacheManager
    from sharpinference_b200.engine.scheduler import Request, Scheduler
    from sharpinference_b200.weights.source import DeclaringWeights
    arch = get_architecture("Sufopel")
    _, cfg = resolve(copy.deepcopy(CASE_A), "test")
    model = arch.build(cfg, DeclaringWeights(torch.float32))
    cache = CacheManager(model.schedule, model.blocks, page_size=4, num_pages=16, max_requests=2, dtype=torch.float32, device="cpu",
                         allocate=False)
    s = Scheduler(cache, max_batch=2, max_tokens_per_step=8, max_positions=10)
    req = Request("a", [1] * 7, SamplingParams(max_new_tokens=50))
    s.add(req)
    run = 0
    while s.has_work:
        plan = s.plan()
        cache.reserve([(e.request.request_id, e.count) for e in plan.entries])
        for e in plan.entries:
            run = max(run, e.start + e.count)
            cache.commit(e.request.request_id, e.count)
        s.complete(plan, [3] * sum(e.want_last for e in plan.entries))
    assert req.finish_reason == "length" and len(req.generated) == 4 and run == 10


# -- the plain implementation --------------------------------------------------------------
def test_plain_delta_rule_is_a_corrected_memory():
    """With decay 1 and step 1 a key reads back the value it was last given; a channel with decay 0 holds nothing older; the
    state may be handed on anywhere."""
    k = plain.unit(_rand(1, 1, 6, seed=1)).expand(3, 1, 6)
    v = _rand(3, 1, 4, seed=2)
    one = torch.ones(3, 1, 6, dtype=F64)
    o, S = plain.delta_rule(k, k, v, one, torch.ones(3, 1, dtype=F64))
    norm2 = (k[0, 0] @ k[0, 0])
    for t in range(3):
        assert torch.allclose(o[t, 0], v[t, 0] * norm2, atol=1e-5)               # the old value is gone, not added to
    g = torch.ones(2, 1, 6, dtype=F64)
    g[:, :, 2] = 0.0
    q = torch.zeros(2, 1, 6, dtype=F64)
    q[:, :, 2] = 1.0
    o, _ = plain.delta_rule(q, plain.unit(_rand(2, 1, 6, seed=3)), _rand(2, 1, 4, seed=4), g, torch.zeros(2, 1, dtype=F64),
                            state=_rand(1, 6, 4, seed=5))
    assert float(o.abs().max()) == 0.0
    q, k, v = _rand(20, 2, 5, seed=6), plain.unit(_rand(20, 2, 5, seed=7)), _rand(20, 2, 3, seed=8)
    g, b = torch.sigmoid(_rand(20, 2, 5, seed=9)), torch.sigmoid(_rand(20, 2, seed=10))
    o, S = plain.delta_rule(q, k, v, g, b)
    o1, S1 = plain.delta_rule(q[:8], k[:8], v[:8], g[:8], b[:8])
    o2, S2 = plain.delta_rule(q[8:], k[8:], v[8:], g[8:], b[8:], state=S1)
    assert torch.allclose(torch.cat([o1, o2]), o, atol=1e-12) and torch.allclose(S2, S, atol=1e-12)


def test_plain_delta_rule_in_chunks():
    """The closed form over a chunk (a triangular system and two products with the state before it) gives the rows one by
    one."""
    n, d, dv = 9, 5, 4
    q, k, v = _rand(n, 1, d, seed=1), plain.unit(_rand(n, 1, d, seed=2)), _rand(n, 1, dv, seed=3)
    g, b = torch.sigmoid(_rand(n, 1, d, seed=4)), torch.sigmoid(_rand(n, 1, seed=5))
    S0 = _rand(1, d, dv, seed=6)
    want, S = plain.delta_rule(q, k, v, g, b, state=S0)
    P = lambda s, t: torch.stack([torch.ones(d, dtype=F64)] + [g[r, 0] for r in range(s + 1, t + 1)]).prod(0)
    A = torch.tensor([[float((k[t, 0] * P(s, t) * k[s, 0]).sum()) if s < t else 0.0 for s in range(n)] for t in range(n)], dtype=F64)
    B = torch.tensor([[float((q[t, 0] * P(s, t) * k[s, 0]).sum()) if s <= t else 0.0 for s in range(n)] for t in range(n)], dtype=F64)
    D = torch.stack([P(-1, t) for t in range(n)])
    solve = torch.linalg.inv(torch.eye(n, dtype=F64) + b * A) * b.T
    U = solve @ v[:, 0] - solve @ (D * k[:, 0]) @ S0[0]
    o = B @ U + (D * q[:, 0]) @ S0[0]
    last = D[-1].view(d, 1) * S0[0] + torch.stack([P(s, n - 1) * k[s, 0] for s in range(n)]).T @ U
    assert torch.allclose(o, want[:, 0], atol=1e-12) and torch.allclose(last, S[0], atol=1e-12)


def test_plain_convolution_decay_and_heads():
    u, w = _rand(7, 3, seed=1), _rand(3, 4, seed=2)
    y = plain.causal_conv(u, w)
    want = torch.nn.functional.conv1d(torch.nn.functional.pad(u.T[None], (3, 0)), w[:, None], groups=3)[0].T
    assert torch.allclose(y, want, atol=1e-12) and torch.allclose(y[0], u[0] * w[:, 3], atol=1e-12)
    m = {"heads": 4, "kv_heads": 2, "dim": 3, "vdim": 2}
    t = {"a1": _rand(5, 6, seed=3), "a2": _rand(12, 5, seed=4), "dt_bias": _rand(12, seed=5), "A_log": _rand(4, seed=6), "b": _rand(4, 6, seed=7)}
    h = _rand(8, 6, seed=8)
    g = plain.channel_decay(h, m, t, "")
    z = h @ t["a1"].T @ t["a2"].T + t["dt_bias"]
    assert float(g[3, 2, 1]) == pytest.approx(math.exp(-math.exp(float(t["A_log"][2])) * math.log1p(math.exp(float(z[3, 2 * 3 + 1])))))
    for s, n in (("q", 6), ("k", 6), ("v", 8)):
        t[s], t[s + ".conv"] = _rand(n, 6, seed=ord(s)), _rand(n, 2, seed=ord(s) + 1)
    q, k, v, g, b = plain.delta_inputs(h, m, t, "")
    assert torch.equal(q[:, 0], q[:, 1]) and torch.equal(k[:, 2], k[:, 3]) and not torch.equal(q[:, 1], q[:, 2])
    assert torch.allclose(k.norm(dim=-1), torch.ones(8, 4, dtype=F64), atol=1e-3)
    assert torch.allclose(q.norm(dim=-1), torch.full((8, 4), 3 ** -0.5, dtype=F64), atol=1e-3)


def test_plain_router_groups_sum_two_choice_scores():
    """A group wins by its two best together, not by its best; a kept group's expert with a negative choice score is chosen before
    any expert of a group that is not kept; the weights come from the scores without the correction, as they are."""
    router = {"experts": 6, "top": 2, "groups": {"count": 2, "keep": 1}}
    choice = torch.tensor([[0.9, -0.8, -0.9, 0.3, 0.2, -0.7]], dtype=F64)
    assert plain.group_scores(choice, 2).tolist() == [[pytest.approx(0.1), pytest.approx(0.5)]]
    assert plain.choose(choice, router).tolist() == [[3, 4]]
    router["top"] = 3
    assert plain.choose(choice, router).tolist() == [[3, 4, 5]]
    assert plain.group_scores(choice, 6).tolist() == [choice[0].tolist()]
    W = 5
    h = _rand(4, W, seed=1)
    t = {"router": _rand(6, W, seed=2), "correction": _rand(6, seed=3)}
    for e in range(6):
        t.update({f"e{e}.gate": _rand(3, W, seed=10 + e), f"e{e}.up": _rand(3, W, seed=20 + e), f"e{e}.down": _rand(W, 3, seed=30 + e)})
    out, idx, c = plain.mixture(h, {"router": router, "expert": {"limit": 0.5}}, t, "")
    s = torch.sigmoid(h @ t["router"].T)
    assert torch.allclose(c, s + t["correction"])
    for n in range(4):
        want = sum(s[n, e] * plain.expert(h[n:n + 1], t, f"e{int(e)}.", 0.5)[0] for e in idx[n])
        assert torch.allclose(out[n], want, atol=1e-12)


def test_plain_expert_clamps_and_gelu():
    W = 3
    t = {"gate": torch.eye(W, dtype=F64), "up": torch.eye(W, dtype=F64) * 2, "down": torch.eye(W, dtype=F64)}
    h = torch.tensor([[-9.0, 0.3, 9.0]], dtype=F64)
    y = plain.expert(h, t, "", 1.5)[0]
    sig = lambda z: 1 / (1 + math.exp(-z))
    assert float(y[0]) == pytest.approx(-9.0 * sig(1.702 * -9.0) * (-1.5 + 1))      # the gate has no lower limit
    assert float(y[1]) == pytest.approx(0.3 * sig(1.702 * 0.3) * 1.6)
    assert float(y[2]) == pytest.approx(1.5 * sig(1.702 * 1.5) * 2.5)
    z = _rand(50, seed=1, scale=3.0)
    assert torch.allclose(plain.gelu_tanh(z), torch.nn.functional.gelu(z, approximate="tanh"), atol=1e-12)


def test_plain_token_side_reads_its_layers_slice():
    cfg = {"token_side": {"dim": 3}, "norm": {"eps": 1e-5}}
    t = {"side.embed": _rand(7, 9, seed=1), "l2.side.gate": _rand(3, 5, seed=2), "l2.side.proj": _rand(5, 3, seed=3), "l2.side.norm": _rand(5, seed=4)}
    x = _rand(2, 5, seed=5)
    y = plain.token_side(x, [4, 0], 2, cfg, t)
    for i, tok in enumerate((4, 0)):
        g = plain.gelu_tanh(t["l2.side.gate"] @ x[i]) * t["side.embed"][tok, 6:9]
        p = t["l2.side.proj"] @ g
        assert torch.allclose(y[i], p / torch.sqrt((p * p).mean() + 1e-5) * t["l2.side.norm"], atol=1e-12)


@pytest.mark.parametrize("name", sorted(CASES))
def test_random_folder_loads_and_runs_plain(tmp_path, name):
    folder = write(name, str(tmp_path))
    cfg, w = plain.load_folder(folder)
    toks = traces.random_tokens(cfg["vocab"], 40, seed=1)
    layers = []
    logits = plain.forward(cfg, w, toks, layers_out=layers)
    assert logits.shape == (40, cfg["vocab"]) and len(layers) == len(cfg["layers"]) and bool(torch.isfinite(logits).all())
    assert torch.allclose(plain.forward(cfg, w, toks[:17]), logits[:17], atol=1e-9)       # causal


def test_every_constant_and_tensor_shows_in_the_plain_logits(tmp_path):
    """The comparison with the plain model is sharp: every constant and every tensor moves the plain logits by far more than the
    tolerance when it is changed or dropped."""
    folder = write("A", str(tmp_path))
    cfg, w = plain.load_folder(folder)
    toks = traces.random_tokens(cfg["vocab"], 90, seed=2)
    right = plain.forward(cfg, w, toks)
    scale = float(right.abs().max())

    def moved(edit=None, other_w=None):
        c = copy.deepcopy(cfg)
        if edit:
            edit(c)
        return float((plain.forward(c, other_w or w, toks) - right).abs().max()) / scale

    mix = lambda c, i: c["layers"][i]["mixer"]
    assert moved(lambda c: c["embedding"].update(scale=1.0)) > 1e-2
    assert moved(lambda c: c.update(logit_scale=0.5)) > 1e-2
    assert moved(lambda c: c["norm"].update(eps=1e-2)) > 1e-3
    assert moved(lambda c: mix(c, 1).update(scale=0.45)) > 1e-3
    assert moved(lambda c: mix(c, 3).update(scale=0.45)) > 1e-3
    router = lambda c: c["layers"][1]["mlp"]["router"]
    assert moved(lambda c: router(c).pop("groups")) > 1e-3
    assert moved(lambda c: router(c)["groups"].update(keep=3)) > 1e-3
    assert moved(lambda c: router(c).update(top=2)) > 1e-3
    assert moved(lambda c: c["layers"][1]["mlp"]["expert"].update(limit=2.0)) > 1e-3
    for name in sorted(w):
        if w[name].dim() == 2 and (".mlp.e" in name):
            continue                                                             # any single expert may be idle
        w2 = dict(w)
        w2[name] = torch.zeros_like(w[name])
        assert moved(None, w2) > 1e-3, name
    w2 = dict(w)                                        # the oldest tap alone
    w2["l0.mix.q.conv"] = w["l0.mix.q.conv"].clone()
    w2["l0.mix.q.conv"][:, 0] = 0
    assert moved(None, w2) > 1e-3
