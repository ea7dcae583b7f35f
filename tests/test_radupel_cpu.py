"""Radupel without a GPU: the configuration reader, the tensor declaration, the schedule, the pages and state that the
cache manager hands to the layers, the step planner of the linear attention, how weights are laid side by side, and the
plain implementation checked against each mechanism's defining property."""
import copy
import math

import pytest
import torch

import plain_radupel as plain
import traces
from radupel_models import CASE_A, CASE_B, CASE_C, CASE_D, CASE_E, CASES, write

from sharpinference_b200.config import ConfigError, RadupelConfig
from sharpinference_b200.registry import get_architecture, resolve
from sharpinference_b200.weights.loading import declared_tensors

F64 = torch.float64


def _rand(*shape, seed=0, scale=1.0):
    return scale * torch.randn(*shape, generator=torch.Generator().manual_seed(seed), dtype=F64)


# -- configuration -------------------------------------------------------------------------
@pytest.mark.parametrize("case", [CASE_A, CASE_B, CASE_C, CASE_D, CASE_E])
def test_config_round_trip(case):
    arch, cfg = resolve(copy.deepcopy(case), "test")
    assert arch.name == "Radupel" and isinstance(cfg, RadupelConfig)
    assert RadupelConfig.from_dict(cfg.to_dict()) == cfg
    assert cfg.to_dict() == case
    assert cfg.layer_runs() == plain.layer_order(case)
    for got, raw in zip(cfg.layers, case["layers"]):
        assert (got.mlp is None) == (raw["mlp"] is None)
        assert got.right.decay == tuple(raw["mixer"]["right"]["decay"])


def test_layer_runs():
    runs = resolve(copy.deepcopy(CASE_A), "test")[1].layer_runs()
    assert runs == [(0, False), (1, False), (2, False), (1, True), (2, False), (3, False)]
    assert [i for i, again in resolve(copy.deepcopy(CASE_D), "test")[1].layer_runs() if again] == [0, 0, 0]
    assert not any(again for _, again in resolve(copy.deepcopy(CASE_B), "test")[1].layer_runs())


def test_defaults_of_absent_keys():
    case = copy.deepcopy(CASE_A)
    del case["loop"], case["logit_softcap"]
    m = case["layers"][0]["mixer"]
    for key in ("kv_heads", "vdim", "scale", "conv", "rot"):
        del m["left"][key]
    del m["right"]["vdim"], m["left_scale"], m["right_scale"]
    r = case["layers"][2]["mlp"]["router"]
    for key in ("scale", "identity", "groups"):
        del r[key]
    del case["layers"][2]["mlp"]["shared"]
    _, cfg = resolve(case, "test")
    a = cfg.layers[0]
    assert (a.left.kv_heads, a.left.vdim, a.left.conv, a.left.rot_dims) == (4, 16, 1, 0) and a.left.scale == pytest.approx(0.25)
    assert a.right.vdim == 8 and (a.left_scale, a.right_scale) == (1.0, 1.0)
    mix = cfg.layers[2].mlp
    assert (mix.scale, mix.identity, mix.groups, mix.keep, mix.shared_ff) == (1.0, 0, 1, 1, 0)
    assert cfg.loop_times == 0 and cfg.logit_softcap == 0 and len(cfg.layer_runs()) == 4


def test_config_problems_are_listed_together():
    bad = copy.deepcopy(CASE_A)
    del bad["width"]
    bad["layers"][0]["mixer"]["left"]["kv_heads"] = 3              # 4 heads are no multiple of 3
    bad["layers"][1]["mixer"]["right"]["decay"] = [0.5]            # two heads
    bad["layers"][2]["mlp"]["router"]["groups"]["count"] = 2       # nine experts in two groups
    bad["layers"][3]["mixer"]["left"]["rot"]["dims"] = 18          # beyond the head
    bad["layers"].append({"type": "serial", "mixer": {}, "mlp": None})
    bad["loop"]["stop"] = 9
    with pytest.raises(ConfigError) as err:
        resolve(bad, "test")
    text = str(err.value)
    for piece in ("width", "kv_heads", "decay", "groups.count", "rot.dims", "serial", "stop"):
        assert piece in text, (piece, text)
    bad = copy.deepcopy(CASE_A)
    bad["layers"][2]["mlp"]["router"]["top"] = 7                   # the two kept groups hold six
    with pytest.raises(ConfigError, match="top"):
        resolve(bad, "test")


def test_declared_tensors_follow_the_configuration():
    arch = get_architecture("Radupel")
    _, cfg = resolve(copy.deepcopy(CASE_A), "test")
    decls = {d.name: d.shape for d in declared_tensors(arch, cfg)}
    assert decls["embed"] == (97, 64) and "head" not in decls and decls["final.norm"] == (64,)
    assert decls["l0.mix.left.q"] == (64, 64) and decls["l0.mix.left.k"] == (32, 64) and decls["l0.mix.left.v"] == (48, 64)
    assert decls["l0.mix.left.q.conv"] == (64, 3) and decls["l0.mix.left.v.conv"] == (48, 3)
    assert decls["l0.mix.left.g"] == (4, 64) and decls["l0.mix.left.o"] == (64, 96)
    assert decls["l0.mix.right.q"] == (24, 64) and decls["l0.mix.right.v"] == (36, 64) and decls["l0.mix.right.g"] == (36, 64)
    assert decls["l0.mix.right.norm"] == (36,) and decls["l0.mix.right.o"] == (64, 36)
    assert decls["l0.mlp.gate.b"] == (40,) and decls["l0.mlp.down.b"] == (64,)
    assert "l1.norm2" not in decls and "l1.mlp.gate" not in decls            # no feed-forward, no second norm
    assert decls["l2.mlp.router"] == (9, 64) and decls["l2.mlp.correction"] == (9,)
    assert "l2.mlp.e6.up" in decls and "l2.mlp.e7.up" not in decls           # identity experts have no tensors
    assert decls["l2.mlp.shared.sg"] == (1, 64) and "l2.mlp.e0.gate.b" not in decls


def test_schedule_pages_and_state_in_the_cache_manager():
    """Every pass of a looped layer has pages and state of its own; pages hold the padded head size; the convolution's state
    holds the unpadded channels; a layer with one tap has no such state."""
    from sharpinference_b200.cache import CacheManager
    from sharpinference_b200.weights.source import DeclaringWeights
    arch = get_architecture("Radupel")
    _, cfg = resolve(copy.deepcopy(CASE_A), "test")
    model = arch.build(cfg, DeclaringWeights(torch.float32))
    assert [(e.layer, e.before) for e in model.schedule] == [(0, None), (1, None), (2, None), (1, 0), (2, None), (3, None)]
    cache = CacheManager(model.schedule, model.blocks, page_size=4, num_pages=8, max_requests=3, dtype=torch.float32,
                         device="cpu", model_state_specs=model.state_specs)
    slots = cache.layer_slots()
    assert len({s.kv.data_ptr() for s in slots}) == 6
    assert slots[0].kv.shape[1:] == (2, 2, 4, 32) and slots[1].kv.shape[1:] == (2, 1, 4, 32)
    assert slots[0].states["left.conv"].shape == (3, 2 * (6 * 16 + 2 * 24))
    assert slots[0].states["right.S"].shape == (3, 3 * 8 * 12)
    assert slots[1].states["right.S"].data_ptr() != slots[3].states["right.S"].data_ptr()
    _, cfg = resolve(copy.deepcopy(CASE_B), "test")
    model = arch.build(cfg, DeclaringWeights(torch.float32))
    assert "left.conv" not in model.blocks[2].mixer.state_specs and "left.conv" in model.blocks[1].mixer.state_specs


def test_planner_cuts_long_requests_into_chunks():
    from sharpinference_b200.parts import LightningPlanner
    p = LightningPlanner()
    p.WALK_ROWS_UP_TO = 16
    d = p.plan([0, 5, 9, 0], [1, 130, 16, 17])
    assert d.arrays["walk"].tolist() == [0, 2] and d.values["num_walk"] == 2
    assert d.arrays["chunks"].tolist() == [[1, 64, 1, 0], [65, 64, 1, 0], [129, 2, 1, 0], [147, 17, 3, 0]]
    assert d.arrays["spans"].tolist() == [[1, 0, 3, 0], [3, 3, 1, 0]]
    d = p.plan([4, 5], [1, 1])                                  # nothing to list when every request is walked
    assert d.arrays["walk"].size == 0 and d.arrays["chunks"].size == 0 and d.values["num_walk"] == 2


def test_weights_side_by_side_and_the_bias_as_columns():
    """The joint product of a mixer and a dense feed-forward equals the two products and the bias, in float32 and, for a
    bias that no single bfloat16 number holds, in bfloat16 columns."""
    from sharpinference_b200.parts import DenseSwiGLU, Linear
    from sharpinference_b200.parts.branches import pad_columns, side_by_side
    H, n, ff = 6, 5, 11
    wm, wd, b = _rand(H, n, seed=1), _rand(H, ff, seed=2), _rand(H, seed=3)
    for dtype, tol in ((torch.float32, 1e-6), (torch.bfloat16, 1e-6)):
        ffn = DenseSwiGLU(gate_up=Linear(torch.zeros(2 * ff, H, dtype=dtype)), act_dtype=dtype,
                          down=Linear(wd.to(dtype), bias=b.float()))
        w = ffn.take_out_weight()
        assert w.shape == (H, ffn.out_columns) and w.shape[1] % 8 == 0
        joint = side_by_side([wm.to(dtype), w]).double()
        assert joint.shape[1] == pad_columns(n) + w.shape[1]
        ones = 1 if dtype == torch.float32 else 3
        cols = torch.zeros(4, joint.shape[1], dtype=F64)
        a, act = _rand(4, n, seed=4), _rand(4, ff, seed=5)
        cols[:, :n] = a
        cols[:, pad_columns(n): pad_columns(n) + ff] = act
        cols[:, pad_columns(n) + ff: pad_columns(n) + ff + ones] = 1.0
        want = a @ wm.to(dtype).double().T + act @ wd.to(dtype).double().T + b.float().double()
        assert float((cols @ joint.T - want).abs().max()) < tol


# -- the plain implementation --------------------------------------------------------------
def test_plain_convolution_and_rotation():
    u, w = _rand(7, 3, seed=1), _rand(3, 4, seed=2)
    y = plain.causal_conv(u, w)
    want = torch.nn.functional.conv1d(torch.nn.functional.pad(u.T[None], (3, 0)), w[:, None], groups=3)[0].T
    assert torch.allclose(y, want, atol=1e-12)
    assert torch.allclose(y[0], u[0] * w[:, 3], atol=1e-12)                    # the last tap is the current token's
    v = _rand(9, 2, 6, seed=3)
    r = plain.rotate_halves(v, 4, 50.0)
    assert torch.equal(r[..., 4:], v[..., 4:]) and torch.equal(r[0], v[0])
    c, s = math.cos(5.0), math.sin(5.0)                                        # pair 0 turns by its position
    assert float(r[5, 1, 0]) == pytest.approx(float(v[5, 1, 0]) * c - float(v[5, 1, 2]) * s)
    assert float(r[5, 1, 2]) == pytest.approx(float(v[5, 1, 2]) * c + float(v[5, 1, 0]) * s)
    a, b = _rand(1, 1, 4, seed=4).expand(9, 1, 4), _rand(1, 1, 4, seed=5).expand(9, 1, 4)
    ra, rb = plain.rotate_halves(a, 4, 50.0)[:, 0], plain.rotate_halves(b, 4, 50.0)[:, 0]
    assert float(ra[5] @ rb[2]) == pytest.approx(float(ra[8] @ rb[5]), abs=1e-12)      # the distance alone counts


def test_plain_decayed_sums_are_a_weighted_sum_over_the_past():
    q, k, v = _rand(20, 2, 5, seed=1), _rand(20, 2, 5, seed=2), _rand(20, 2, 3, seed=3)
    decay = [0.8, 0.99]
    o, S = plain.decayed_sums(q, k, v, decay)
    for h in range(2):
        for t in (0, 7, 19):
            want = sum(decay[h] ** (t - j) * float(q[t, h] @ k[j, h]) * v[j, h] for j in range(t + 1))
            assert torch.allclose(o[t, h], want, atol=1e-12)
    o1, S1 = plain.decayed_sums(q[:8], k[:8], v[:8], decay)
    o2, S2 = plain.decayed_sums(q[8:], k[8:], v[8:], decay, state=S1)
    assert torch.allclose(torch.cat([o1, o2]), o, atol=1e-12) and torch.allclose(S2, S, atol=1e-12)


def test_plain_router_groups_with_negative_choice_scores():
    """A kept group's expert with a negative choice score is chosen before any expert of a group that is not kept, and the
    weights come from the scores without the correction."""
    router = {"experts": 4, "identity": 2, "top": 2, "scale": 3.0, "groups": {"count": 3, "keep": 1}}
    choice = torch.tensor([[-0.1, -0.9, -0.2, -0.3, -0.4, -0.5]], dtype=F64)
    assert plain.choose(choice, router).tolist() == [[0, 1]]
    router["groups"]["keep"] = 2
    assert plain.choose(choice, router).tolist() == [[0, 2]]
    W = 5
    h = _rand(4, W, seed=1)
    t = {"router": _rand(6, W, seed=2), "correction": _rand(6, seed=3)}
    for e in range(4):
        t.update({f"e{e}.gate": _rand(3, W, seed=10 + e), f"e{e}.up": _rand(3, W, seed=20 + e), f"e{e}.down": _rand(W, 3, seed=30 + e)})
    out, idx, c = plain.mixture(h, {"router": router, "expert": {"limit": 0.5}}, t, "")
    s = torch.softmax(h @ t["router"].T, -1)
    assert torch.allclose(c, s + t["correction"])
    for n in range(4):
        w = s[n, idx[n]] / s[n, idx[n]].sum() * 3.0
        want = sum(w[j] * (plain.expert(h[n:n + 1], t, f"e{int(e)}.", 0.5)[0] if e < 4 else h[n]) for j, e in enumerate(idx[n]))
        assert torch.allclose(out[n], want, atol=1e-12)


def test_plain_expert_clamps():
    W = 3
    t = {"gate": torch.eye(W, dtype=F64), "up": torch.eye(W, dtype=F64) * 2, "down": torch.eye(W, dtype=F64)}
    h = torch.tensor([[-9.0, 0.3, 9.0]], dtype=F64)
    y = plain.expert(h, t, "", 1.5)[0]
    sig = lambda z: 1 / (1 + math.exp(-z))
    assert float(y[0]) == pytest.approx(-9.0 * sig(1.702 * -9.0) * (-1.5 + 1))      # the gate has no lower limit
    assert float(y[1]) == pytest.approx(0.3 * sig(1.702 * 0.3) * 1.6)
    assert float(y[2]) == pytest.approx(1.5 * sig(1.702 * 1.5) * 2.5)


@pytest.mark.parametrize("name", sorted(CASES))
def test_random_folder_loads_and_runs_plain(tmp_path, name):
    folder = write(name, str(tmp_path))
    cfg, w = plain.load_folder(folder)
    toks = traces.random_tokens(cfg["vocab"], 40, seed=1)
    layers = []
    logits = plain.forward(cfg, w, toks, layers_out=layers)
    assert logits.shape == (40, cfg["vocab"]) and len(layers) == len(plain.layer_order(cfg)) and bool(torch.isfinite(logits).all())
    # causal: a prefix gives the same logits
    assert torch.allclose(plain.forward(cfg, w, toks[:17]), logits[:17], atol=1e-9)


def test_every_constant_shows_in_the_plain_logits(tmp_path):
    """The comparison with the plain model is sharp: every constant and mechanism moves the plain logits by far more than
    the tolerance when it is dropped or changed."""
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

    def mix(c, i, side):
        return c["layers"][i]["mixer"][side]
    assert moved(lambda c: c.pop("logit_softcap")) > 1e-2
    assert moved(lambda c: c.pop("loop")) > 1e-2
    assert moved(lambda c: c["loop"].update(times=3)) > 1e-2
    assert moved(lambda c: mix(c, 0, "left").pop("rot")) > 1e-3
    assert moved(lambda c: mix(c, 0, "left")["rot"].update(base=200.0)) > 1e-3
    assert moved(lambda c: mix(c, 1, "left").update(scale=0.6)) > 1e-3
    assert moved(lambda c: mix(c, 1, "right").update(decay=[0.9, 0.99])) > 1e-3
    assert moved(lambda c: c["layers"][1]["mixer"].update(right_scale=0.6)) > 1e-3
    router = lambda c: c["layers"][2]["mlp"]["router"]
    assert moved(lambda c: router(c).pop("groups")) > 1e-3
    assert moved(lambda c: router(c).update(scale=1.0)) > 1e-3
    assert moved(lambda c: c["layers"][2]["mlp"]["expert"].update(limit=2.0)) > 1e-3
    assert moved(lambda c: c["layers"][2]["mlp"]["shared"].update(limit=2.0)) > 1e-3
    assert moved(lambda c: c["layers"][2]["mlp"].update(shared=None)) > 1e-3
    for name in ("l0.mix.left.k.conv", "l1.mix.left.v.conv", "l2.mlp.correction", "l0.mlp.down.b", "l0.mlp.up.b", "l0.mix.left.g",
                 "l3.mix.right.g", "l2.mlp.shared.sg"):
        w2 = dict(w)
        w2[name] = torch.zeros_like(w[name])
        assert moved(None, w2) > 1e-3, name
    w2 = dict(w)                                        # the oldest tap alone
    w2["l0.mix.left.q.conv"] = w["l0.mix.left.q.conv"].clone()
    w2["l0.mix.left.q.conv"][:, 0] = 0
    assert moved(None, w2) > 1e-3
