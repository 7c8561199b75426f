"""The Pukatar configuration on the CPU: what its config.json turns into, what is refused, the tensors a model wants,
what the cache manager is asked for, the rotation's table, and the plain implementation's own consistency."""
import copy

import pytest
import torch

import plain_pukatar as pp
import pukatar_models as pm
from litellmengine_b200.cache import CacheManager, PagedNeed, StateNeed
from litellmengine_b200.config import ConfigError, PukatarConfig, config_from_dict
from litellmengine_b200.config.specs import ModelPlan, NormSpec, PositionSpec, RejoinSpec, StageSpec
from litellmengine_b200.parts.model import Model, model_parameters
from litellmengine_b200.parts.registry import lookup

ALL = (pm.PUK_A, pm.PUK_B, pm.PUK_C, pm.PUK_D, pm.PUK_E)


def test_plan_of_a_configuration():
    cfg = config_from_dict(pm.PUK_A)
    assert isinstance(cfg, PukatarConfig) and cfg.to_dict() == pm.PUK_A
    plan = cfg.plan()
    assert [(s.block, s.starts_pass) for s in plan.order] == [(0, None), (1, 0), (2, None), (1, 1), (2, None), (1, 2), (2, None), (3, None)]
    assert plan.rejoin == RejoinSpec(3) and plan.embedding_norm == plan.final_norm == NormSpec("layernorm", 1e-5, "", True)
    assert all(b.arrangement == "parallel_pre_norm" and b.feed_forward_norm is None for b in plan.blocks)
    d, a, d2, a2 = (b.mixer for b in plan.blocks)
    assert d.kind == "delta_rule" and (d.num_heads, d.num_kv_heads, d.head_dim, d.value_dim) == (4, 2, 12, 20)
    assert dict(d.params) == {"taps": 3, "eps": 1e-5, "decay_rank": None, "gate_rank": None}
    assert a.kind == "gated_attention" and not a.bias and a.qk_norm is None and a.output_gate is None and a.learned_sink
    assert (a.window, a.keep_first, a.scale, a.value_dim) == (9, 3, 0.3, 24)
    assert (a.position.kind, a.position.theta, a.position.rotary_dim) == ("rope_half", 500.0, 8)
    assert plan.blocks[3].feed_forward is None and plan.blocks[0].feed_forward.kind == "swiglu"
    ff = dict(plan.blocks[1].feed_forward.params)
    assert (ff["experts"], ff["top"], ff["limit"], ff["score"], ff["router_bias"]) == (5, 2, 1.1, "softmax", True)
    assert (ff["shared"], ff["shared_limit"], ff["shared_gate"], ff["shared_activation"]) == (24, 0.7, True, "clamped_swish")
    assert "shared" not in dict(plan.blocks[2].feed_forward.params)


@pytest.mark.parametrize("cfg", ALL)
def test_tensors_are_the_designs_names(cfg):
    want = pm.tensor_shapes(cfg)
    got = model_parameters(config_from_dict(cfg).plan())
    assert set(got) == set(want)
    for n, p in got.items():       # -1: the ranks of the low-rank projections, which only the tensors know
        assert len(p.shape) == len(want[n]) and all(a in (-1, b) for a, b in zip(p.shape, want[n])), n


@pytest.mark.parametrize("cfg", ALL)
def test_run_order_is_the_plain_one(cfg):
    assert config_from_dict(cfg).run_order() == pp.run_order(cfg)


def test_no_loop_means_no_rejoin():
    plan = config_from_dict(pm.PUK_D).plan()
    assert plan.rejoin is None and all(s.starts_pass is None for s in plan.order)


def test_what_is_refused():
    def broken(change):
        d = copy.deepcopy(pm.PUK_A)
        change(d)
        with pytest.raises(ConfigError):
            config_from_dict(d)
    broken(lambda d: d["layers"][0].update(type="conv"))
    broken(lambda d: d["layers"][0]["mixer"].update(kv_heads=3))
    broken(lambda d: d["layers"][0]["mixer"].pop("conv"))
    broken(lambda d: d["layers"][1]["mixer"].update(kv_heads=3))
    broken(lambda d: d["layers"][1]["mixer"]["rot"].update(dims=7))
    broken(lambda d: d["layers"][1]["mixer"]["rot"].update(dims=18))
    broken(lambda d: d["layers"][1]["mixer"]["rot"].update(base=0.0))
    broken(lambda d: d["layers"][1]["mixer"]["mask"].update(keep_first=-1))
    broken(lambda d: d["layers"][1]["mlp"]["router"].update(top=6))
    broken(lambda d: d["layers"][1]["mlp"]["expert"].update(limit=0.0))
    broken(lambda d: d["layers"][1]["mlp"]["shared"].pop("limit"))
    broken(lambda d: d["layers"][1]["mlp"].update(kind="sparse"))
    broken(lambda d: d["loop"].update(stop=5))
    broken(lambda d: d["loop"].update(start=3))
    broken(lambda d: d["loop"].update(times=0))
    broken(lambda d: d.pop("norm"))


def test_a_pass_needs_a_rejoin():
    plan = config_from_dict(pm.PUK_D).plan()
    bad = ModelPlan(**{**plan.__dict__, "order": (StageSpec(0, None, 0),)})
    with pytest.raises(ValueError):
        bad.validate()


def test_options_that_may_be_absent():
    d = copy.deepcopy(pm.PUK_A)
    m = d["layers"][1]["mixer"]
    del m["mask"], m["rot"], d["loop"]
    d["layers"][1]["mlp"].pop("shared")
    a = config_from_dict(d).plan().blocks[1].mixer
    assert a.window is None and a.keep_first == 0 and a.position.kind == "none" and a.learned_sink


def test_rotation_of_halves():
    pos = lookup("position", "rope_half")(PositionSpec("rope_half", 700.0, 12), 16, "cpu")
    for i, got in enumerate(pos.freq.tolist()):
        assert abs(got - 700.0 ** (-2.0 * i / 12)) < 1e-7 * got
    assert pos.kernel_args()[1:] == (12, 1.0, False)


def test_cache_needs():
    model = Model(config_from_dict(pm.PUK_A).plan(), dtype="float32", device="meta")
    needs = model.stage_needs()
    assert len(needs) == 8 and needs[1] == PagedNeed(2, 16, 9, 24, 3) == needs[3] == needs[5]      # three passes, a cache each
    assert needs[7] == PagedNeed(2, 8, 30, None, 20)
    state = lambda H, G, D, V, taps: StateNeed((-(-(H * V * 32 + taps * (2 * G * D + H * V)) // 4) * 4,), "float32")
    assert needs[0] == state(4, 2, 12, 20, 3) and needs[2] == needs[4] == needs[6] == state(3, 3, 32, 16, 4)
    m = CacheManager([needs[1], needs[3], needs[7], needs[2]], page_size=16, max_total_tokens=128, max_slots=2)
    assert [g.stages for g in m.groups] == [[0, 1], [2]]


# ---- the plain implementation against itself: what the comparisons rest on ---------------------------------
def test_plain_delta_rule_moves_a_written_value_towards_its_target():
    """Writing v at a unit key k with step size one and no decay replaces what the state held at k; a half step goes
    half way; a decay of zero on a row forgets it."""
    k = torch.tensor([0.6, 0.0, 0.8], dtype=torch.float64).view(1, 1, 3)
    one = torch.ones(1, 1, 3, dtype=torch.float64)
    v, w = (torch.randn(1, 1, 2, dtype=torch.float64, generator=torch.Generator().manual_seed(s)) for s in (1, 2))
    b = lambda x: torch.full((1, 1), x, dtype=torch.float64)
    o, S = pp.delta_rule(k, k, v, b(1.0), one)
    assert (o[0, 0] - v[0, 0]).abs().max() < 1e-12
    o, S2 = pp.delta_rule(k, k, w, b(1.0), one, S)
    assert (o[0, 0] - w[0, 0]).abs().max() < 1e-12
    o, _ = pp.delta_rule(k, k, w, b(0.5), one, S)
    assert (o[0, 0] - (v[0, 0] + w[0, 0]) / 2).abs().max() < 1e-12
    gone = one.clone()
    gone[..., 0] = 0.0
    _, S3 = pp.delta_rule(k, k, w, b(0.0), gone, S2)
    assert S3[0, 0].abs().max() == 0 and (S3[0, 2] - S2[0, 2]).abs().max() == 0


def test_plain_convolution_is_causal_and_its_last_tap_is_the_token():
    x = torch.randn(7, 2, dtype=torch.float64, generator=torch.Generator().manual_seed(1))
    taps = torch.tensor([[0.0, 0.0, 1.0], [1.0, 0.0, 0.0]], dtype=torch.float64)
    y = pp.short_conv(x, taps)
    assert torch.equal(y[:, 0], x[:, 0]) and torch.equal(y[2:, 1], x[:-2, 1]) and y[:2, 1].abs().max() == 0
    assert pp.short_conv(x[:1], taps).shape == (1, 2)


def test_plain_window_edges_and_kept_keys():
    vis = pp.visible_keys(12, {"size": 3, "keep_first": 2})
    assert [j for j in range(12) if vis[9, j]] == [0, 1, 7, 8, 9]
    assert [j for j in range(12) if vis[3, j]] == [0, 1, 2, 3] and [j for j in range(12) if vis[0, j]] == [0]
