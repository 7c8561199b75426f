"""The Purivik configuration on the CPU: what its config.json turns into, what is refused, the tensors a model wants, what
the cache manager is asked for and how it forgets by chunks, the rotation's table, what the norms' weights take in when a
layer is loaded, and the plain implementation's own consistency."""
import copy
import math

import pytest
import torch

import plain_purivik as pp
import purivik_models as pm
from litellmengine_b200.cache import CacheError, CacheManager, PagedNeed
from litellmengine_b200.config import ConfigError, PurivikConfig, config_from_dict
from litellmengine_b200.config.specs import MixerSpec, ModelPlan, NormSpec, PositionSpec, RejoinSpec
from litellmengine_b200.parts.attention import decode_reach, key_span
from litellmengine_b200.parts.model import Model, model_parameters
from litellmengine_b200.parts.registry import lookup

ALL = (pm.PUR_A, pm.PUR_B, pm.PUR_C, pm.PUR_D, pm.PUR_E)


def test_plan_of_a_configuration():
    cfg = config_from_dict(pm.PUR_A)
    assert isinstance(cfg, PurivikConfig) and cfg.to_dict() == pm.PUR_A
    plan = cfg.plan()
    assert [(s.block, s.starts_pass) for s in plan.order] == [(0, None), (1, 0), (2, None), (1, 1), (2, None), (1, 2), (2, None), (3, None)]
    assert plan.rejoin == RejoinSpec(3, kind="add") and plan.embedding_scale == 0.3 and plan.tie_word_embeddings
    assert plan.final_norm == NormSpec("rmsnorm", 1e-5, "")
    assert all(b.arrangement == "sandwich_norm" and b.branch_scale == 0.7 and b.layer_scale_names == ("ls1", "ls2") for b in plan.blocks)
    a = plan.blocks[0].mixer
    assert a.kind == "gated_attention" and not a.bias and a.qk_norm is None and a.output_gate is None and not a.learned_sink
    assert (a.window, a.chunk, a.scale, a.value_dim, a.num_heads, a.num_kv_heads, a.head_dim) == (None, 37, 0.3, 24, 4, 2, 16)
    assert (a.position.kind, a.position.theta, a.position.rotary_dim) == ("rope_half", 500.0, 8)
    assert dict(a.position.params) == {"wavelengths": (3.0, 1.0, 5.0, 60.0)}
    assert dict(plan.blocks[1].mixer.position.params) == {} and plan.blocks[3].mixer.position.kind == "none"
    assert plan.blocks[3].feed_forward is None and plan.blocks[1].feed_forward.kind == "swiglu"
    assert dict(plan.blocks[1].feed_forward.params) == {"activation": "clamped_swish", "limit": 0.9}
    ff = dict(plan.blocks[0].feed_forward.params)
    assert (ff["experts"], ff["top"], ff["score"], ff["normalize"], ff["weight_on_input"], ff["activation"]) == (5, 2, "sigmoid", False, True, "silu")


@pytest.mark.parametrize("cfg", ALL)
def test_tensors_are_the_designs_names(cfg):
    want = pm.tensor_shapes(cfg)
    got = model_parameters(config_from_dict(cfg).plan())
    head = got.pop("head")                                   # the embedding table itself, unless a file brought one
    assert head.optional_alias == "embed"
    assert {n: tuple(p.shape) for n, p in got.items()} == want


@pytest.mark.parametrize("cfg", ALL)
def test_run_order_is_the_plain_one(cfg):
    """The plain order says where the embedding output joins: in front of every pass but the first."""
    assert [(i, t is not None and t > 0) for i, t in config_from_dict(cfg).run_order()] == pp.run_order(cfg)


def test_no_loop_means_no_rejoin():
    plan = config_from_dict(pm.PUR_D).plan()
    assert plan.rejoin is None and all(s.starts_pass is None for s in plan.order)
    with pytest.raises(ValueError):
        ModelPlan(**{**plan.__dict__, "rejoin": RejoinSpec(1, kind="other")}).validate()


def test_what_is_refused():
    def broken(change):
        d = copy.deepcopy(pm.PUR_A)
        change(d)
        with pytest.raises(ConfigError):
            config_from_dict(d)
    broken(lambda d: d["layers"][0].update(type="channel_delta"))
    broken(lambda d: d["layers"][0].pop("mixer"))
    broken(lambda d: d["layers"][0]["mixer"].update(kv_heads=3))
    broken(lambda d: d["layers"][0]["mixer"].pop("scale"))
    broken(lambda d: d["layers"][0]["mixer"]["mask"].update(size=0))
    broken(lambda d: d["layers"][0]["mixer"]["rot"].update(dims=7))
    broken(lambda d: d["layers"][0]["mixer"]["rot"].update(dims=18))
    broken(lambda d: d["layers"][0]["mixer"]["rot"].update(base=0.0))
    broken(lambda d: d["layers"][0]["mixer"]["rot"]["scaling"].pop("low"))
    broken(lambda d: d["layers"][0]["mixer"]["rot"]["scaling"].update(high=0.5))
    broken(lambda d: d["layers"][0]["mlp"]["router"].update(top=6))
    broken(lambda d: d["layers"][0]["mlp"].pop("expert"))
    broken(lambda d: d["layers"][1]["mlp"].update(limit=0.0))
    broken(lambda d: d["layers"][1]["mlp"].pop("limit"))
    broken(lambda d: d["layers"][1]["mlp"].update(kind="sparse"))
    broken(lambda d: d["loop"].update(stop=5))
    broken(lambda d: d["loop"].update(start=3))
    broken(lambda d: d["loop"].update(times=0))
    broken(lambda d: d.pop("norm"))
    broken(lambda d: d.pop("embedding"))
    broken(lambda d: d.pop("residual_mult"))


def test_frequencies_stretched_by_wavelength():
    """Against the plain table, with pairs on both sides of the ramp and on it, and with a ramp of no width."""
    for base, dims, scaling in ((500.0, 8, (3.0, 1.0, 5.0, 60)), (250.0, 64, (4.0, 1.0, 4.0, 128)), (1e4, 32, (8.0, 2.0, 2.0, 512)),
                                (30.0, 6, None)):
        rot = {"base": base, "dims": dims}
        params = ()
        if scaling:
            rot["scaling"] = dict(zip(("factor", "low", "high", "original"), scaling))
            params = (("wavelengths", scaling),)
        pos = lookup("position", "rope_half")(PositionSpec("rope_half", base, dims, params), dims + 4, "cpu")
        want = pp.frequencies(rot)
        assert ((pos.freq.double() - want).abs() <= 1e-7 * want).all()
        assert pos.kernel_args()[1:] == (dims, 1.0, False)
        if scaling and scaling[1] < scaling[2]:
            ratio = want / torch.tensor([base ** (-2.0 * i / dims) for i in range(dims // 2)], dtype=torch.float64)
            assert ratio.max() == 1.0 and abs(ratio.min() - 1.0 / scaling[0]) < 1e-12
            assert ((ratio < 1.0 - 1e-9) & (ratio > 1.0 / scaling[0] + 1e-9)).any()
    with pytest.raises(ValueError):
        lookup("position", "rope_half")(PositionSpec("rope_half", 1e4, 8, (("wavelengths", (2.0, 4.0, 1.0, 64)),)), 8, "cpu")
    with pytest.raises(ValueError):
        lookup("position", "rope_half")(PositionSpec("rope_half", 1e4, 8, (("wavelengths", (2.0, 1.0, 4.0, 64)), ("scaling", (2.0, 64, 8, 1)))), 8, "cpu")


def test_key_spans():
    class B:
        max_kv_len = 50
    span = lambda **k: key_span(MixerSpec(kind="gated_attention", **k))
    assert (span(), span(window=7), span(chunk=9)) == (None, 7, -9)
    assert (decode_reach(B, None), decode_reach(B, 7), decode_reach(B, -9), decode_reach(B, -90)) == (50, 7, 9, 50)
    for bad in (dict(window=0), dict(chunk=0), dict(window=4, chunk=4)):
        with pytest.raises(ValueError):
            span(**bad)


def test_cache_needs():
    model = Model(config_from_dict(pm.PUR_A).plan(), dtype="float32", device="meta")
    needs = model.stage_needs()
    assert len(needs) == 8 and needs[0] == PagedNeed(2, 16, None, 24, 0, 37)
    assert needs[1] == PagedNeed(2, 8, None, None, 0, 9) == needs[3] == needs[5]            # three passes, a cache each
    m = CacheManager(needs, page_size=16, max_total_tokens=128, max_slots=2)
    assert [g.stages for g in m.groups] == [[0], [1, 3, 5], [2, 4, 6], [7]]


def test_cache_forgets_by_chunks():
    """Pages wholly before the next position's chunk go back, whatever portions the request came in; a page that a chunk's
    edge cuts stays until the chunk that ends in it is over; requests may be longer than the pool."""
    P = 4
    for chunk in (1, 3, 4, 10, 12, 17):
        for portions in ([60], [1] * 60, [7, 2, 13, 1, 1, 20, 16]):
            m = CacheManager([PagedNeed(1, 8, chunk=chunk)], page_size=P, max_total_tokens=64, max_slots=2, max_request_tokens=200)
            g, slot, n = m.groups[0], m.admit(), 0
            for k in portions:
                held = set(g.held_pages(slot))
                m.ensure(slot, n + k)
                first = n // chunk * chunk                                       # what the portion's first token still sees
                for pos in range(first, n + k):
                    assert int(g.table[slot, pos // P]) in set(g.held_pages(slot))
                assert held <= set(g.held_pages(slot))
                n += k
                m.commit(slot, n)
                lo = n // chunk * chunk // P
                assert int(g.first_held[slot]) == lo and len(g.held_pages(slot)) == -(-n // P) - lo
                m.check_invariants()
            m.release(slot)
            m.check_invariants()
            assert g.pool.free_count == g.pool.num_pages
    m = CacheManager([PagedNeed(1, 8, chunk=8)], page_size=P, max_total_tokens=16, max_slots=1, max_request_tokens=100)
    slot = m.admit()
    for n in range(5, 101, 5):                                                   # 100 tokens through four pages
        m.ensure(slot, n)
        m.commit(slot, n)
    with pytest.raises(CacheError):
        CacheManager([PagedNeed(1, 8, window=4, chunk=8)], page_size=P, max_total_tokens=16, max_slots=1)


def test_a_layers_factors_join_the_output_norms_weights():
    """After loading, the norm on a sublayer's output carries weight * layer scale * residual factor; the norms in front
    and the model's last norm are what the file holds."""
    from litellmengine_b200.parts.block import Block
    cfg, w = pm.PUR_D, pm.random_weights(pm.PUR_D, 1)
    spec = config_from_dict(cfg).plan().blocks[1]
    block = Block(spec, cfg["width"], torch.float32, "cpu")
    block.load({n[3:]: t for n, t in w.items() if n.startswith("l1.")})
    m = cfg["residual_mult"]
    assert torch.allclose(block.mixer_post_norm.weight, w["l1.norm1b"] * w["l1.ls1"] * m, rtol=1e-6)
    assert torch.allclose(block.feed_forward_post_norm.weight, w["l1.norm2b"] * w["l1.ls2"] * m, rtol=1e-6)
    assert torch.equal(block.mixer_norm.weight, w["l1.norm1"]) and torch.equal(block.feed_forward_norm.weight, w["l1.norm2"])
    bad = spec.__class__(**{**spec.__dict__, "mixer_post_norm": None})
    with pytest.raises(ValueError):
        Block(bad, cfg["width"], torch.float32, "cpu")


# ---- the plain implementation against itself: what the comparisons rest on ---------------------------------
def test_plain_chunk_edges():
    vis = pp.visible_keys(12, {"size": 5})
    assert [j for j in range(12) if vis[4, j]] == [0, 1, 2, 3, 4] and [j for j in range(12) if vis[5, j]] == [5]
    assert [j for j in range(12) if vis[11, j]] == [10, 11] and [j for j in range(12) if vis[9, j]] == [5, 6, 7, 8, 9]
    assert pp.visible_keys(6, {"size": 1}).equal(torch.eye(6, dtype=torch.bool))
    assert pp.visible_keys(6, None).equal(pp.visible_keys(6, {"size": 6}))


def test_plain_weight_acts_on_the_input():
    """With one expert chosen, the result is the expert run on the weighted input, which is not its weighted output."""
    g = torch.Generator().manual_seed(1)
    w = {"router": torch.randn(4, 6, generator=g), **{f"e{e}.{k}": torch.randn(*s, generator=g) for e in range(4)
                                                      for k, s in (("gate", (5, 6)), ("up", (5, 6)), ("down", (6, 5)))}}
    u = torch.randn(3, 6, generator=g, dtype=torch.float64)
    pick, weight = pp.route(u, w, "", 1)
    out = pp.routed_ff(u, w, "", {"router": {"top": 1}})
    for t in range(3):
        e, a = int(pick[t, 0]), float(weight[t, 0])
        assert abs(a - 1.0 / (1.0 + math.exp(-float(u[t] @ w["router"][e].double())))) < 1e-12
        assert (out[t] - pp.expert(a * u[t:t + 1], w, f"e{e}.")[0]).abs().max() < 1e-12
        assert (out[t] - a * pp.expert(u[t:t + 1], w, f"e{e}.")[0]).abs().max() > 1e-3


def test_plain_clamps():
    u = torch.eye(3, dtype=torch.float64)
    w = {"gate": torch.tensor([[9.0, -9.0, 0.5]]), "up": torch.tensor([[9.0, -9.0, 0.5]]), "down": torch.tensor([[1.0]])}
    got = pp.dense_ff(u, w, "", 2.0)[:, 0]
    f = lambda a, b: a / (1 + math.exp(-1.702 * a)) * (b + 1)
    assert all(abs(float(x) - y) < 1e-12 for x, y in zip(got, (f(2.0, 2.0), f(-9.0, -2.0), f(0.5, 0.5))))
