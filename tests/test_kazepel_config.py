"""The Kazepel configuration on the CPU: what it reads, what it refuses, the tensors it declares (the ranks that
the file decides among them), the run order of a loop, what the cache manager keeps of a window with first
tokens, yarn's frequencies, and the plain restatement's own mechanisms on cases small enough to do by hand."""
import copy
import math
import os
import random

import pytest
import torch

import plain_kazepel as plain
from tiny_kazepel import TINY
from tokenizer_b200.cache.manager import CachePlan, OutOfPages
from tokenizer_b200.config import ConfigError, KazepelConfig, config_from_dict
from tokenizer_b200.parts.base import CacheNeed, KVNeed, StateNeed
from tokenizer_b200.parts.model import declared_tensors
from tokenizer_b200.weights import WeightError, WeightStore, write_random_model
from tokenizer_b200.weights.random_init import SeededTensors


def test_the_registry_finds_the_design_by_its_name():
    cfg = TINY["a"]()[0]
    again = config_from_dict(cfg.to_dict())
    assert isinstance(again, KazepelConfig) and again.to_dict() == cfg.to_dict()
    assert config_from_dict(dict(cfg.to_dict(), architectures=["Kazepel"])).to_dict() == cfg.to_dict()


def test_declared_tensors_follow_the_sizes():
    cfg = TINY["a"]()[0]
    shapes = {t.name: tuple(t.shape) for t in declared_tensors(cfg.model_spec())}
    assert shapes["embed"] == (301, 96) and "head" not in shapes
    assert shapes["loop.in"] == (96, 192) and shapes["loop.step"] == (3, 96)
    for name in ("l0.norm1", "l0.norm2", "l3.norm1", "final.norm"):
        assert shapes[name] == (96,) and shapes[name + ".b"] == (96,) and shapes[name + ".alpha"] == ()
    assert shapes["l0.mix.q"] == (2 * 24, 96) and shapes["l0.mix.k.conv"] == (48, 3) and shapes["l0.mix.v"] == (4 * 16, 96)
    assert shapes["l0.mix.b"] == (4, 96) and shapes["l0.mix.A_log"] == (4,) and shapes["l0.mix.dt_bias"] == (4 * 24,)
    assert shapes["l0.mix.norm"] == (16,) and shapes["l0.mix.a2"][0] == 4 * 24 and shapes["l0.mix.g2"][0] == 4 * 16
    assert shapes["l0.mlp.router"] == (6, 96) and shapes["l0.mlp.correction"] == (6,) and "l0.mlp.e5.up" not in shapes
    assert shapes["l1.mix.o"] == (96, 6 * 32) and shapes["l1.mlp.router"] == (9, 96)
    # no feed-forward: neither its tensors nor the norm in front of it
    assert not any(n.startswith("l2.mlp") or n.startswith("l2.norm2") for n in shapes)
    assert not any(".mix." in n and n.endswith(".b") and ".mix.b" not in n for n in shapes)      # no biases


def test_the_file_decides_the_bottlenecks_ranks(tmp_path):
    cfg, seed, _, sizes = TINY["a"]()
    specs = declared_tensors(cfg.model_spec())
    folder = write_random_model(str(tmp_path / "m"), cfg, seed, sizes=sizes)
    store = WeightStore.from_folder(folder)
    store.check(specs)
    assert store.get("l0.mix.a1").shape == (9, 96) and store.get("l0.mix.a2").shape == (96, 9)
    assert store.get("l2.mix.g1").shape == (5, 96) and store.get("l2.mix.a2").shape == (80, 16)
    WeightStore(SeededTensors(specs, 1)).check(specs)                  # the defaults fit too
    # the two tensors of one bottleneck must agree, and the fixed dimensions stay fixed
    store.tensors["l0.mix.a2"] = torch.zeros(96, 10)
    with pytest.raises(WeightError, match="l0.mix.a2"):
        store.check(specs)
    store.tensors["l0.mix.a2"] = torch.zeros(95, 9)
    with pytest.raises(WeightError, match="l0.mix.a2"):
        store.check(specs)
    assert os.path.exists(os.path.join(folder, "config.json"))


@pytest.mark.parametrize("change,word", [
    (lambda r: r["layers"][0].update(type="other"), "unknown type"),
    (lambda r: r["layers"][0]["mixer"].update(kv_heads=3), "do not divide"),
    (lambda r: r["layers"][0]["mixer"].pop("conv"), "conv"),
    (lambda r: r["layers"][1]["mixer"].pop("scale"), "scale"),
    (lambda r: r["layers"][1]["mixer"].update(mask={"size": 0}), "size"),
    (lambda r: r["layers"][1]["mixer"].update(mask={"keep_first": 3}), "size"),
    (lambda r: r["layers"][1]["mixer"]["mask"].update(keep_first=-1), "keep_first"),
    (lambda r: r["layers"][1]["mixer"]["rot"].update(dims=18), "rot.dims"),
    (lambda r: r["layers"][1]["mixer"]["rot"]["scaling"].pop("fast"), "fast"),
    (lambda r: r["layers"][1]["mixer"]["rot"]["scaling"].update(factor=0.0), "scaling"),
    (lambda r: r["layers"][0]["mlp"]["router"].update(top=4), "cannot give"),
    (lambda r: r["layers"][0]["mlp"]["router"].update(identity=2), "cannot give"),     # seven outputs in two groups
    (lambda r: r["layers"][0]["mlp"]["expert"].pop("limit"), "limit"),
    (lambda r: r["layers"][0]["mlp"].update(kind="dense"), "moe"),
    (lambda r: r["loop"].update(stop=5), "loop"),
    (lambda r: r.pop("norm"), "norm"),
    (lambda r: r.update(layers=[]), "layers"),
])
def test_what_the_configuration_refuses(change, word):
    raw = copy.deepcopy(TINY["a"]()[0].to_dict())
    change(raw)
    with pytest.raises(ConfigError, match=word):
        KazepelConfig.from_dict(raw)


def test_a_loop_repeats_calls_and_every_pass_enters_once():
    spec = TINY["b"]()[0].model_spec()
    assert [c.layer for c in spec.order] == [0, 1, 2] * 2 + [3]
    entries = [(at, c.before.params["index"]) for at, c in enumerate(spec.order) if c.before is not None]
    assert entries == [(0, 0), (3, 1)] and all(c.cache is None for c in spec.order)
    assert spec.order[0].before.kind == "pass_projection"
    raw = copy.deepcopy(TINY["b"]()[0].to_dict())
    raw.pop("loop")
    spec = KazepelConfig.from_dict(raw).model_spec()
    assert [c.layer for c in spec.order] == [0, 1, 2, 3] and all(c.before is None for c in spec.order)
    assert "loop.in" not in {t.name for t in declared_tensors(spec)}


def test_the_model_spec_names_parts_that_other_designs_can_use():
    spec = TINY["a"]()[0].model_spec()
    assert [l.block for l in spec.layers] == ["pre_norm_residual"] * 2 + ["pre_norm_mixer_only"] * 2
    assert [l.parts["mixer"].kind for l in spec.layers] == ["channel_delta_net", "gqa_rotary"] * 2
    a = spec.layers[1].parts["mixer"].params
    assert (a["window"], a["keep_first"], a["unit_sink"], a["bias"], a["chunk"]) == (19, 5, True, False, None)
    assert a["position"].kind == "rope_half" and a["position"].params["scaling"] == \
        {"kind": "yarn", "factor": 3.0, "original": 256.0, "fast": 16.0, "slow": 1.5}
    assert spec.layers[3].parts["mixer"].params["position"].params["scaling"] is None
    routed = spec.layers[1].parts["feed_forward"].params
    assert (routed["score"], routed["groups"], routed["group_keep"], routed["group_worth"], routed["identity"],
            routed["renormalize"], routed["limit"]) == ("softmax", 3, 2, 1, 3, True, 0.7)
    assert spec.final_norm.params["scale"] == 0.3 and "scale" not in spec.layers[0].parts["mixer_norm"].params
    assert spec.head.params["tied_to"] == "embed"
    open_ = TINY["c"]()[0].model_spec()
    assert open_.layers[2].parts["mixer"].params["window"] is None and open_.layers[2].parts["mixer"].params["position"] is None
    assert "scale" not in open_.final_norm.params


# ---- windows that keep the first tokens, in the cache manager ---------------------------------------------
def test_pages_of_the_first_tokens_stay_and_the_ones_between_go():
    plan = CachePlan([CacheNeed(kv=KVNeed(2, 16, 9, keep_first=6))], num_pages=16, page_size=4, max_requests=2)
    r = plan.open("r")
    plan.reserve(r, 3)
    plan.commit(r, 3)
    plan.reserve(r, 27)
    plan.commit(r, 27)                 # next position 30: the window reaches back to 21, the first six are kept
    assert [p >= 0 for p in r.tables[0]] == [True, True, False, False, False, True, True, True]
    plan.check()
    before = r.tables[0][:2]
    for _ in range(20):
        plan.reserve(r, 1)
        plan.commit(r, 1)
        plan.check()
    assert r.tables[0][:2] == before and len(r.pages_held(0)) <= 2 + 4
    plan.close(r)
    assert plan.allocators[0].all_released()


def test_calls_that_keep_unlike_numbers_of_first_tokens_do_not_share_a_group():
    needs = [CacheNeed(kv=KVNeed(2, 16, 9, keep_first=k)) for k in (6, 0, 6, 7)]
    plan = CachePlan(needs, 8, 4, 2)
    assert [(g.keep_first, g.calls) for g in plan.groups] == [(6, [0, 2]), (0, [1]), (7, [3])]


@pytest.mark.parametrize("seed", range(6))
def test_every_key_a_query_can_see_has_a_page_under_random_orders(seed):
    rng = random.Random(seed)
    window, keep, page = rng.choice([0, 3, 10, 17]), rng.choice([0, 1, 4, 9, 30]), rng.choice([2, 4, 8])
    plan = CachePlan([CacheNeed(kv=KVNeed(1, 16, window, keep_first=keep)), CacheNeed(state=StateNeed((4,)))], 40, page, 4)
    live = {}
    for step in range(300):
        if rng.random() < 0.3 and len(live) < 4:
            live[step] = plan.open(step)
        elif live and rng.random() < 0.1:
            plan.close(live.pop(rng.choice(sorted(live))))
        elif live and rng.random() < 0.1:
            plan.release_pages(live[rng.choice(sorted(live))])
        elif live:
            cache, n = live[rng.choice(sorted(live))], rng.randrange(1, 13)
            if not plan.can_reserve(cache, n):
                with pytest.raises(OutOfPages):
                    plan.reserve(cache, n)
                plan.close(live.pop(cache.request_id))
                continue
            plan.reserve(cache, n)
            for q in range(cache.length, cache.length + n):
                for key in range(q + 1):
                    if q - key <= window or key < keep:
                        assert cache.tables[0][key // page] >= 0
            plan.commit(cache, n)
        plan.check()
    for cache in live.values():
        plan.close(cache)
    assert plan.allocators[0].all_released()


# ---- yarn's rotation ------------------------------------------------------------------------------------
@pytest.mark.parametrize("base,dims,scaling", [(5000.0, 32, (3.0, 256, 16.0, 1.5)), (70000.0, 16, (2.0, 64, 8.0, 0.5)),
                                               (50.0, 8, (1.5, 128, 3.0, 1.0)), (10000.0, 64, (40.0, 4096, 32.0, 1.0)),
                                               (1000.0, 16, (16.0, 32, 8.0, 2.0)), (100.0, 2, (4.0, 32, 4.0, 1.0))])
def test_yarn_frequencies_of_the_rotation_part(base, dims, scaling):
    from tokenizer_b200.parts.position import scaled_frequencies, scaled_magnitude
    named = dict(zip(("factor", "original", "fast", "slow"), scaling))
    freq = [base ** (-2.0 * i / dims) for i in range(dims // 2)]
    got = scaled_frequencies(freq, dict(named, kind="yarn"), base)
    want, magnitude = plain.yarn_frequencies(base, dims, named)
    assert got == pytest.approx(want, rel=1e-14)
    assert scaled_magnitude(dict(named, kind="yarn")) == pytest.approx(magnitude) == pytest.approx(0.1 * math.log(scaling[0]) + 1.0)
    assert scaled_magnitude(None) == 1.0 and scaled_magnitude({"kind": "linear", "factor": 4.0}) == 1.0


def test_yarn_by_hand():
    # base 100 over 8 lanes, original 2 pi 100: the pair that turns t times has index 4 ln(100 / t) / ln 100
    freqs, _ = plain.yarn_frequencies(100.0, 8, {"factor": 10.0, "original": 2.0 * math.pi * 100.0, "fast": 10.0, "slow": 1.0})
    # fast 10: index 2 exactly (lo = 2); slow 1: index 4 (hi = 4): pairs 0..2 kept, pair 3 halfway
    plain_freqs = [100.0 ** (-i / 4.0) for i in range(4)]
    assert freqs[:3] == pytest.approx(plain_freqs[:3])
    assert freqs[3] == pytest.approx(plain_freqs[3] * (0.5 / 10.0 + 0.5))


# ---- the plain restatement, by hand ---------------------------------------------------------------------
def test_plain_windows_count_as_the_design_says():
    seen = plain.seen_keys(7, {"size": 2, "keep_first": 1})
    assert seen[5].tolist() == [True, False, False, False, True, True, False]       # the kept first, itself and one before
    assert seen[0].tolist() == [True] + [False] * 6 and seen[1].tolist() == [True, True] + [False] * 5
    assert plain.seen_keys(3, {"size": 1})[2].tolist() == [False, False, True]
    assert plain.seen_keys(3, None)[2].tolist() == [True, True, True]


def test_plain_softmax_has_one_more_in_its_denominator():
    s = torch.tensor([[0.0, math.log(3.0), -math.inf]], dtype=torch.float64)
    assert plain.softmax_one(s)[0].tolist() == pytest.approx([1.0 / 5.0, 3.0 / 5.0, 0.0])
    low = torch.full((1, 4), -1000.0, dtype=torch.float64)
    assert float(plain.softmax_one(low).sum()) == 0.0                 # nothing stands out: the sink takes it all
    high = torch.tensor([[900.0, 0.0]], dtype=torch.float64)
    assert plain.softmax_one(high)[0].tolist() == pytest.approx([1.0, 0.0])


def test_plain_router_by_hand():
    z = torch.log(torch.tensor([0.4, 0.1, 0.3, 0.2], dtype=torch.float64))
    none = torch.zeros(4, dtype=torch.float64)
    assert plain.route(z, none, 2, 1, 1) == pytest.approx({0: 0.4 / 0.7, 2: 0.3 / 0.7})
    # groups {0, 1} and {2, 3}: by the largest score the first is better although the sums are equal
    assert plain.route(z, none, 2, 2, 1) == pytest.approx({0: 0.8, 1: 0.2})
    # choice scores below zero still beat an expert of a closed group
    assert plain.route(z, torch.tensor([-1.0, -1.0, -2.0, -2.0], dtype=torch.float64), 2, 2, 1) == pytest.approx({0: 0.8, 1: 0.2})
    # the correction moves the choice, not the weight
    assert plain.route(z, torch.tensor([0.0, 1.0, 0.0, 0.0], dtype=torch.float64), 1, 1, 1) == {1: 1.0}


def test_plain_delta_rule_decays_every_row_by_its_own_factor():
    q = torch.tensor([[1.0, 0.0], [1.0, 1.0]], dtype=torch.float64)
    k = torch.tensor([[0.6, 0.8], [0.0, 0.0]], dtype=torch.float64)
    v = torch.tensor([[10.0], [0.0]], dtype=torch.float64)
    decay = torch.tensor([[0.3, 0.9], [0.5, 0.25]], dtype=torch.float64)
    o, S = plain.channel_delta_rule(q, k, v, torch.tensor([0.5, 1.0], dtype=torch.float64), decay)
    # token 0 writes 5 k; token 1 decays the rows by 1/2 and 1/4 and writes nothing
    assert S[:, 0].tolist() == pytest.approx([1.5, 1.0]) and o[:, 0].tolist() == pytest.approx([3.0, 2.5])


def test_plain_expert_clamps_the_gate_above_and_the_up_lanes_on_both_sides():
    w = {"gate": torch.tensor([[1.0], [1.0], [1.0]], dtype=torch.float64) * torch.tensor([[9.0], [-9.0], [1.0]], dtype=torch.float64),
         "up": torch.tensor([[9.0], [-9.0], [1.0]], dtype=torch.float64), "down": torch.eye(3, dtype=torch.float64)}
    out = plain.clamped_expert(torch.ones(1, 1, dtype=torch.float64), w, "", 2.0)[0]
    sig = lambda x: 1.0 / (1.0 + math.exp(-x))
    assert out.tolist() == pytest.approx([2.0 * sig(3.404) * 3.0, -9.0 * sig(-9 * 1.702) * -1.0, sig(1.702) * 2.0])


def test_plain_norm_and_pass_entry_by_hand():
    x = torch.tensor([[0.5, -3.0]], dtype=torch.float64)
    got = plain.dynamic_tanh(x, torch.tensor(2.0, dtype=torch.float64), torch.tensor([2.0, 3.0]), torch.tensor([0.1, 0.2]))
    assert got[0].tolist() == pytest.approx([2.0 * math.tanh(1.0) + 0.1, 3.0 * math.tanh(-6.0) + 0.2])
    w_in = torch.tensor([[1.0, 0.0, 10.0, 0.0], [0.0, 1.0, 0.0, 100.0]], dtype=torch.float64)
    entered = plain.enter_pass(x, torch.tensor([[1.0, 2.0]], dtype=torch.float64), w_in, torch.tensor([0.25, 0.5]))
    assert entered[0].tolist() == pytest.approx([0.5 + 10.0 + 0.25, -3.0 + 200.0 + 0.5])
