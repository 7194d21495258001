"""The Kerudra configuration on the CPU: what it reads, what it refuses, the tensors it declares, the run order of a
loop, what the parts fold at load time, and the plain restatement's own mechanisms on cases small enough to do by
hand."""
import copy
import math

import pytest
import torch

import plain_kerudra as plain
from tiny_kerudra import TINY, make_folder
from tokenizer_b200.cache.manager import CachePlan
from tokenizer_b200.config import ConfigError, KerudraConfig, ModelSpec, config_from_dict
from tokenizer_b200.config.spec import PartSpec
from tokenizer_b200.parts.base import Runtime, build_part, part_class
from tokenizer_b200.parts.model import declared_tensors
from tokenizer_b200.weights import WeightStore


def test_the_registry_finds_the_design_by_its_name():
    cfg = TINY["a"]()[0]
    again = config_from_dict(cfg.to_dict())
    assert isinstance(again, KerudraConfig) and again.to_dict() == cfg.to_dict()
    assert config_from_dict(dict(cfg.to_dict(), architectures=["Kerudra"])).to_dict() == cfg.to_dict()


def test_declared_tensors_follow_the_sizes(tmp_path_factory):
    cfg = TINY["a"]()[0]
    shapes = {t.name: tuple(t.shape) for t in declared_tensors(cfg.model_spec())}
    assert shapes["embed"] == (301, 96) and "head" not in shapes and shapes["final.norm"] == (96,)
    for name in ("l0.hc1", "l0.hc2", "l3.hc1"):
        assert shapes[name + ".in"] == (3,) and shapes[name + ".out"] == (3,) and shapes[name + ".mix"] == (3, 3)
    assert shapes["l0.mix.q"] == (72, 96) and shapes["l0.mix.v"] == (48, 96) and shapes["l0.mix.g"] == (48, 96)
    assert shapes["l0.mix.i"] == (3, 96) and shapes["l0.mix.f.b"] == (3,) and shapes["l0.mix.norm"] == (48,)
    assert shapes["l1.mix.q"] == (5 * 24, 96) and shapes["l1.mix.dkv"] == (48, 96) and shapes["l1.mix.dkv.norm"] == (40,)
    assert shapes["l1.mix.uk"] == (80, 40) and shapes["l1.mix.uv"] == (120, 40) and shapes["l1.mix.g"] == (120, 96)
    assert shapes["l1.mix.o"] == (96, 120) and "l1.mix.dq" not in shapes and "l1.mix.sink" not in shapes
    # the attention's values are its keys: neither a matrix nor a bias of their own
    assert shapes["l2.mix.k"] == (64, 96) and shapes["l2.mix.k.b"] == (64,) and shapes["l2.mix.q.b"] == (192,)
    assert "l2.mix.v" not in shapes and "l2.mix.v.b" not in shapes
    assert shapes["l1.mlp.up"] == (104, 96) and shapes["l1.mlp.down"] == (96, 104) and "l1.mlp.gate" not in shapes
    # no feed-forward: neither its tensors nor the norm in front of it nor its connection
    assert not any(n.startswith(("l3.mlp", "l3.norm2", "l3.hc2")) for n in shapes)
    folder = make_folder(tmp_path_factory, "a")[0]
    WeightStore.from_folder(folder).check(declared_tensors(cfg.model_spec()))


@pytest.mark.parametrize("change,word", [
    (lambda r: r["layers"][0].update(type="other"), "unknown type"),
    (lambda r: r["layers"][0]["mixer"].pop("gate_cap"), "gate_cap"),
    (lambda r: r["layers"][0]["mixer"].update(gate_cap=0.0), "gate_cap"),
    (lambda r: r["layers"][1]["mixer"].pop("kv_rank"), "kv_rank"),
    (lambda r: r["layers"][1]["mixer"].pop("rot"), "rot"),
    (lambda r: r["layers"][1]["mixer"].update(mask={"size": 0}), "size"),
    (lambda r: r["layers"][1]["mixer"].update(mask={}), "size"),
    (lambda r: r["layers"][1]["mixer"]["rot"].update(dims=10), "rot.dims"),
    (lambda r: r["layers"][2]["mixer"].update(kv_heads=4), "do not divide"),
    (lambda r: r["layers"][2]["mixer"].update(vdim=16), "values are the keys"),
    (lambda r: r["layers"][2]["mixer"]["rot"].update(dims=34), "rot.dims"),
    (lambda r: r["layers"][2]["mixer"].pop("scale"), "scale"),
    (lambda r: r["layers"][0]["mlp"].update(kind="moe"), "dense"),
    (lambda r: r["layers"][0]["mlp"].pop("ff"), "ff"),
    (lambda r: r["loop"].update(stop=5), "loop"),
    (lambda r: r.update(streams=0), "streams"),
    (lambda r: r.pop("streams"), "streams"),
    (lambda r: r.pop("norm"), "norm"),
    (lambda r: r.update(layers=[]), "layers"),
])
def test_what_the_configuration_refuses(change, word):
    raw = copy.deepcopy(TINY["a"]()[0].to_dict())
    change(raw)
    with pytest.raises(ConfigError, match=word):
        KerudraConfig.from_dict(raw)


def test_a_loop_repeats_calls_that_keep_caches_and_states_of_their_own():
    spec = TINY["b"]()[0].model_spec()
    assert [c.layer for c in spec.order] == [0, 1, 2] * 2 + [3, 4, 5]
    assert all(c.cache is None and c.before is None for c in spec.order)
    raw = copy.deepcopy(TINY["b"]()[0].to_dict())
    raw.pop("loop")
    assert [c.layer for c in KerudraConfig.from_dict(raw).model_spec().order] == [0, 1, 2, 3, 4, 5]
    raw["loop"] = {"start": 2, "stop": 2, "times": 5}
    assert [c.layer for c in KerudraConfig.from_dict(raw).model_spec().order] == [0, 1, 2, 3, 4, 5]


def test_the_model_spec_names_parts_that_other_designs_can_use():
    spec = TINY["a"]()[0].model_spec()
    assert spec.streams == 3
    assert [l.block for l in spec.layers] == ["connected_streams"] * 3 + ["connected_streams_mixer_only"]
    assert [l.parts["mixer"].kind for l in spec.layers] == ["matrix_memory", "latent_attention", "gqa_rotary", "latent_attention"]
    latent = spec.layers[1].parts["mixer"].params
    assert (latent["window"], latent["q_rank"], latent["output_gate"], latent["position"].kind) == (19, None, True, "rope_interleaved")
    attn = spec.layers[2].parts["mixer"].params
    assert (attn["values_are_keys"], attn["bias"], attn["window"], attn["position"].kind) == (True, True, None, "rope_half")
    assert spec.layers[0].parts["mixer"].params["gate_cap"] == 9.0
    assert spec.layers[1].parts["feed_forward"].params["activation"] == "relu_squared"
    assert spec.layers[1].parts["feed_forward_connection"].params == {"streams": 3, "mult": 0.6}
    assert spec.final_norm.params["gain_scale"] == 0.3 and spec.embedding.params["scale"] == 9.0
    assert spec.head.params["tied_to"] == "embed"
    plain_numbers = TINY["c"]()[0]
    assert (plain_numbers.residual_mult, plain_numbers.embedding_scale, plain_numbers.logit_scale) == (1.0, 1.0, 1.0)
    assert plain_numbers.model_spec().layers[2].parts["mixer"].params["position"] is None
    assert TINY["d"]()[0].model_spec().layers[4].parts["mixer"].params["window"] is None


def test_a_model_with_streams_takes_no_injections():
    from tokenizer_b200.config.spec import LayerCall
    spec = TINY["a"]()[0].model_spec()
    entry = PartSpec("pass_entry", {"tensor": "t", "passes": 1, "hidden_size": 96, "index": 0}, "t")
    fields = {k: getattr(spec, k) for k in spec.__dataclass_fields__}
    with pytest.raises(ConfigError, match="one stream"):
        ModelSpec(**dict(fields, order=(LayerCall(0, before=entry),))).validate()
    with pytest.raises(ConfigError, match="at least one stream"):
        ModelSpec(**dict(fields, streams=0)).validate()


def test_the_cache_keeps_latents_in_one_plane_keys_in_two_and_matrices_in_slots():
    spec = TINY["a"]()[0].model_spec()
    store = _store(spec)
    runtime = Runtime(torch.device("cpu"), torch.float32)
    needs = [build_part("mixer", spec.layers[c.layer].parts["mixer"], store, runtime).cache_need() for c in spec.order]
    plan = CachePlan(needs, 32, 8, 2)
    assert [(g.kv_heads, g.head_dim, g.planes, g.window, g.calls) for g in plan.groups] == \
        [(1, 48, 1, 19, [1, 3, 5]), (2, 32, 2, None, [2, 4, 6]), (1, 32, 1, 32, [7])]
    assert plan.state_calls == [0] and needs[0].state.shape == (-(-(3 * 17 * 24 + 3) // 4) * 4,)


def _store(spec, scale=1.0):
    g = torch.Generator().manual_seed(3)
    return WeightStore({t.name: (torch.randn(t.shape, generator=g) * scale) for t in declared_tensors(spec)})


@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
def test_queries_fold_into_the_latents_lanes_and_values_stay_apart(dtype):
    """q . k through the folded queries is q . (Wuk c) and the rotated lanes come through; the value weights are zero
    beyond the latent's lanes; blocks of the input product start on whole 8s of columns."""
    spec = TINY["a"]()[0].model_spec()
    store, params = _store(spec), spec.layers[1].parts["mixer"]
    part = build_part("mixer", params, store, Runtime(torch.device("cpu"), dtype))
    heads, dim, rot, rank, row, vdim = 5, 16, 8, 40, 48, 24
    assert part.row == row and part.q_at == 48 and part.g_at == 48 + heads * row and part.g_at % 8 == 0
    h, c = torch.randn(96, dtype=torch.float64), torch.randn(rank, dtype=torch.float64)
    folded = part.inputs.weight[part.q_at:part.g_at].double().view(heads, row, 96) @ h
    q = (store.get("l1.mix.q").double() @ h).view(heads, dim + rot)
    keys = (store.get("l1.mix.uk").double() @ c).view(heads, dim)
    want = (q[:, :dim] * keys).sum(-1)
    tol = 1e-5 if dtype == torch.float32 else 3e-2
    assert torch.allclose(folded[:, :rank] @ c, want, atol=tol * float(want.abs().max()) * 5)
    assert torch.allclose(folded[:, rank:rank + rot], q[:, dim:], atol=tol * 30) and float(folded[:, rank + rot:].abs().sum()) == 0
    values = part.values if dtype == torch.bfloat16 else part.values.transpose(1, 2)
    assert values.shape == (heads, vdim, row) and float(values[:, :, rank:].abs().sum()) == 0
    assert torch.allclose(values[:, :, :rank].reshape(heads * vdim, rank).float(), store.get("l1.mix.uv"), rtol=1e-2)


def test_a_latent_query_and_a_gate_go_together_too():
    """The two parameters are independent: a query latent with gated values, and neither."""
    base = dict(hidden_size=40, heads=2, dim=8, vdim=6, kv_rank=12, rot_dim=4, eps=1e-6, scale=0.3, window=None, sink=False,
                position=PartSpec("rope_interleaved", {"base": 100.0, "dims": 4}))
    for q_rank in (None, 10):
        for gate in (False, True):
            part = PartSpec("latent_attention", dict(base, q_rank=q_rank, output_gate=gate), "m")
            names = {t.name for t in part_class("mixer", "latent_attention").tensors(part)}
            assert ("m.q" in names) == (q_rank is None) and ("m.dq" in names) == (q_rank is not None) and ("m.g" in names) == gate
            tensors = {t.name: torch.randn(t.shape) for t in part_class("mixer", "latent_attention").tensors(part)}
            built = build_part("mixer", part, WeightStore(tensors), Runtime(torch.device("cpu"), torch.float32))
            columns = (0 if q_rank is None else 10) + 16
            if q_rank is None or gate:
                columns = -(-columns // 8) * 8 + (2 * 16 if q_rank is None else 0) + (16 if gate else 0)
            assert built.inputs.out_features == columns and built.out.in_features == (12 if gate else 2 * 16)


# ---- the plain restatement, by hand ---------------------------------------------------------------------
F64 = torch.float64


def test_plain_windows_count_as_the_design_says():
    seen = plain.seen_keys(6, 2)
    assert seen[4].tolist() == [False, False, False, True, True, False] and seen[0].tolist() == [True] + [False] * 5
    assert plain.seen_keys(3, 1)[2].tolist() == [False, False, True]
    assert plain.seen_keys(3)[2].tolist() == [True, True, True]


def test_plain_rotations_turn_the_pairs_of_their_layout():
    x = torch.tensor([[[1.0, 2.0, 3.0, 4.0, 5.0]]], dtype=F64)
    c, s, c2, s2 = math.cos(3.0), math.sin(3.0), math.cos(0.3), math.sin(0.3)
    half = plain.rotate(x, torch.tensor([3]), 100.0, 4, "half")[0, 0]
    assert half.tolist() == pytest.approx([c - 3 * s, 2 * c2 - 4 * s2, 3 * c + s, 4 * c2 + 2 * s2, 5.0])
    pairs = plain.rotate(x, torch.tensor([3]), 100.0, 4, "interleaved")[0, 0]
    assert pairs.tolist() == pytest.approx([c - 2 * s, 2 * c + s, 3 * c2 - 4 * s2, 4 * c2 + 3 * s2, 5.0])


def test_plain_matrix_memory_by_hand():
    q = torch.tensor([[1.0], [2.0], [1.0]], dtype=F64)
    k, v = torch.tensor([[3.0], [1.0], [0.0]], dtype=F64), torch.tensor([[5.0], [7.0], [0.0]], dtype=F64)
    log_in = torch.tensor([-1.0, 2.0, -30.0], dtype=F64)
    log_forget = torch.tensor([-0.5, -1.0, -2.0], dtype=F64)
    o, (S, n, top) = plain.matrix_memory(q, k, v, log_in, log_forget)
    # token 0: the maximum starts at 0, so it falls to -0.5 only and the write weighs exp(-0.5)
    w0 = math.exp(-0.5)
    assert float(o[0, 0]) == pytest.approx(15 * w0 / (max(3 * w0, math.exp(0.5)) + 1e-6))
    # token 1: the maximum rises to 2; what is there counts exp(-1 - 0.5 - 2)
    keep = math.exp(-3.5)
    s1, n1 = keep * 15 * w0 + 7, keep * 3 * w0 + 1
    assert float(o[1, 0]) == pytest.approx(2 * s1 / (max(2 * n1, math.exp(-2.0)) + 1e-6))
    # token 2 writes nothing; the maximum falls with the forget gate, the kept matrix is as it was
    assert float(top) == 0.0 and float(S) == pytest.approx(s1) and float(n) == pytest.approx(n1)
    assert float(o[2, 0]) == pytest.approx(s1 / (max(n1, 1.0) + 1e-6))


def test_plain_gates_are_capped_in_front_of_the_logarithm():
    w = {"i": torch.tensor([[100.0]], dtype=F64), "i.b": torch.tensor([1.0], dtype=F64),
         "f": torch.tensor([[-100.0]], dtype=F64), "f.b": torch.tensor([0.0], dtype=F64)}
    log_in, log_forget = plain.capped_gates(torch.ones(1, 1, dtype=F64), w, "", 4.0)
    assert float(log_in) == pytest.approx(4.0) and float(log_forget) == pytest.approx(-4.0 - math.log1p(math.exp(-4.0)))


def test_plain_streams_mix_from_the_old_ones_all_at_once():
    xs = torch.tensor([[[1.0]], [[10.0]]], dtype=F64)
    mix = torch.tensor([[2.0, 3.0], [5.0, 7.0]], dtype=F64)          # from the row to the column
    out = plain.mix_and_add(xs, mix, torch.tensor([0.5, -1.0], dtype=F64), torch.tensor([[100.0]], dtype=F64), 0.1)
    assert out[0, 0, 0].item() == pytest.approx(2 + 50 + 5) and out[1, 0, 0].item() == pytest.approx(3 + 70 - 10)
    assert plain.combine(xs, torch.tensor([4.0, -1.0], dtype=F64)).item() == pytest.approx(-6.0)


def test_plain_values_are_the_keys_before_the_rotation():
    m = {"heads": 1, "kv_heads": 1, "dim": 2, "vdim": 2, "scale": 0.0, "rot": {"base": 10.0, "dims": 2}}
    w = {"q": torch.eye(2, dtype=F64), "q.b": torch.zeros(2, dtype=F64), "k": torch.eye(2, dtype=F64),
         "k.b": torch.tensor([1.0, 0.0], dtype=F64), "o": torch.eye(2, dtype=F64)}
    out = plain.shared_key_value_attention(torch.tensor([[1.0, 2.0], [3.0, 4.0]], dtype=F64), w, "", m)
    assert out[1].tolist() == pytest.approx([3.0, 3.0])              # the mean of (2, 2) and (4, 4)
