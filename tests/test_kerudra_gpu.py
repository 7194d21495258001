"""The Kerudra decoder on the GPU against the plain restatement: each mechanism's kernels alone, with weights or
inputs made so that a fault shows (a key just outside a window, a far write in a matrix, gates that open and close), then
whole models (four tiny configurations of unlike sizes) whole, token by token, in portions, in mixed batches on few pages
and slots, and through the generation entry point."""
import numpy as np
import pytest
import torch

import plain_kerudra as plain
import replay_util as ru
from tiny import random_ids
from tiny_kerudra import SHARPEN, TINY, make_folder, reference_logits

pytestmark = pytest.mark.gpu
DEV = "cuda:0"


def ops():
    from tokenizer_b200.kernels import ops as o
    return o


def rnd(*shape, seed=0, dtype=torch.float32, scale=1.0):
    g = torch.Generator().manual_seed(seed)
    return (torch.randn(*shape, generator=g) * scale).to(dtype).to(DEV)


def close(got, want, dtype, what="", tol=None):
    got, want = got.detach().float().cpu(), want.detach().float().cpu()
    tol = tol if tol is not None else (2e-5 if dtype == torch.float32 else 2e-2)
    bound = tol * max(1.0, float(want.abs().max()))
    err = float((got - want).abs().max())
    assert torch.isfinite(got).all() and err <= bound, f"{what}: max |diff| {err:.3e} > {bound:.3e}"


def ints(values):
    return torch.tensor(list(values), dtype=torch.int32, device=DEV)


def part_of(category, kind, params, tensors, dtype=torch.float32, prefix="p"):
    from tokenizer_b200.config.spec import PartSpec
    from tokenizer_b200.parts.base import Runtime, build_part
    from tokenizer_b200.weights.store import WeightStore
    return build_part(category, PartSpec(kind, params, prefix), WeightStore(tensors), Runtime(torch.device(DEV), dtype))


def double(t):
    return t.double().cpu()


# ---- the streams ----------------------------------------------------------------------------------------
@pytest.mark.parametrize("out_dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("streams,width", [(1, 50), (2, 320), (3, 2048), (4, 4100), (5, 9001), (8, 96)])
@pytest.mark.parametrize("form", ["bf16", "f32", "partials"])
def test_the_step_between_two_sublayers(streams, width, form, out_dtype):
    """Every stream anew from all the old ones and the output, the weighted sum of the new ones and its norm; from
    streams that are still equal and from streams that are not; the sum of the wanted rows alone."""
    o = ops()
    n, eps = 5, 1e-3
    gain = rnd(width, seed=2) + 1.0
    y = rnd(3, n, width, seed=4) if form == "partials" else rnd(n, width, seed=4, dtype=torch.bfloat16 if form == "bf16" else torch.float32)
    mix, share, read = rnd(streams, streams, seed=5), rnd(streams, seed=6), rnd(streams, seed=7)
    added = double(y).sum(0) if form == "partials" else double(y)
    for equal in (True, False):
        x = rnd(n, width, seed=1, scale=2.0) if equal else rnd(n, streams, width, seed=8, scale=2.0)
        old = double(x).expand(streams, n, width) if equal else double(x).transpose(0, 1)
        want = plain.mix_and_add(old, double(mix), double(share), added, 1.0)
        u = plain.combine(want, double(read))
        # nothing pending: the weighted sum of what is there
        h = torch.full((n, width), float("nan"), dtype=out_dtype, device=DEV)
        same = o.streams_step(x, streams, read=read, gain=gain, eps=eps, out=h)
        assert same is x
        close(h, plain.rms(plain.combine(old, double(read)), eps) * double(gain), out_dtype, "before")
        # the wanted rows' sum, what is pending counted in; the streams stay
        rows, kept = ints([4, 0, 4]), x.clone()
        some = torch.full((3, width), float("nan"), dtype=out_dtype, device=DEV)
        o.streams_step(x, streams, y, mix, share, gain=gain, eps=eps, out=some, rows=rows)
        close(some, (plain.rms(want.sum(0), eps) * double(gain))[[4, 0, 4]], out_dtype, "wanted rows")
        assert torch.equal(x, kept)
        # without a norm, then with
        raw = torch.full((n, width), float("nan"), device=DEV)
        first = o.streams_step(x.clone(), streams, y, mix, share, read=read, out=raw)
        close(raw, u, torch.float32, "the weighted sum")
        h.fill_(float("nan"))
        new = o.streams_step(x.clone(), streams, y, mix, share, read=read, gain=gain, eps=eps, out=h)
        assert tuple(new.shape) == (n, streams, width) and torch.equal(new, first)
        close(new.transpose(0, 1), want, torch.float32, "the streams")
        close(h, plain.rms(u, eps) * double(gain), out_dtype, "the norm")
        # the update alone, in place once the streams differ
        again = o.streams_step(x.clone(), streams, y, mix, share)
        assert torch.equal(again, new)


def test_the_bundle_keeps_one_output_pending():
    from tokenizer_b200.parts.base import Runtime, StreamBundle
    runtime = Runtime(torch.device(DEV), torch.float32)
    n, width, streams = 4, 40, 3
    tensors = {f"p{i}.{name}": rnd(*shape, seed=10 * i + j).cpu() for i in range(2)
               for j, (name, shape) in enumerate((("in", (streams,)), ("out", (streams,)), ("mix", (streams, streams))))}
    links = [part_of("connection", "stream_connection", {"streams": streams, "mult": 0.3}, tensors, prefix=f"p{i}") for i in range(2)]
    norm = part_of("norm", "rms_norm", {"size": width, "eps": 1e-5, "tensor": "g"}, {"g": torch.rand(width) + 0.5})
    layer = part_of("norm", "layer_norm", {"size": width, "eps": 1e-5, "tensor": "g"},
                    {"g": torch.rand(width) + 0.5, "g.b": torch.rand(width)})
    x, y0, y1 = rnd(n, width, seed=1), rnd(n, width, seed=2), rnd(n, width, seed=3)
    bundle = StreamBundle(x.clone(), streams)
    w = {k: v.double() for k, v in tensors.items()}
    xs = double(x).expand(streams, n, width)
    bundle.read(norm, links[0], runtime)
    bundle.add(y0, links[0])
    bundle.add(y1, links[1])
    for i, y in enumerate((y0, y1)):
        xs = plain.mix_and_add(xs, w[f"p{i}.mix"], w[f"p{i}.out"], double(y), 0.3)
    # a norm that no kernel of the streams folds in
    bundle.add(y0, links[1])
    xs = plain.mix_and_add(xs, w["p1.mix"], w["p1.out"], double(y0), 0.3)
    u = plain.combine(xs, w["p0.in"])
    want = (u - u.mean(-1, keepdim=True)) / torch.sqrt(u.var(-1, unbiased=False, keepdim=True) + 1e-5) * double(layer.gain) + double(layer.bias)
    close(bundle.read(layer, links[0], runtime), want, torch.float32, "a layer norm")
    close(bundle.flush(), xs.sum(0), torch.float32, "the sum")
    bundle.add(y1, links[0])
    xs = plain.mix_and_add(xs, w["p0.mix"], w["p0.out"], double(y1), 0.3)
    close(bundle.finish(norm, ints([3, 1]), runtime), (plain.rms(xs.sum(0), 1e-5) * double(norm.gain))[[3, 1]], torch.float32, "the wanted rows")


# ---- attention: values that are the keys, the latent with its queries and its gated values ------------------
@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("layout", ["half", "interleaved"])
@pytest.mark.parametrize("heads,kv,dim,dims", [(6, 2, 32, 16), (4, 4, 64, 64), (5, 1, 6, 0), (3, 3, 10, 4), (2, 1, 128, 40)])
def test_values_are_the_keys_as_projected(heads, kv, dim, dims, layout, dtype):
    o = ops()
    n, row, extra = 6, -(-dim // 16) * 16, 4
    proj, bias = rnd(n, extra + (heads + kv) * dim + 8, seed=11), rnd((heads + kv) * dim, seed=12)
    pos, slots = [0, 1, 2, 900, 77, 40000], [3, 0, 5, 1, 7, 2]
    freq = torch.tensor([300.0 ** (-2.0 * i / dims) for i in range(dims // 2)], dtype=torch.float64, device=DEV) if dims else None
    q = torch.full((n, heads * row), float("nan"), dtype=dtype, device=DEV)
    pools = [torch.full((8, kv, row), float("nan"), dtype=dtype, device=DEV) for _ in range(2)]
    o.qkv_rotate_store(proj, extra, bias, freq, dims, ints(pos), ints(slots), ints([0] * n), q, pools[0], pools[1],
                       heads, kv, dim, dim, row, layout=layout, values_are_keys=True)
    p = double(proj)[:, extra:extra + (heads + kv) * dim] + double(bias)
    turn = lambda x: plain.rotate(x, torch.tensor(pos), 300.0, dims, layout) if dims else x
    keys = p[:, heads * dim:].view(n, kv, dim)
    close(q.view(n, heads, row)[:, :, :dim], turn(p[:, :heads * dim].view(n, heads, dim)), dtype, "queries")
    close(pools[0][slots][:, :, :dim], turn(keys), dtype, "keys")
    close(pools[1][slots][:, :, :dim], keys, dtype, "values")
    for t in (q.view(n, heads, row)[:, :, dim:], pools[0][slots][:, :, dim:], pools[1][slots][:, :, dim:]):
        assert t.numel() == 0 or float(t.float().abs().max()) == 0.0
    assert torch.isnan(pools[0][4].float()).all() and torch.isnan(pools[1][6].float()).all()       # slots of nobody


@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("heads,rank,rot,dims", [(5, 40, 8, 8), (1, 11, 2, 2), (9, 96, 32, 32), (3, 150, 10, 10), (2, 20, 12, 4)])
def test_the_latents_row_and_the_queries_in_its_lanes(heads, rank, rot, dims, dtype):
    o = ops()
    n, row, eps = 6, -(-(rank + rot) // 16) * 16, 1e-3
    c_at, q_at = 3, 3 + rank + rot
    proj, gain = rnd(n, q_at + heads * row + 5, seed=21), rnd(rank, seed=22) + 1.0
    pos, slots = [0, 5, 123456, 900, 77, 1], [1, -1, 6, 0, 2, 5]
    freq = torch.tensor([700.0 ** (-2.0 * i / dims) for i in range(dims // 2)], dtype=torch.float64, device=DEV)
    q = torch.full((n, heads * row), float("nan"), dtype=dtype, device=DEV)
    pool = torch.full((8, 1, row), float("nan"), dtype=dtype, device=DEV)
    o.latent_rotate_store(proj, c_at, q_at, heads, rank, rot, dims, row, gain, eps, freq, ints(pos), ints([0] * 5 + [-1]),
                          ints(slots), q, pool)
    p, where = double(proj), torch.tensor(pos)
    want_q = p[:, q_at:q_at + heads * row].view(n, heads, row).clone()
    want_q[..., rank:rank + rot] = plain.rotate(want_q[..., rank:rank + rot], where, 700.0, dims, "interleaved")
    close(q.view(n, heads, row)[:5], want_q[:5], dtype, "queries")
    assert torch.isnan(q[5].float()).all() and torch.isnan(pool[[3, 4, 5, 7]].float()).all()       # an idle row, slots of nobody
    c = plain.rms(p[:, c_at:c_at + rank], eps) * double(gain)
    shared = plain.rotate(p[:, None, c_at + rank:c_at + rank + rot], where, 700.0, dims, "interleaved")[:, 0]
    for t in (0, 2, 3, 4):
        close(pool[slots[t], 0, :rank], c[t], dtype, "latent")
        close(pool[slots[t], 0, rank:rank + rot], shared[t], dtype, "shared key part")
        assert row == rank + rot or float(pool[slots[t], 0, rank + rot:].float().abs().max()) == 0.0
    # without slots only the queries are written
    before = pool.clone()
    o.latent_rotate_store(proj, c_at, q_at, heads, rank, rot, dims, row, gain, eps, freq, ints(pos), ints([0] * n), None, q, pool)
    assert torch.equal(pool.nan_to_num(), before.nan_to_num())


@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("heads,vdim,row", [(4, 64, 128), (1, 7, 16), (5, 24, 48), (3, 130, 80), (2, 128, 576)])
def test_values_from_weighted_latents_through_a_gate(heads, vdim, row, dtype):
    o = ops()
    for n in (1, 16, 63, 65, 200):
        mixed, gate = rnd(n, heads * row, seed=31, dtype=dtype), rnd(n, 8 + heads * vdim, seed=32, scale=2.0)
        w = rnd(heads, vdim, row, seed=33, dtype=dtype, scale=row ** -0.5)
        out = torch.full((n, heads * vdim), float("nan"), dtype=dtype, device=DEV)
        o.latent_values(mixed, w if dtype == torch.bfloat16 else w.transpose(1, 2).contiguous(), gate, 8, heads, vdim, row, out)
        want = torch.einsum("hvr,thr->thv", double(w), double(mixed).view(n, heads, row)).reshape(n, -1)
        close(out, want * plain.sigmoid(double(gate)[:, 8:8 + heads * vdim]), dtype, f"{n} rows")


def run_engine(raw, weights, steps, dtype, max_tokens, page, max_requests=2, use_graphs=True):
    """Steps through an engine on tensors handed over as they are; {step: logits}."""
    from tokenizer_b200.config import KerudraConfig
    from tokenizer_b200.engine import Engine, StepEntry
    from tokenizer_b200.engine.step import parse_dtype
    from tokenizer_b200.parts.base import Runtime
    from tokenizer_b200.parts.model import DecoderModel
    from tokenizer_b200.weights.store import WeightStore
    model = DecoderModel(KerudraConfig.from_dict(raw).model_spec(), WeightStore(dict(weights)), Runtime(torch.device(DEV), parse_dtype(dtype)))
    engine = Engine(model, num_pages=-(-max_tokens // page), page_size=page, max_requests=max_requests, use_graphs=use_graphs)
    live, out = {}, {}
    for record in steps:
        entries = []
        for item in record["entries"]:
            if item["id"] not in live:
                live[item["id"]] = engine.cache.open(item["id"])
            engine.cache.reserve(live[item["id"]], len(item["tokens"]))
            entries.append(StepEntry(live[item["id"]], item["tokens"], item.get("want", [])))
        logits = engine.step(entries)
        if logits.shape[0]:
            out[record["step"]] = logits.cpu()
        for name in record.get("end", []):
            engine.cache.close(live.pop(name))
    engine.check()
    return out


def needle_model(kind, size, dim, seed=0):
    """One layer of attention whose asking token (id 1) finds the needle (id 0) wherever it sees it: lane 0 of the
    stream marks the needle, lane 1 the asker, and a query and key lane that no rotation turns carries a score far above
    all others.  Returns (configuration, weights)."""
    from tiny_kerudra import attention, config, latent
    from tokenizer_b200.parts.model import declared_tensors
    width = 64
    if kind == "latent":
        cfg = config([latent(2, dim, 8, 16, dim, 1.0, 100.0, size=size)], vocab=30, width=width, eps=1e-6, streams=2, mult=0.8)
    else:
        cfg = config([attention(4, 2, dim, 1.0, rot=(100.0, 8))], vocab=30, width=width, eps=1e-6, streams=2, mult=0.8)
    g = torch.Generator().manual_seed(seed)
    w = {t.name: (torch.randn(t.shape, generator=g) * 0.3).to(torch.bfloat16) for t in declared_tensors(cfg.model_spec())}
    w["embed"][:, :2] = 0.0
    w["embed"][0, 0] = w["embed"][1, 1] = 3.0
    w["l0.norm1"] = torch.ones(width, dtype=torch.bfloat16)
    for name in ("l0.mix.q", "l0.mix.k", "l0.mix.dkv", "l0.mix.uk"):
        if name in w:
            w[name] = w[name] * 0.1
            if name != "l0.mix.uk":
                w[name][:, :2] = 0.0
    if kind == "latent":
        w["l0.mix.dkv.norm"] = torch.ones(dim, dtype=torch.bfloat16)
        w["l0.mix.q"].view(2, dim + 8, width)[:, 3, 1] = 8.0          # an unrotated query lane of both heads
        w["l0.mix.dkv"][5, 0] = 8.0                                    # one lane of the latent
        w["l0.mix.uk"].view(2, dim, dim)[:, 3, 5] = 2.0
    else:
        w["l0.mix.q"].view(4, dim, width)[:, dim - 1, 1] = 8.0         # behind the rotated lanes
        w["l0.mix.k"].view(2, dim, width)[:, dim - 1, 0] = 8.0
    return cfg, w


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("alone", [True, False])
@pytest.mark.parametrize("kind,size,dim", [("latent", 40, 24), ("latent", 130, 56), ("latent", 1, 40), ("latent", 64, 136),
                                           ("attention", None, 32), ("attention", None, 64), ("attention", None, 128)])
def test_a_key_that_stands_out_far_back_and_at_the_windows_edge(kind, size, dim, alone, dtype):
    """The asker at the end of hundreds of tokens, in a prompt or decoded alone; the needle far back, just inside and
    just outside the window, on both sides of a page's border and at the start."""
    from tokenizer_b200.config import KerudraConfig
    cfg, weights = needle_model(kind, size, dim)
    raw, w64 = cfg.to_dict(), {k: v.double() for k, v in weights.items()}
    n, page = 420, 16
    filler = [2 + (7 * i) % 28 for i in range(n)]
    places = [n - size, n - size - 1, n - 1 - size // 2] if size is not None else [0, 15, 16, 200, n - 2]
    base = plain.forward(raw, w64, filler[:-1] + [1])[-1]
    for at in places:
        ids = list(filler)
        if at < n - 1:
            ids[at] = 0
        ids[-1] = 1
        want = plain.forward(raw, w64, ids)[-1]
        steps = [{"step": 0, "entries": [{"id": "r", "tokens": ids if not alone else ids[:-1], "want": [n - 1] if not alone else []}]}]
        if alone:
            steps.append({"step": 1, "entries": [{"id": "r", "tokens": ids[-1:], "want": [0]}]})
        got = run_engine(raw, weights, steps, dtype, 512, page)[int(alone)]
        close(got[0], want, torch.float32 if dtype == "float32" else torch.bfloat16, f"needle at {at}", 1e-4 if dtype == "float32" else 3e-2)
        seen = at < n - 1 and (size is None or n - 1 - at < size)
        moved = float((want - base).abs().max()) / float(base.abs().max())
        assert moved > 0.1 if seen else moved < 1e-9 or at == n - 1, f"the needle at {at} {'counts' if seen else 'does not count'}: {moved}"


# ---- the matrix memory ------------------------------------------------------------------------------------
MEMORY_SIZES = [(3, 24, 16), (1, 6, 10), (2, 128, 128), (4, 64, 96), (2, 136, 8), (1, 256, 20), (3, 7, 5), (1, 1, 1), (2, 32, 33), (1, 100, 63)]


class Memory:
    """A product's columns and a state for the memory's kernels, and the plain answer a head."""

    def __init__(self, heads, dim, vdim, total, seed, slots=5, cap=7.0):
        self.heads, self.dim, self.vdim, self.cap = heads, dim, vdim, cap
        self.at = dict(q=4, k=4 + heads * dim + 3)
        self.at["v"] = self.at["k"] + heads * dim
        self.at["g"] = self.at["v"] + heads * vdim + 1
        self.at["i"] = self.at["g"] + heads * vdim
        self.at["f"] = self.at["i"] + heads + 2
        self.proj = rnd(total, self.at["f"] + heads + 3, seed=seed)
        self.proj[:, self.at["i"]:self.at["i"] + heads] *= 4.0                 # gates that open and close
        self.proj[:, self.at["f"]:self.at["f"] + heads] *= 3.0
        self.ib, self.fb = rnd(heads, seed=seed + 1), rnd(heads, seed=seed + 2) + 2.0
        self.gain = rnd(heads * vdim, seed=seed + 3) + 1.0
        self.m_off = heads * (vdim + 1) * dim
        self.state = torch.zeros(slots, -(-(self.m_off + heads) // 4) * 4, device=DEV)

    def gates(self, sub, spans, who):
        gates = torch.full((3, self.heads, sub.shape[0] + 2), float("nan"), device=DEV)
        ops().mlstm_gates(sub, self.at["i"], self.at["f"], self.ib, self.fb, self.cap, self.heads, self.state, self.m_off, spans, who, gates)
        return gates

    def portion(self, sub, spans, who, row_req, eps, dtype, segments=None):
        o, n = ops(), sub.shape[0]
        gates = self.gates(sub, spans, who)
        y = torch.full((n, self.heads * self.vdim), float("nan"), device=DEV)
        yn = torch.full((n, self.heads), float("nan"), device=DEV)
        o.mlstm_scan(sub, self.at["q"], self.at["k"], self.at["v"], self.heads, self.dim, self.vdim, gates, self.state, spans, who, y, yn, segments)
        out = torch.full((n, self.heads * self.vdim), float("nan"), dtype=dtype, device=DEV)
        o.mlstm_out_norm(y, yn, gates, sub, self.at["g"], self.gain, eps, self.heads, self.vdim, row_req, out)
        return out

    def plain(self, proj, eps):
        """(outputs [T, heads, vdim], [(S, n, maximum)] a head) of one request's rows from its start."""
        p, heads, dim, vdim = double(proj), self.heads, self.dim, self.vdim
        n = p.shape[0]
        take = lambda name, lanes: p[:, self.at[name]:self.at[name] + heads * lanes].view(n, heads, lanes)
        w = {"i": torch.eye(heads, dtype=torch.float64), "f": torch.eye(heads, dtype=torch.float64), "i.b": double(self.ib), "f.b": double(self.fb)}
        log_in = plain.capped_gates(take("i", 1)[..., 0], w, "", self.cap)[0]
        log_forget = plain.capped_gates(take("f", 1)[..., 0], w, "", self.cap)[1]
        outs, states = [], []
        for a in range(heads):
            o, state = plain.matrix_memory(take("q", dim)[:, a] * dim ** -0.5, take("k", dim)[:, a], take("v", vdim)[:, a], log_in[:, a], log_forget[:, a])
            outs.append(plain.rms(o, eps))
            states.append(state)
        y = torch.stack(outs, 1).reshape(n, -1) * double(self.gain) * plain.sigmoid(take("g", vdim).reshape(n, -1))
        return y, states

    def check_state(self, slot, states, tol=2e-5):
        mats = self.state[slot, :self.m_off].view(self.heads, self.vdim + 1, self.dim)
        for a, (S, n, top) in enumerate(states):
            close(mats[a, :self.vdim].t(), S, torch.float32, f"the matrix of head {a}", tol)
            close(mats[a, self.vdim], n, torch.float32, f"the normaliser of head {a}", tol)
            close(self.state[slot, self.m_off + a], top, torch.float32, f"the maximum of head {a}", tol)


@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("heads,dim,vdim", MEMORY_SIZES)
def test_the_memory_in_portions_carries_matrix_normaliser_and_maximum(heads, dim, vdim, dtype):
    """Three requests in slots that are not their indices, cut into portions of 1, 2, 3 and many rows, an idle request
    as a padded step has it, against the recurrence token by token."""
    lengths, slots, eps = [37, 1, 150], [2, 0, 3], 1e-4
    cuts = [[0, 1, 3, 4, 7, 20, 37], [0, 1], [0, 129, 132, 133, 135, 150]]
    total = sum(lengths)
    m = Memory(heads, dim, vdim, total, 30)
    m.state[1] = 7.0                                       # a slot nobody holds must stay as it is
    out = torch.full((total, heads * vdim), float("nan"), dtype=dtype, device=DEV)
    starts = np.concatenate(([0], np.cumsum(lengths)))
    for i in range(max(len(c) for c in cuts) - 1):
        rows, spans, who, req = [], [0], [], []
        for r in range(3):
            if i + 1 < len(cuts[r]):
                here = list(range(starts[r] + cuts[r][i], starts[r] + cuts[r][i + 1]))
                rows += here
                req += [len(who)] * len(here)
                spans.append(len(rows))
                who.append(slots[r])
        idx = torch.tensor(rows, device=DEV)
        out[idx] = m.portion(m.proj[idx].contiguous(), ints(spans + [spans[-1]]), ints(who + [0]), ints(req), eps, dtype,
                             segments=(None, 1, 3)[i % 3])
    for r in range(3):
        want, states = m.plain(m.proj[starts[r]:starts[r + 1]], eps)
        close(out[starts[r]:starts[r + 1]], want, dtype, f"request {r}", 1e-4 if dtype == torch.float32 else 2e-2)
        m.check_state(slots[r], states)
    assert torch.all(m.state[1] == 7.0) and torch.all(m.state[4] == 0.0)


@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("heads,dim,vdim", MEMORY_SIZES)
def test_a_step_of_single_tokens_through_the_memory_in_one_kernel(heads, dim, vdim, dtype):
    """Token by token, three requests of which one is absent from some steps, an idle row at the end."""
    eps, slots = 1e-4, [3, 0, 1]
    m = Memory(heads, dim, vdim, 1, 40)
    width, a = m.proj.shape[1], m.at
    fed = {r: [] for r in range(3)}
    for step in range(12):
        present = [0, 1, 2] if step % 3 else [0, 2]
        proj = rnd(len(present) + 1, width, seed=50 + step, scale=2.0)
        out = torch.full((len(present) + 1, heads * vdim), float("nan"), dtype=dtype, device=DEV)
        ops().mlstm_step(proj, a["q"], a["k"], a["v"], a["g"], a["i"], a["f"], m.ib, m.fb, m.cap, heads, dim, vdim, m.gain, eps,
                         m.state, m.m_off, ints(list(range(len(present))) + [-1]), ints([slots[r] for r in present] + [2]), out)
        assert torch.isnan(out[-1].float()).all()
        for i, r in enumerate(present):
            fed[r].append(proj[i])
            want, _ = m.plain(torch.stack(fed[r]), eps)
            close(out[i], want[-1], dtype, f"step {step} request {r}", 1e-4 if dtype == torch.float32 else 2e-2)
    for r in range(3):
        m.check_state(slots[r], m.plain(torch.stack(fed[r]), eps)[1])
    assert float(m.state[2].abs().max()) == 0.0 and float(m.state[4].abs().max()) == 0.0


@pytest.mark.parametrize("segments", [1, 2, 7, 16])
@pytest.mark.parametrize("heads,dim,vdim", [(2, 64, 32), (1, 24, 40), (1, 128, 63)])
def test_segments_side_by_side_give_what_one_run_gives(heads, dim, vdim, segments):
    lengths, eps = [700, 3, 90], 1e-5
    total = sum(lengths)
    m = Memory(heads, dim, vdim, total, 60)
    starts = np.concatenate(([0], np.cumsum(lengths))).tolist()
    req = [r for r in range(3) for _ in range(lengths[r])]
    out = m.portion(m.proj, ints(starts), ints([1, 2, 4]), ints(req), eps, torch.float32, segments)
    for r, slot in enumerate([1, 2, 4]):
        want, states = m.plain(m.proj[starts[r]:starts[r + 1]], eps)
        close(out[starts[r]:starts[r + 1]], want, torch.float32, f"request {r}", 1e-4)
        m.check_state(slot, states)


CHUNK_SIZES = [(3, 24, 16), (1, 6, 10), (2, 128, 128), (4, 64, 96), (2, 100, 8), (3, 7, 5), (1, 1, 1), (2, 32, 33), (1, 120, 63), (2, 32, 48)]


@pytest.mark.parametrize("heads,dim,vdim", CHUNK_SIZES)
def test_chunks_on_tensor_cores_carry_the_same_state(heads, dim, vdim):
    """Portions cut in the middle of a chunk, on its border, of one token and of many chunks, three requests side by side
    and an idle one: q, k and v as bfloat16 numbers, everything else to 32-bit accuracy (the state tells, the outputs
    are rounded)."""
    o, eps = ops(), 1e-4
    lengths, slots = [200, 64, 331], [2, 0, 3]
    cuts = [[0, 1, 64, 128, 131, 200], [0, 64], [0, 129, 193, 194, 330, 331]]
    total = sum(lengths)
    m = Memory(heads, dim, vdim, total, 110)
    for name, lanes in (("q", dim), ("k", dim), ("v", vdim)):
        part = m.proj[:, m.at[name]:m.at[name] + heads * lanes]
        part.copy_(part.bfloat16().float())
    m.state[1] = 7.0
    out = torch.full((total, heads * vdim), float("nan"), dtype=torch.bfloat16, device=DEV)
    starts = np.concatenate(([0], np.cumsum(lengths)))
    assert o.mlstm_chunks_supported(dim, vdim)
    for i in range(5):
        rows, spans, who = [], [0], []
        for r in range(3):
            if i + 1 < len(cuts[r]):
                rows += list(range(starts[r] + cuts[r][i], starts[r] + cuts[r][i + 1]))
                spans.append(len(rows))
                who.append(slots[r])
        idx = torch.tensor(rows, device=DEV)
        sub, spans, who = m.proj[idx].contiguous(), ints(spans + [spans[-1]]), ints(who + [0])
        gates = torch.full((3, heads, len(rows) + 1), float("nan"), device=DEV)
        start = torch.full((who.shape[0], heads), float("nan"), device=DEV)
        o.mlstm_gates(sub, m.at["i"], m.at["f"], m.ib, m.fb, m.cap, heads, m.state, m.m_off, spans, who, gates, start)
        y = torch.full((len(rows), heads * vdim), float("nan"), dtype=torch.bfloat16, device=DEV)
        o.mlstm_chunks(sub, m.at["q"], m.at["k"], m.at["v"], m.at["g"], heads, dim, vdim, gates, start, m.gain, eps, m.state, spans, who, y)
        out[idx] = y
    for r in range(3):
        want, states = m.plain(m.proj[starts[r]:starts[r + 1]], eps)
        close(out[starts[r]:starts[r + 1]], want, torch.bfloat16, f"request {r}", 6e-3)
        m.check_state(slots[r], states, 1e-5)
    assert torch.all(m.state[1] == 7.0) and torch.all(m.state[4] == 0.0)


@pytest.mark.parametrize("forget", [-14.0, -3.0, 14.0])
def test_chunks_keep_their_digits_under_closed_and_open_gates(forget):
    """Forget gates that all but close (their logarithms add up to hundreds inside a chunk and cancel) or stay open, for
    every token: the state to 32-bit accuracy, and a write of the chunk before last that an open gate keeps."""
    o, heads, dim, vdim, total, eps = ops(), 2, 64, 32, 300, 1e-4
    m = Memory(heads, dim, vdim, total, 120, cap=15.0)
    m.proj = m.proj.bfloat16().float()
    m.fb.fill_(4.0 * forget)
    gates, start = torch.empty(3, heads, total, device=DEV), torch.empty(1, heads, device=DEV)
    spans, who = ints([0, total]), ints([1])
    o.mlstm_gates(m.proj, m.at["i"], m.at["f"], m.ib, m.fb, m.cap, heads, m.state, m.m_off, spans, who, gates, start)
    y = torch.empty(total, heads * vdim, dtype=torch.bfloat16, device=DEV)
    o.mlstm_chunks(m.proj, m.at["q"], m.at["k"], m.at["v"], m.at["g"], heads, dim, vdim, gates, start, m.gain, eps, m.state, spans, who, y)
    want, states = m.plain(m.proj, eps)
    assert float(start.abs().max()) == 0.0
    close(y, want, torch.bfloat16, "outputs", 6e-3)
    m.check_state(1, states, 1e-5)


def test_a_write_behind_a_thousand_tokens_and_a_maximum_that_starts_at_zero():
    """One token writes with an open input gate; every later one keeps (forget gate near one) and hardly writes; the last
    reads it back, through portions' borders.  And: with every input gate nearly shut the maximum falls from zero by the
    forget gates alone, where a maximum from minus infinity would follow the input gates."""
    heads, dim, vdim, total, eps = 1, 64, 16, 1003, 1e-9
    m = Memory(heads, dim, vdim, total, 70, cap=30.0)
    m.ib.zero_(), m.fb.zero_()
    m.proj[:, m.at["i"]] = -25.0
    m.proj[:, m.at["f"]] = 25.0
    m.proj[3, m.at["i"]] = 10.0
    m.proj[:, m.at["k"]:m.at["k"] + dim] *= 0.05
    m.proj[3, m.at["k"]:m.at["k"] + dim] = m.proj[total - 1, m.at["q"]:m.at["q"] + dim]
    outs, at = [], 0
    for n in (2, 2, 500, 1, 498):
        outs.append(m.portion(m.proj[at:at + n].contiguous(), ints([0, n]), ints([1]), ints([0] * n), eps, torch.float32))
        at += n
    want, states = m.plain(m.proj, eps)
    got = torch.cat(outs)
    close(got, want, torch.float32, "all tokens", 1e-4)
    m.check_state(1, states)
    v = double(m.proj)[3, m.at["v"]:m.at["v"] + vdim]
    alone = plain.rms(v, 0.0) * double(m.gain) * plain.sigmoid(double(m.proj)[-1, m.at["g"]:m.at["g"] + vdim])
    close(got[-1], alone, torch.float32, "what token 3 wrote", 1e-3)
    shut = Memory(2, 16, 8, 40, 80, cap=20.0)
    shut.ib.fill_(-15.0), shut.fb.fill_(-1.0)
    shut.portion(shut.proj, ints([0, 40]), ints([0]), ints([0] * 40), 1e-3, torch.float32)
    states = shut.plain(shut.proj, 1e-3)[1]
    shut.check_state(0, states)
    # the first token: nothing but the forget gate moves the maximum
    first = Memory(2, 16, 8, 40, 80, cap=20.0)
    first.ib.fill_(-15.0), first.fb.fill_(-1.0)
    gates = first.gates(first.proj[:1].contiguous(), ints([0, 1]), ints([0]))
    assert float(gates[2, :, 0].min()) >= 1.0 and float(first.state[0, first.m_off:first.m_off + 2].min()) > -6.0


# ---- the dense feed-forward ---------------------------------------------------------------------------------
ACT = {"relu_squared": lambda z: torch.clamp(z, min=0.0) ** 2, "relu": lambda z: torch.clamp(z, min=0.0),
       "silu": lambda z: z * plain.sigmoid(z), "gelu_pytorch_tanh": lambda z: torch.nn.functional.gelu(z, approximate="tanh")}


@pytest.mark.parametrize("activation", sorted(ACT))
@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
def test_the_activation_as_a_kernel_of_its_own(activation, dtype):
    for shape in ((3, 7), (40, 64), (1, 1)):
        z = rnd(*shape, seed=91, dtype=dtype, scale=3.0)
        want = ACT[activation](double(z))
        out = torch.empty_like(z)
        ops().activate(z, activation, out)
        close(out, want, dtype, str(shape))
        ops().activate(z, activation)
        assert torch.equal(z, out)


@pytest.mark.parametrize("activation", ["relu_squared", "gelu_pytorch_tanh"])
@pytest.mark.parametrize("rows,n,k", [(1, 200, 96), (8, 72, 64), (16, 4096, 1024), (5, 8192, 2048), (20, 640, 512), (48, 256, 128), (48, 4104, 128),
                                      (130, 384, 256), (256, 384, 256), (300, 1000, 264), (300, 37, 50), (9, 9, 14), (2300, 520, 136), (2048, 256, 64)])
def test_the_activation_in_the_products_epilogue(rows, n, k, activation):
    """Whichever kernel the row count selects applies the activation to the 32-bit sums."""
    from tokenizer_b200.parts.linear import Linear
    a, w = rnd(rows, k, seed=92, dtype=torch.bfloat16), rnd(n, k, seed=93, dtype=torch.bfloat16, scale=2.0 * k ** -0.5)
    want = ACT[activation](double(a) @ double(w).t())
    close(Linear(w).forward(a, activation=activation), want, torch.bfloat16, "bfloat16", 1.5e-2)
    bias = rnd(n, seed=94)
    want = ACT[activation](double(a) @ double(w).t() + double(bias))
    close(Linear(w, bias).forward(a, activation=activation), want, torch.bfloat16, "with a bias", 1.5e-2)
    if rows < 50:
        close(Linear(w.float()).forward(a.float(), activation=activation), ACT[activation](double(a) @ double(w).t()), torch.float32, "float32")


@pytest.mark.parametrize("rows,n,k", [(60, 256, 128), (300, 520, 264), (1000, 2048, 64)])
def test_the_activation_in_the_tile_kernels_epilogue(rows, n, k):
    """The tensor-core tile kernels of lone CTAs and of pairs, at sizes that other kernels usually take."""
    o = ops()
    a, w, bias = rnd(rows, k, seed=92, dtype=torch.bfloat16), rnd(n, k, seed=93, dtype=torch.bfloat16, scale=2.0 * k ** -0.5), rnd(n, seed=94)
    z = double(a) @ double(w).t()
    for b, add in ((None, 0.0), (bias, double(bias))):
        for kind in (None, o.PAIR_PLAIN, o.PAIR_PLAIN_128):
            out = torch.full((rows, n), float("nan"), dtype=torch.bfloat16, device=DEV)
            if kind is None:
                o.gemm_tcgen05(a, w, b, out, activation="relu_squared")
            else:
                o.gemm_tcgen05_pair(a, w, b, out, kind, "relu_squared")
            close(out, ACT["relu_squared"](z + add), torch.bfloat16, str(kind), 1.5e-2)
    plain_out = torch.empty(rows, n, dtype=torch.bfloat16, device=DEV)
    o.gemm_tcgen05(a, w, None, plain_out)
    close(plain_out, z, torch.bfloat16, "no activation", 1.5e-2)
    with pytest.raises(ValueError):
        o.gemm_tcgen05(a, w, None, torch.empty(rows, n, device=DEV), activation="relu_squared")       # a 32-bit result has no such epilogue


@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("rows", [1, 40, 300])
def test_the_dense_feed_forward(rows, dtype):
    width, inner = 48, 88
    store = {"p.up": rnd(inner, width, seed=95, scale=0.3).cpu().bfloat16(), "p.down": rnd(width, inner, seed=96, scale=0.2).cpu().bfloat16()}
    part = part_of("feed_forward", "dense_mlp", {"hidden_size": width, "inner_size": inner, "activation": "relu_squared"}, store, dtype)
    h = rnd(rows, width, seed=97, dtype=dtype)
    got = part.forward(h)
    got = got.sum(0) if got.dim() == 3 else got
    close(got, plain.squared_relu_feed_forward(double(h), {k: v.double() for k, v in store.items()}, "p."), dtype)


# ---- whole models -----------------------------------------------------------------------------------
LENGTHS = {"a": [1, 2, 23, 100, 131, 49], "b": [5, 19, 97, 201, 260, 100], "c": [3, 40, 130, 64, 1, 90],
           "d": [4, 31, 77, 150, 9, 60]}


@pytest.fixture(scope="module", params=sorted(TINY))
def model(request, tmp_path_factory):
    folder, cfg, page = make_folder(tmp_path_factory, request.param)
    requests = {f"r{i}": random_ids(n, cfg.vocab, 300 + i) for i, n in enumerate(LENGTHS[request.param])}
    want = reference_logits(folder, requests)
    return folder, cfg, page, requests, want


def replay(folder, dtype, steps, max_tokens, page, max_requests=4, use_graphs=True):
    """What the replay program does, inside this process: every step through `Engine.step` on a pool of
    `max_tokens` tokens and `max_requests` slots; returns {step: logits}."""
    from tokenizer_b200.engine import Engine, StepEntry
    engine = Engine.from_folder(folder, dtype=dtype, num_pages=-(-max_tokens // page), page_size=page,
                                max_requests=max_requests, use_graphs=use_graphs)
    live, out = {}, {}
    for record in steps:
        entries = []
        for item in record["entries"]:
            if item["id"] not in live:
                live[item["id"]] = engine.cache.open(item["id"])
            engine.cache.reserve(live[item["id"]], len(item["tokens"]))
            entries.append(StepEntry(live[item["id"]], item["tokens"], item.get("want", [])))
        logits = engine.step(entries)
        if logits.shape[0]:
            out[record["step"]] = logits.cpu().numpy()
        for name in record.get("end", []):
            engine.cache.close(live.pop(name))
        engine.cache.check()
    engine.check()
    return out


def compare(got, want, dtype, what):
    """float32: every logit within 1e-4.  bfloat16: per position, the root mean square of the difference (its
    mean over the vocabulary taken off) against that of the logits themselves: the operands' rounding reaches the
    logits of these tiny models at a few parts in a hundred, while a key, a window's edge or a state that is wrong moves a
    position's logits by their own size.  Where n . q of a head lies near zero under an open gate, o is a quotient of two
    small numbers: one position in two hundred may lie beyond the bound."""
    if dtype == "float32":
        return ru.compare(got, want, dtype, what)
    rel, where = [], []
    for name in sorted(got):
        for position in sorted(got[name]):
            row, ref = got[name][position], want[name][position]
            assert np.isfinite(row).all(), f"{what}: {name}[{position}] not finite"
            d, c = row - ref, ref - ref.mean()
            rel.append(float(np.sqrt(((d - d.mean()) ** 2).mean()) / np.sqrt((c ** 2).mean())))
            where.append((name, position))
    rel = np.array(rel)
    worst = int(rel.argmax())
    print(f"{what} (bfloat16): median {np.median(rel):.4f}, 90 % {np.percentile(rel, 90):.4f}, worst {rel[worst]:.4f} at {where[worst]}")
    far = int((rel > 0.2).sum())
    assert far <= 0.005 * len(rel), \
        f"{what} (bfloat16): {far} of {len(rel)} positions are off, the worst request {where[worst][0]!r} position {where[worst][1]}: {rel[worst]:.3f}"
    assert np.percentile(rel, 90) <= 0.08, f"{what} (bfloat16): a tenth of the positions is off by {np.percentile(rel, 90):.3f} and more"


def test_every_layer_leaves_the_stream_the_plain_layers_leave(model):
    """The residual stream after every layer run, float32."""
    from tokenizer_b200.engine import Engine, StepEntry
    folder, cfg, page, requests, _ = model
    ids = max(requests.values(), key=len)
    raw, w = plain.load_folder(folder)
    want = []
    plain.forward(raw, w, ids, want)
    engine = Engine.from_folder(folder, dtype="float32", num_pages=-(-len(ids) // page) + 1, page_size=page,
                                max_requests=1, use_graphs=False)
    got = []
    for block in set(engine.model.blocks):
        def run(stream, ctx, cache, inner=block.forward):
            inner(stream, ctx, cache)
            got.append(stream.flush().clone())
        block.forward = run
    cache = engine.cache.open("r")
    engine.cache.reserve(cache, len(ids))
    engine.step([StepEntry(cache, ids, [0])])
    assert len(got) == len(want) == len(cfg.run_order())
    for at, (a, b) in enumerate(zip(got, want)):
        err, size = float((a.cpu()[:len(ids)] - b.float()).abs().max()), float(b.abs().max())
        assert err <= 1e-4 * max(1.0, size), f"the stream after layer run {at}: {err:.3e}"


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_whole_prompts(model, dtype):
    folder, cfg, page, requests, want = model
    steps = ru.steps_whole(requests)
    budget = max(ru.rounded64(len(v)) for v in requests.values())
    got = ru.collect(steps, replay(folder, dtype, steps, budget, page))
    assert {k: len(v) for k, v in got.items()} == {k: len(v) for k, v in requests.items()}
    compare(got, want, dtype, "whole")


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_prompt_then_token_by_token(model, dtype):
    """The last 60 tokens one by one: more than most of the windows, so that their edges pass under decoded tokens
    and pages behind them are given back."""
    folder, cfg, page, requests, want = model
    steps = ru.steps_decode_tail(requests, 60)
    budget = max(ru.rounded64(len(v)) for v in requests.values())
    got = ru.collect(steps, replay(folder, dtype, steps, budget, page))
    compare(got, want, dtype, "decode tail")


def test_every_token_alone_from_the_first(model):
    """A sequence fed one token a step from its very first."""
    folder, cfg, page, requests, want = model
    some = {k: v for k, v in requests.items() if len(v) <= 50}
    steps = ru.steps_portions(some, (1,))
    budget = max(ru.rounded64(len(v)) for v in some.values())
    got = ru.collect(steps, replay(folder, "float32", steps, budget, page))
    ru.compare(got, {k: want[k] for k in some}, "float32", "token by token from the start")


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("sizes", [(2, 7, 3, 16, 2, 33, 5, 2, 64, 9), (2,), (31, 1, 1, 96)])
def test_portions(model, dtype, sizes):
    folder, cfg, page, requests, want = model
    if sizes == (2,):
        requests = {k: v for k, v in requests.items() if len(v) <= 100}
    steps = ru.steps_portions(requests, sizes)
    budget = max(ru.rounded64(len(v)) for v in requests.values())
    got = ru.collect(steps, replay(folder, dtype, steps, budget, page))
    assert {k: len(v) for k, v in got.items()} == {k: len(v) for k, v in requests.items()}
    compare(got, want, dtype, f"portions {sizes}")


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("live", [4, 2])
def test_mixed_batches_on_pages_and_slots_that_are_used_again(model, dtype, live):
    folder, cfg, page, requests, want = model
    steps, peak = ru.steps_mixed(requests, max_live=live, seed=live)
    assert peak < sum(ru.rounded64(len(v)) for v in requests.values()) and len(requests) > live
    got = ru.collect(steps, replay(folder, dtype, steps, peak, page, max_requests=live))
    assert {k: len(v) for k, v in got.items()} == {k: len(v) for k, v in requests.items()}
    compare(got, want, dtype, "mixed")


@pytest.mark.parametrize("longest", [2, 20])
def test_mixed_batches_with_portions_in_chunks(model, longest, monkeypatch):
    """Portions that usually run on the scan, down to two tokens, in chunks on tensor cores, single tokens of others
    beside them."""
    from tokenizer_b200.parts import recurrent
    monkeypatch.setattr(recurrent, "MEMORY_CHUNKS_FROM", longest)
    folder, cfg, page, requests, want = model
    steps, peak = ru.steps_mixed(requests, max_live=3, seed=7)
    got = ru.collect(steps, replay(folder, "bfloat16", steps, peak, page, max_requests=3))
    compare(got, want, "bfloat16", "mixed, in chunks")


def test_sizes_that_tiny_models_make_equal_or_one(tmp_path_factory):
    """One head, one lane of most things; models of one kind of mixer alone (no keys kept at all, no matrices kept at
    all); a loop over every layer; no feed-forward anywhere; eight streams."""
    from tiny_kerudra import attention, config, dense, latent, memory
    from tokenizer_b200 import write_random_model
    ones = config([attention(1, 1, 16, 0.25, rot=(10.0, 2), mlp=dense(1)), memory(1, 1, 1, 1.0, mlp=dense(8)),
                   latent(1, 1, 2, 1, 1, 0.5, 10.0, size=2, mlp=dense(3))],
                  vocab=40, width=16, eps=1e-5, streams=2, mult=1.0, embedding=1.0, logit_scale=1.0, loop=(0, 3, 2))
    matrices = config([memory(4, 32, 32, 5.0, mlp=dense(48)), memory(2, 64, 36, 10.0)], vocab=90, width=48, eps=1e-6, streams=8, embedding=4.0)
    keys = config([attention(8, 8, 16, 0.3, rot=(100.0, 16)), attention(2, 1, 80, 0.2), latent(4, 16, 6, 16, 10, 0.3, 50.0, size=9),
                   latent(4, 16, 6, 16, 10, 0.3, 50.0, size=10), latent(2, 8, 4, 8, 12, 0.3, 50.0)],
                  vocab=60, width=40, eps=1e-6, streams=3, mult=0.4, embedding=5.0, logit_scale=2.0, loop=(0, 5, 1))
    for at, cfg in enumerate((ones, matrices, keys)):
        folder, page = str(tmp_path_factory.mktemp(f"kerudra_more{at}")), 16
        write_random_model(folder, cfg, 11 + at, scale=SHARPEN)
        requests = {f"r{i}": random_ids(n, cfg.vocab, 500 + i) for i, n in enumerate([2, 70, 35, 141, 18, 66])}
        want = reference_logits(folder, requests)
        steps = ru.steps_whole(requests)
        got = ru.collect(steps, replay(folder, "float32", steps, max(ru.rounded64(len(v)) for v in requests.values()), page))
        ru.compare(got, want, "float32", f"model {at}, whole")
        steps, peak = ru.steps_mixed(requests, max_live=3, seed=5)
        got = ru.collect(steps, replay(folder, "float32", steps, peak, page, max_requests=3))
        ru.compare(got, want, "float32", f"model {at}, mixed")


def test_steps_launched_anew_agree_with_replayed_ones(model):
    folder, cfg, page, requests, want = model
    steps, peak = ru.steps_mixed(requests, max_live=3, seed=5)
    got = ru.collect(steps, replay(folder, "float32", steps, peak, page, max_requests=3, use_graphs=False))
    ru.compare(got, want, "float32", "without graphs")


def test_many_requests_decode_side_by_side(model):
    """24 rows a step, against each request alone."""
    folder, cfg, page, requests, want = model
    names = list(requests) * 4
    ids = [requests[n][:40] for n in names]
    steps = [{"step": 0, "entries": [{"id": i, "tokens": t[:1], "want": [0]} for i, t in enumerate(ids)]}]
    for at in range(1, 40):
        entries = [{"id": i, "tokens": [t[at]], "want": [0]} for i, t in enumerate(ids) if at < len(t)]
        if entries:
            steps.append({"step": at, "entries": entries})
    got = ru.collect(steps, replay(folder, "float32", steps, len(ids) * 64, page, max_requests=len(ids)))
    ru.compare({i: got[i] for i in got}, {i: want[names[i]] for i in range(len(ids))}, "float32", "24 rows a step")


def test_replay_program_drives_the_same_engine(model, tmp_path):
    folder, cfg, page, requests, want = model
    steps, peak = ru.steps_mixed(requests, max_live=3, seed=9)
    out = ru.run_trace(folder, "float32", steps, str(tmp_path), peak, page)
    ru.compare(ru.collect(steps, out), want, "float32", "the replay program")


# ---- generation ---------------------------------------------------------------------------------------
def near_best(cfg, w, prompt, tokens, dtype):
    logits = plain.forward(cfg, w, list(prompt) + list(tokens)).float()
    lead = logits[len(prompt) - 1:-1]
    chosen = lead.gather(1, torch.tensor(tokens)[:, None])[:, 0]
    slack = 1e-4 if dtype == "float32" else 0.1 * float(logits.abs().max())
    gap = lead.max(dim=1).values - chosen
    assert float(gap.max()) <= slack, f"token {int(gap.argmax())} lies {float(gap.max())} below the best logit"


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_greedy_generation_through_the_entry_point(model, dtype):
    import tokenizer_b200 as tb
    folder, cfg, page, requests, _ = model
    raw, w = plain.load_folder(folder)
    engine_model = tb.load_model(folder, dtype=dtype)
    for n in (1, 9, 70):
        prompt = random_ids(n, cfg.vocab, 500 + n)
        out = tb.generate(engine_model, prompt, tb.GenerateParams.greedy(24))
        assert out.reason == tb.StopReason.MAX_TOKENS and len(out.tokens) == 24
        near_best(raw, w, prompt, out.tokens, dtype)


def test_a_batch_through_the_scheduler_with_preemption_gives_each_request_its_own_ids(model):
    """Five prompts on a pool that cannot hold them all: requests are preempted and computed again."""
    import tokenizer_b200 as tb
    folder, cfg, page, requests, _ = model
    raw, w = plain.load_folder(folder)
    engine_model = tb.load_model(folder, dtype="float32")
    prompts = [random_ids(n, cfg.vocab, 600 + n) for n in (30, 7, 55, 18, 41)]
    engine = tb.engine_for(engine_model, 192, page_size=page, max_requests=3, share_prefixes=False)
    results = tb.generate_batch(engine, prompts, tb.GenerateParams.greedy(20), max_batch_size=3, token_budget=48,
                                page_size=page)
    for prompt, result in zip(prompts, results):
        near_best(raw, w, prompt, result.tokens, "float32")


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_long_decoding_on_the_device(model, dtype):
    """300 greedy steps without a visit to the host between them (captured and replayed): windows pass under
    decoded tokens, pages behind them are given back."""
    from tokenizer_b200.engine import Engine, StepEntry
    folder, cfg, page, requests, _ = model
    raw, w = plain.load_folder(folder)
    engine = Engine.from_folder(folder, dtype=dtype, num_pages=-(-2 * 384 // page), page_size=page, max_requests=2)
    prompts = [random_ids(5, cfg.vocab, 700), random_ids(41, cfg.vocab, 701)]
    caches, first = [], []
    for i, prompt in enumerate(prompts):
        c = engine.cache.open(i)
        engine.cache.reserve(c, len(prompt))
        first.append(int(engine.step([StepEntry(c, prompt, [len(prompt) - 1])]).argmax()))
        caches.append(c)
    history = engine.decode_steps([StepEntry(c, [t], [0]) for c, t in zip(caches, first)], 300)
    for i, prompt in enumerate(prompts):
        near_best(raw, w, prompt, [first[i]] + [step[i] for step in history], dtype)


def test_the_command_line_generates_from_a_configuration_of_this_design(tmp_path):
    """`--random-weights config.json` draws the weights the configuration declares; two prompts go through the
    scheduler and print ids that the plain implementation ranks best."""
    import json
    import os
    import subprocess
    import sys
    import tokenizer_b200 as tb
    cfg = TINY["a"]()[0]
    page = TINY["a"]()[2]
    path = str(tmp_path / "config.json")
    with open(path, "w") as fh:
        json.dump(cfg.to_dict(), fh)
    folder = tb.write_random_model(str(tmp_path / "same"), cfg, 0)        # the command line's default seed
    raw, w = plain.load_folder(folder)
    prompts = [random_ids(11, cfg.vocab, 801), random_ids(40, cfg.vocab, 802)]
    cli = os.path.join(os.path.dirname(os.path.dirname(os.path.abspath(__file__))), "bin", "qwen-infer")
    args = [sys.executable, cli, "--random-weights", path, "--weights-seed", "0", "--dtype", "float32",
            "--max-tokens", "10", "--page-size", str(page)]
    for prompt in prompts:
        args += ["--ids", ",".join(str(t) for t in prompt)]
    proc = subprocess.run(args, capture_output=True, text=True, timeout=600)
    assert proc.returncode == 0, proc.stderr
    lines = proc.stdout.strip().splitlines()
    assert len(lines) == 2
    for prompt, line in zip(prompts, lines):
        near_best(raw, w, prompt, [int(t) for t in line.split()], "float32")
