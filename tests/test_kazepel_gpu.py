"""The Kazepel decoder on the GPU against the plain restatement: each mechanism's kernels alone, with weights or
inputs made so that a fault shows (a key just outside a window, the last kept first token, the sink alone, a far
write in a matrix), then whole models (four tiny configurations of unlike sizes) whole, token by token, in
portions, in mixed batches on few pages and slots, and through the generation entry point."""
import math

import numpy as np
import pytest
import torch

import plain_kazepel as plain
import replay_util as ru
from tiny import random_ids
from tiny_kazepel import SHARPEN, TINY, make_folder, reference_logits

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


# ---- the norm without statistics and the stream's update ------------------------------------------------
@pytest.mark.parametrize("out_dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("width", [50, 320, 2048, 9001])
@pytest.mark.parametrize("form", ["none", "bf16", "f32", "partials", "carried", "restart"])
def test_the_update_of_the_stream_and_the_norm_behind_it(width, form, out_dtype):
    """x <- (x or a vector) + y + share * carried in place, then tanh(alpha x) gain + bias of the new x."""
    o = ops()
    n, alpha = 6, 0.7
    x, gain, bias = rnd(n, width, seed=1, scale=2.0), rnd(width, seed=2) + 1.0, rnd(width, seed=3)
    y = base = carried = share = None
    want = x.double().cpu()
    if form in ("bf16", "carried"):
        y = rnd(n, width, seed=4, dtype=torch.bfloat16)
    elif form in ("f32", "restart"):
        y = rnd(n, width, seed=4)
    elif form == "partials":
        y = rnd(3, n, width, seed=4)
    if form == "restart":
        base = rnd(width, seed=5)
        want = base.double().cpu().expand(n, width)
        x = torch.full_like(x, float("nan"))               # the stream's own value is not read
    if form == "carried":
        carried = rnd(n, width, seed=6, dtype=out_dtype)
        shares = rnd(n, 5, seed=7)
        share = shares[:, 3]                                # a column of a wider matrix
        want = want + share.double().cpu()[:, None] * carried.double().cpu()
    if y is not None:
        want = want + (y.double().cpu().sum(0) if y.dim() == 3 else y.double().cpu())
    out = torch.full((n, width), float("nan"), dtype=out_dtype, device=DEV)
    got = x.clone()
    o.stream_update(got, y, base, carried, share, alpha=alpha, gain=gain, bias=bias, out=out)
    close(got, want, torch.float32, "the stream")
    normed = plain.dynamic_tanh(want, alpha, gain.double().cpu(), bias.double().cpu())
    close(out, normed, out_dtype, "the norm")
    if form == "none":
        assert torch.equal(got, x)
        rows = ints([4, 0, 4])
        some = torch.empty(3, width, dtype=out_dtype, device=DEV)
        o.stream_update(got, alpha=alpha, gain=gain, bias=bias, out=some, rows=rows)
        close(some, normed[[4, 0, 4]], out_dtype, "gathered rows")
    # the update alone, and the operand of a pass: the new stream and a second matrix side by side
    again = x.clone()
    o.stream_update(again, y, base, carried, share)
    assert torch.equal(again, got)
    beside = rnd(n, width, seed=8)
    joined = torch.full((n, 2 * width), float("nan"), dtype=out_dtype, device=DEV)
    again = x.clone()
    o.stream_update(again, y, base, carried, share, beside=beside, out=joined)
    assert torch.equal(joined[:, :width], got.to(out_dtype)) and torch.equal(joined[:, width:], beside.to(out_dtype))


def part_of(category, kind, params, tensors, dtype=torch.float32, prefix="p"):
    from tokenizer_b200.config.spec import PartSpec
    from tokenizer_b200.parts.base import Runtime, build_part
    from tokenizer_b200.weights.store import WeightStore
    return build_part(category, PartSpec(kind, params, prefix), WeightStore(tensors), Runtime(torch.device(DEV), dtype))


def test_the_final_norm_carries_a_constant_on_the_logits():
    w, b, alpha = rnd(72, seed=1).cpu() + 1.0, rnd(72, seed=2).cpu(), torch.tensor(1.3)
    norm = part_of("norm", "dynamic_tanh", {"size": 72, "tensor": "n", "scale": 0.35}, {"n": w, "n.b": b, "n.alpha": alpha})
    x = rnd(5, 72, seed=3, scale=2.0)
    want = 0.35 * plain.dynamic_tanh(x.double().cpu(), alpha.double(), w.double(), b.double())
    close(norm.forward(x), want, torch.float32, "all rows")
    close(norm.forward(x, rows=ints([2, 2, 0])), want[[2, 2, 0]], torch.float32, "gathered")
    delta = rnd(5, 72, seed=4)
    moved = x.clone()
    close(norm.forward(moved, delta=delta), 0.35 * plain.dynamic_tanh((x + delta).double().cpu(), alpha.double(), w.double(), b.double()),
          torch.float32, "with a pending add")
    assert torch.equal(moved, x + delta)


@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("rows,width", [(3, 50), (40, 96), (130, 128)])
def test_a_pass_starts_from_the_projected_stream_and_embedding(rows, width, dtype):
    from tokenizer_b200.parts.base import ResidualStream, StreamUpdate
    w_in, steps = rnd(width, 2 * width, seed=1, scale=0.2).cpu(), rnd(3, width, seed=2).cpu()
    part = part_of("injection", "pass_projection", {"projection": "in", "tensor": "step", "passes": 3, "hidden_size": width, "index": 1},
                   {"in": w_in.bfloat16(), "step": steps}, dtype)
    x, x0, y, h = (rnd(rows, width, seed=s) for s in (3, 4, 5, 6))
    share = rnd(rows, 1, seed=7)[:, 0]
    for pending in ("nothing", "an output", "an output and the input handed through"):
        stream = ResidualStream(x.clone())
        now = x.double().cpu()
        if pending == "an output":
            stream.add(y)
            now = now + y.double().cpu()
        elif pending != "nothing":
            stream.add(StreamUpdate(y, carried=h, share=share))
            now = now + y.double().cpu() + share.double().cpu()[:, None] * h.double().cpu()
        part.forward(stream, x0)
        want = plain.enter_pass(now, x0.double().cpu(), w_in.bfloat16().double(), steps[1].double())
        close(stream.flush(), want, dtype, pending)
        assert stream.x.dtype == torch.float32


# ---- yarn's rotation on keys and queries ----------------------------------------------------------------
@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("heads,kv,dim,vdim,dims", [(6, 2, 64, 128, 32), (3, 3, 10, 20, 4), (4, 1, 32, 16, 32), (2, 2, 24, 24, 8)])
def test_rotation_by_yarn_multiplies_cosine_and_sine(heads, kv, dim, vdim, dims, dtype):
    o = ops()
    n, row = 6, -(-max(dim, vdim) // 16) * 16
    scaling = {"factor": 6.0, "original": 128, "fast": 12.0, "slow": 1.0}
    position = part_of("position", "rope_half", {"base": 2000.0, "dims": dims, "scaling": dict(scaling, kind="yarn")}, {})
    proj = rnd(n, heads * dim + kv * (dim + vdim) + 4, seed=11)
    pos = [0, 1, 2, 900, 77, 40000]
    q = torch.full((n, heads * row), float("nan"), dtype=dtype, device=DEV)
    pools = [torch.full((n, kv, row), float("nan"), dtype=dtype, device=DEV) for _ in range(2)]
    o.qkv_rotate_store(proj, 0, None, position.inv_freq64, dims, ints(pos), ints(range(n)), ints([0] * n), q, pools[0], pools[1],
                       heads, kv, dim, vdim, row, layout=position.layout, magnitude=position.magnitude)
    freqs, magnitude = plain.yarn_frequencies(2000.0, dims, scaling)
    p, where = proj.double().cpu(), torch.tensor(pos)
    want_q = plain.rotate_halves(p[:, :heads * dim].view(n, heads, dim), where, freqs, magnitude)
    want_k = plain.rotate_halves(p[:, heads * dim:(heads + kv) * dim].view(n, kv, dim), where, freqs, magnitude)
    close(q.view(n, heads, row)[:, :, :dim], want_q, dtype, "queries")
    close(pools[0][:, :, :dim], want_k, dtype, "keys")
    close(pools[1][:, :, :vdim], p[:, (heads + kv) * dim:(heads + kv) * dim + kv * vdim].view(n, kv, vdim), dtype, "values")
    assert magnitude > 1.1 and float((want_q - plain.rotate_halves(p[:, :heads * dim].view(n, heads, dim), where, freqs, 1.0)).abs().max()) > 0.1


# ---- windows that keep the first tokens, and the sink, in every attention kernel ------------------------------
def paged(lengths, kv, row, dtype, seed):
    g = torch.Generator().manual_seed(seed)
    return [[torch.randn(n, kv, row, generator=g).to(dtype), torch.randn(n, kv, row, generator=g).to(dtype)] for n in lengths]


def scatter(dense, kv, row, page, dtype, seed, held):
    """Keys and values on shuffled pages; pages of which `held(request, first, last key)` is false do not exist
    (their table entries are -1, as the cache manager leaves them)."""
    g = torch.Generator().manual_seed(seed)
    n_pages = sum(-(-k.shape[0] // page) for k, _ in dense) + 2
    order = torch.randperm(n_pages, generator=g).tolist()
    pools = [torch.full((n_pages * page, kv, row), float("nan"), dtype=dtype) for _ in range(2)]
    tables = torch.full((len(dense), max(-(-k.shape[0] // page) for k, _ in dense) + 1), -1, dtype=torch.int32)
    for r, (k, v) in enumerate(dense):
        for b in range(-(-k.shape[0] // page)):
            rows = slice(b * page, min(k.shape[0], (b + 1) * page))
            if not held(r, rows.start, rows.stop - 1):
                continue
            pg = order.pop()
            tables[r, b] = pg
            pools[0][pg * page:pg * page + rows.stop - rows.start] = k[rows]
            pools[1][pg * page:pg * page + rows.stop - rows.start] = v[rows]
    return pools, tables


def run_attention(kernel, q, pools, tables, row_req, pos, spans, heads, kv, row, page, scale, window, keep, sink):
    from tokenizer_b200.parts.attention import RowTiles
    o = ops()
    out = torch.full((len(pos), heads * row), float("nan"), dtype=q.dtype, device=DEV)
    args = (q.to(DEV).view(len(pos), -1), pools[0].to(DEV), pools[1].to(DEV), out, tables.to(DEV), ints(row_req), ints(pos))
    if kernel == "generic":
        o.paged_attention_generic(*args, heads, kv, row, page, window, scale, sink=sink, keep_first=keep)
    elif kernel == "decode":
        o.decode_attention(*args, heads, kv, row, page, window, scale, sink=sink, keep_first=keep)
    else:
        note = RowTiles(o.WIDE_TILE_ROWS if kernel == "wide" else o.PREFILL_TILE_ROWS)
        words = np.zeros(note.capacity(len(pos), len(spans)), dtype=np.int32)
        counts = np.array([m for _, _, m in spans], dtype=np.int32)
        firsts = np.concatenate(([0], np.cumsum(counts)[:-1])).astype(np.int32)
        n_tiles = note.fill(words, firsts, counts, np.array([f for _, f, _ in spans], dtype=np.int32), False)
        tiles = torch.tensor(words, device=DEV).view(-1, 2)
        run = o.attention_tcgen05 if kernel == "wide" else o.prefill_attention
        run(*args, tiles, n_tiles, heads, kv, row, page, window, scale, sink=sink, keep_first=keep)
    return out.view(len(pos), heads, row).float().cpu()


def plain_rows(q, dense, row_req, pos, scale, mask, sink=True):
    heads = q.shape[1]
    out = torch.zeros(q.shape, dtype=torch.float64)
    for t in range(q.shape[0]):
        k, v = dense[row_req[t]]
        seen = torch.tensor([j <= pos[t] and (mask is None or pos[t] - j < mask["size"] or j < mask["keep_first"])
                             for j in range(k.shape[0])])
        for h in range(heads):
            g = h // (heads // k.shape[1])
            s = (k[:, g].double() @ q[t, h].double() * scale).masked_fill(~seen, -math.inf)
            out[t, h] = (plain.softmax_one(s[None])[0] if sink else torch.softmax(s, dim=0)) @ v[:, g].double()
    return out


ATTENTION_CASES = [
    # kernel, dtype, heads, kv heads, lanes, window's keys, kept first tokens
    ("generic", torch.float32, 3, 3, 48, 50, 7), ("generic", torch.bfloat16, 4, 2, 144, 33, 40), ("generic", torch.float32, 2, 1, 32, 1, 1),
    ("generic", torch.float32, 2, 1, 16, 140, 130), ("generic", torch.float32, 2, 1, 16, 21, 0),
    ("decode", torch.bfloat16, 4, 2, 32, 96, 16), ("decode", torch.bfloat16, 16, 1, 64, 37, 5), ("decode", torch.bfloat16, 2, 2, 128, 300, 300),
    ("decode", torch.bfloat16, 2, 2, 48, 700, 33), ("decode", torch.bfloat16, 4, 1, 64, 1, 2), ("decode", torch.bfloat16, 2, 1, 80, 64, 0),
    ("tiles", torch.bfloat16, 3, 3, 48, 37, 3), ("tiles", torch.bfloat16, 4, 2, 80, 160, 70), ("tiles", torch.bfloat16, 2, 2, 16, 1, 64),
    ("tiles", torch.bfloat16, 2, 1, 64, 64, 65), ("tiles", torch.bfloat16, 2, 1, 96, 90, 0),
    ("wide", torch.bfloat16, 4, 2, 128, 160, 20), ("wide", torch.bfloat16, 6, 3, 128, 37, 128), ("wide", torch.bfloat16, 2, 1, 64, 96, 129),
    ("wide", torch.bfloat16, 2, 1, 64, 1, 1), ("wide", torch.bfloat16, 2, 1, 64, 200, 0)]


@pytest.mark.parametrize("kernel,dtype,heads,kv,row,size,keep", ATTENTION_CASES)
def test_window_edges_and_kept_first_tokens_in_every_attention_kernel(kernel, dtype, heads, kv, row, size, keep):
    """For every request's last row the key just outside the window, the oldest one inside, the last kept first
    token and the first token that is not kept get scores that stand out and values of their own.  Requests end
    right behind, on and before the edge, one is a single token; pages that no row can see any more do not exist."""
    page = 16
    reach = size + keep
    lengths = [2 * reach + size + 2, reach + 1, 1, 3 * size + keep + 40, max(keep, 1)]
    dense = paged(lengths, kv, row, dtype, seed=60)
    scale = 1.0 / math.sqrt(row)
    if kernel == "decode":
        spans = [(r, n - 1, 1) for r, n in enumerate(lengths)]
    else:
        spans = [(r, n - min(n, 150), min(n, 150)) for r, n in enumerate(lengths)]
    row_req = [r for r, _, m in spans for _ in range(m)]
    pos = [first + i for _, first, m in spans for i in range(m)]
    q = rnd(len(pos), heads, row, seed=61, dtype=dtype).cpu()
    planted = 0
    for t in range(len(pos)):
        if t + 1 < len(pos) and row_req[t + 1] == row_req[t]:
            continue
        start = max(0, pos[t] - size + 1)
        k, v = dense[row_req[t]]
        direction = q[t, 0].float() / q[t, 0].float().norm()
        for key, strength, value in ((start - 1, 40.0, 50.0), (keep, 38.0, -60.0), (keep - 1, 20.0, 7.0), (start, 20.0, -9.0)):
            if 0 <= key < k.shape[0] and not (strength > 30.0 and (key >= start or key < keep)):
                k[key, 0] = (direction * strength).to(dtype)
                v[key, 0] = value
                planted += strength > 30.0
    first_row = {r: first for r, first, _ in spans}
    held = lambda r, a, b: b >= first_row[r] - size + 1 or a < keep
    pools, tables = scatter(dense, kv, row, page, dtype, 62, held)
    sink = torch.zeros(heads, device=DEV)
    got = run_attention(kernel, q, pools, tables, row_req, pos, spans, heads, kv, row, page, scale, size - 1, keep, sink)
    mask = {"size": size, "keep_first": keep}
    some = sorted({0, 1, len(pos) - 1} | {t for t in range(len(pos)) if t + 1 == len(pos) or row_req[t + 1] != row_req[t]} |
                  set(range(0, len(pos), 7)))
    want = plain_rows(q[some], dense, [row_req[t] for t in some], [pos[t] for t in some], scale, mask)
    assert torch.isfinite(got).all()
    bound = 2e-5 if dtype == torch.float32 else 3e-2
    assert float((got[some] - want).abs().max()) <= bound * max(1.0, float(want.abs().max()))
    # the edges matter: with one more key outside, or one kept token more or fewer, rows move far
    assert planted > 0
    for other in ({"size": size + 1, "keep_first": keep}, {"size": size, "keep_first": keep + 1}):
        wrong = plain_rows(q[some], dense, [row_req[t] for t in some], [pos[t] for t in some], scale, other)
        assert float((wrong - want).abs().max()) > 1.0


@pytest.mark.parametrize("kernel,dtype,row", [("generic", torch.float32, 48), ("decode", torch.bfloat16, 64),
                                              ("tiles", torch.bfloat16, 48), ("wide", torch.bfloat16, 128)])
def test_the_sink_takes_what_no_key_stands_out_for(kernel, dtype, row):
    """Every score far below zero: the outputs vanish, where a softmax without the one in its denominator gives a
    mean of the values; a far kept key that stands out comes back nearly whole through hundreds of others."""
    heads, kv, page, n, size, keep = 2, 1, 16, 900, 300, 4
    dense = paged([n], kv, row, dtype, seed=70)
    take = 1 if kernel == "decode" else 120
    spans = [(0, n - take, take)]
    row_req, pos = [0] * take, list(range(n - take, n))
    q = torch.ones(take, heads, row).to(dtype)
    q[-1, 1] = -1.0
    k, v = dense[0]
    k[:] = (-torch.rand(n, kv, row, generator=torch.Generator().manual_seed(5)) - 1.0).to(dtype)
    v[:] = 1.0
    k[2, 0] = -3.0
    v[2, 0] = 9.0
    scale = 12.0 / row
    pools, tables = scatter(dense, kv, row, page, dtype, 71, lambda r, a, b: True)
    got = run_attention(kernel, q, pools, tables, row_req, pos, spans, heads, kv, row, page, scale, size - 1, keep,
                        torch.zeros(heads, device=DEV))
    want = plain_rows(q[-1:], dense, [0], [n - 1], scale, {"size": size, "keep_first": keep})
    assert float((got[-1:] - want).abs().max()) <= (2e-5 if dtype == torch.float32 else 3e-2) * 9.0
    assert float(got[-1, 0].abs().max()) < 0.05 and float(want[0, 1].min()) > 8.0
    free = plain_rows(q[-1:], dense, [0], [n - 1], scale, {"size": size, "keep_first": keep}, sink=False)
    assert float((free - want).abs().max()) > 0.5


# ---- the delta rule with a decay a key channel ------------------------------------------------------------------
DELTA_SIZES = [(2, 4, 16, 24, 4), (1, 1, 10, 6, 5), (3, 3, 64, 128, 2), (1, 2, 260, 8, 3), (2, 2, 8, 8, 1), (2, 4, 128, 64, 4),
               (1, 2, 96, 20, 3), (2, 2, 40, 12, 4), (1, 1, 136, 16, 4)]


def delta_inputs(groups, heads, dim, vdim, taps, total, seed, extra):
    channels = 2 * groups * dim + heads * vdim
    proj = rnd(total, extra + channels + heads + 3, seed=seed, scale=1.5)
    pre = rnd(total, heads * (dim + vdim), seed=seed + 1, scale=2.0)
    conv = rnd(channels, taps, seed=seed + 2, scale=0.7)
    a_log, dt_bias = rnd(heads, seed=seed + 3, scale=0.5), rnd(heads * dim, seed=seed + 4) - 2.0
    return proj, pre, conv, a_log, dt_bias, channels


def plain_delta(proj, pre, conv, a_log, dt_bias, groups, heads, dim, vdim, extra):
    """[(o, last matrix)] a head, of one request's rows from its start, in float64."""
    p = proj.double().cpu()
    n, channels = p.shape[0], 2 * groups * dim + heads * vdim
    c = plain.silu(plain.short_convolution(p[:, extra:extra + channels], conv.double().cpu()))
    q = plain.unit_vectors(c[:, :groups * dim].view(n, groups, dim)) * dim ** -0.5
    k = plain.unit_vectors(c[:, groups * dim:2 * groups * dim].view(n, groups, dim))
    v = c[:, 2 * groups * dim:].view(n, heads, vdim)
    beta = plain.sigmoid(p[:, extra + channels:extra + channels + heads])
    a = (pre.double().cpu()[:, :heads * dim] + dt_bias.double().cpu()).view(n, heads, dim)
    decay = torch.exp(-torch.exp(a_log.double().cpu())[None, :, None] * plain.softplus(a))
    return [plain.channel_delta_rule(q[:, h // (heads // groups)], k[:, h // (heads // groups)], v[:, h], beta[:, h], decay[:, h])
            for h in range(heads)]


def state_for(o, groups, heads, dim, vdim, taps, slots):
    channels = 2 * groups * dim + heads * vdim
    conv_off = heads * vdim * o.cdr_padded_dim(dim)
    return torch.zeros(slots, -(-(conv_off + (taps - 1) * channels) // 4) * 4, device=DEV), conv_off


@pytest.mark.parametrize("groups,heads,dim,vdim,taps", DELTA_SIZES)
def test_the_rule_in_portions_carries_matrices_and_kept_inputs(groups, heads, dim, vdim, taps):
    """Three requests in slots that are not their indices, cut into portions of 1, 2, 3 and many rows (in the
    middle of a run of four, shorter than the convolution too), against the recurrence token by token."""
    o = ops()
    lengths = [37, 1, 150]
    cuts = [[0, 1, 3, 4, 7, 20, 37], [0, 1], [0, 129, 132, 133, 135, 150]]
    slots, extra, total = [2, 0, 3], 5, sum(lengths)
    proj, pre, conv, a_log, dt_bias, channels = delta_inputs(groups, heads, dim, vdim, taps, total, 30, extra)
    state, conv_off = state_for(o, groups, heads, dim, vdim, taps, 5)
    padded = o.cdr_padded_dim(dim)
    state[1] = 7.0                                        # a slot nobody holds must stay as it is
    out = torch.full((total, heads * vdim), float("nan"), device=DEV)
    starts = np.concatenate(([0], np.cumsum(lengths)))
    for i in range(max(len(c) for c in cuts) - 1):
        rows, spans, who = [], [0], []
        for r in range(3):
            if i + 1 < len(cuts[r]):
                rows += list(range(starts[r] + cuts[r][i], starts[r] + cuts[r][i + 1]))
                spans.append(len(rows))
                who.append(slots[r])
        idx = torch.tensor(rows, device=DEV)
        sub = proj[idx].contiguous()
        # an idle request at the end, as a padded step has it
        spans_d, who_d = ints(spans + [spans[-1]]), ints(who + [0])
        records = o.cdr_records(len(rows), len(who) + 1, heads, dim, vdim, DEV)
        records.fill_(float("nan"))
        o.cdr_prepare(sub, extra, extra + channels, pre[idx].contiguous(), groups, heads, dim, vdim, taps, conv, a_log, dt_bias,
                      state, conv_off, spans_d, who_d, records)
        o.short_conv_state(sub, extra, channels, taps, state, conv_off, spans_d, who_d)
        got = torch.full((len(rows), heads * vdim), float("nan"), device=DEV)
        o.cdr_scan(records, heads, dim, vdim, state, spans_d, who_d, got)
        out[idx] = got
    for r, n in enumerate(lengths):
        rows = slice(starts[r], starts[r + 1])
        for h, (want, last) in enumerate(plain_delta(proj[rows], pre[rows], conv, a_log, dt_bias, groups, heads, dim, vdim, extra)):
            close(out[rows, h * vdim:(h + 1) * vdim], want, torch.float32, f"request {r} head {h}")
            kept = state[slots[r], :conv_off].view(heads, vdim, padded)[h]
            close(kept[:, :dim].t(), last, torch.float32, f"the matrix of request {r} head {h}")
            assert float(kept[:, dim:].abs().max() if padded > dim else 0) == 0
    assert torch.all(state[1] == 7.0) and torch.all(state[4] == 0.0)


@pytest.mark.parametrize("inside", [True, False])
@pytest.mark.parametrize("out_dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("groups,heads,dim,vdim,taps", DELTA_SIZES + [(1, 1, 512, 150, 4)])
def test_a_step_of_single_tokens_in_one_kernel(groups, heads, dim, vdim, taps, out_dtype, inside):
    """Token by token through `cdr_step` (three requests, one absent from some steps, an idle row of a padded step)
    against the kernels for portions fed the same rows; the second low-rank products inside the kernel or handed in."""
    o = ops()
    extra, ra, rg = 3, 16, 8
    channels = 2 * groups * dim + heads * vdim
    one, conv_off = state_for(o, groups, heads, dim, vdim, taps, 4)
    many = torch.zeros_like(one)
    conv = rnd(channels, taps, seed=71, scale=0.7)
    a_log, dt_bias, gain = rnd(heads, seed=72, scale=0.5), rnd(heads * dim, seed=73) - 1.0, rnd(vdim, seed=74) + 1.0
    w2 = torch.zeros(heads * (dim + vdim), ra + rg, device=DEV)
    w2[:heads * dim, :ra] = rnd(heads * dim, ra, seed=75, scale=0.3)
    w2[heads * dim:, ra:] = rnd(heads * vdim, rg, seed=76, scale=0.3)
    w2 = w2.to(out_dtype)
    low_at, b_at, width = extra + channels, extra + channels + ra + rg, extra + channels + ra + rg + heads
    shift = heads == groups
    for step in range(7):
        present, slots = ([0, 1, 2] if step % 3 else [0, 2]), [3, 0, 1]
        n = len(present) + 1                                                    # the last row is idle
        proj = rnd(n, width, seed=80 + step, scale=1.5)
        row_req, spans = ints(list(range(len(present))) + [-1]), ints(list(range(len(present) + 1)) + [len(present)])
        who = ints([slots[r] for r in present] + [0])
        pre = proj[:, low_at:low_at + ra + rg] @ w2.float().t()
        got = torch.full((n, heads * vdim), float("nan"), dtype=out_dtype, device=DEV)
        o.cdr_step(proj, extra, b_at, low_at, ra, rg, w2, None if inside else pre, groups, heads, dim, vdim, taps, conv, a_log, dt_bias,
                   gain, 1e-5, one, conv_off, row_req, who, shift, got)
        if not shift:
            o.short_conv_state(proj, extra, channels, taps, one, conv_off, spans, who)
        records = o.cdr_records(n, spans.shape[0] - 1, heads, dim, vdim, DEV)
        o.cdr_prepare(proj, extra, b_at, pre, groups, heads, dim, vdim, taps, conv, a_log, dt_bias, many, conv_off, spans, who, records)
        o.short_conv_state(proj, extra, channels, taps, many, conv_off, spans, who)
        raw = torch.zeros(n, heads * vdim, device=DEV)
        o.cdr_scan(records, heads, dim, vdim, many, spans, who, raw)
        o_heads = raw.double().cpu().view(n, heads, vdim)
        want = o_heads / torch.sqrt((o_heads ** 2).mean(-1, keepdim=True) + 1e-5) * gain.double().cpu() * \
            plain.sigmoid(pre.double().cpu()[:, heads * dim:].view(n, heads, vdim))
        close(got[:-1], want.view(n, -1)[:-1], out_dtype, f"step {step}", 1e-4 if out_dtype == torch.float32 else 2e-2)
        assert torch.isnan(got[-1].float()).all()
        normed = torch.full((n, heads * vdim), float("nan"), dtype=out_dtype, device=DEV)
        o.gdn_out_norm(raw, pre, heads * dim, gain, 1.0, 1e-5, normed, heads, vdim, row_req, gate_kind="sigmoid")
        close(normed[:-1], want.view(n, -1)[:-1], out_dtype, "the output norm and its gate", 1e-4 if out_dtype == torch.float32 else 2e-2)
    close(one, many, torch.float32, "matrices and kept inputs")
    assert float(one[3].abs().max()) > 0 and float(one[2].abs().max()) == 0


@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("rows,width,at,n", [(5, 40, 8, 16), (300, 64, 4, 48), (7, 37, 3, 9), (1, 24, 6, 16)])
def test_columns_of_a_product_in_the_compute_type(rows, width, at, n, dtype):
    proj = rnd(rows, width, seed=5)
    out = torch.full((rows, n), float("nan"), dtype=dtype, device=DEV)
    ops().take_columns(proj, at, out)
    assert torch.equal(out, proj[:, at:at + n].to(dtype))


@pytest.mark.parametrize("dim", [32, 64, 128, 256])
def test_a_channel_without_decay_keeps_what_was_written_far_back(dim):
    """Channel 0 never decays, all others lose everything each token: what token 3 wrote along a key of both comes
    back along channel 0 at token 900, scaled by the key's share there; with one decay for the whole matrix it
    could not.  Run boundaries and portions lie between."""
    o = ops()
    vdim, total, taps = 16, 901, 1
    channels = 2 * dim + vdim
    proj = torch.zeros(total, channels + 1, device=DEV)
    big = 50.0                                              # silu is the identity out there, and unit vectors take the size away
    proj[:, dim + 5] = big                                  # keys along channel 5
    proj[:, 5] = big
    proj[:, channels] = -40.0                               # beta 0: nothing is written
    proj[3, dim:2 * dim] = 0.0
    proj[3, dim], proj[3, dim + 1] = 0.6 * big, 0.8 * big   # token 3 writes along channels 0 and 1
    proj[3, 2 * dim:channels] = torch.arange(1, vdim + 1, device=DEV).float() + 30.0
    proj[3, channels] = 40.0
    proj[900, :dim] = 0.0
    proj[900, 0] = big                                      # token 900 reads along channel 0
    pre = torch.full((total, dim), 80.0, device=DEV)        # decay exp(-80)
    pre[:, 0] = -80.0                                       # decay 1
    state, conv_off = state_for(o, 1, 1, dim, vdim, taps, 2)
    conv, a_log, dt = torch.ones(channels, 1, device=DEV), torch.zeros(1, device=DEV), torch.zeros(dim, device=DEV)
    out, at = torch.empty(total, vdim, device=DEV), 0
    for n in (2, 2, 499, 1, 397):
        spans, who = ints([0, n]), ints([1])
        records = o.cdr_records(n, 1, 1, dim, vdim, DEV)
        o.cdr_prepare(proj[at:at + n].contiguous(), 0, channels, pre[at:at + n].contiguous(), 1, 1, dim, vdim, taps, conv, a_log, dt,
                      state, conv_off, spans, who, records)
        o.cdr_scan(records, 1, dim, vdim, state, spans, who, out[at:at + n])
        at += n
    want = 0.6 * (torch.arange(1, vdim + 1).float() + 30.0) * dim ** -0.5
    assert torch.allclose(out[900].cpu(), want, rtol=1e-5)
    assert float(out[899].abs().max()) < 1e-6


# ---- the router ----------------------------------------------------------------------------------------------
@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("experts,identity,top,groups,keep", [(6, 2, 2, 4, 2), (5, 0, 3, 1, 1), (2, 6, 2, 4, 2), (40, 24, 5, 8, 3), (1, 0, 1, 1, 1),
                                                              (3, 1, 4, 1, 1), (600, 424, 9, 64, 7), (70, 30, 4, 50, 49)])
def test_softmax_over_all_outputs_chosen_by_groups_and_renormalised(experts, identity, top, groups, keep, dtype):
    o = ops()
    n, hidden, outputs = 13, 48, experts + identity
    h, router = rnd(n, hidden, seed=31, dtype=dtype), rnd(outputs, hidden, seed=32, scale=0.4)
    correction = rnd(outputs, seed=33, scale=0.5 / outputs) - 1.5 / outputs       # many choice scores lie below zero
    share = torch.full((n, experts + (1 if identity else 0)), float("nan"), device=DEV)
    o.moe_route(h, router, experts, top, None, share, score="softmax", correction=correction, groups=groups, keep=keep,
                identity=identity, group_worth=1, renormalize=True)
    z = h.double().cpu() @ router.double().cpu().t()
    want = torch.zeros(n, experts + (1 if identity else 0), dtype=torch.float64)
    for t in range(n):
        for e, s in plain.route(z[t], correction.double().cpu(), top, groups, keep).items():
            want[t, e if e < experts else experts] += s
    close(share, want, torch.float32, "shares", 2e-5)
    assert float((share.sum(dim=1) - 1.0).abs().max()) < 1e-5


def test_a_groups_worth_is_its_largest_score_or_the_sum_of_two():
    o = ops()
    z = torch.log(torch.tensor([[0.4, 0.02, 0.25, 0.24, 0.05, 0.04]]))
    h, router = torch.eye(6)[:1].to(DEV), torch.zeros(6, 6, device=DEV)
    router[:, 0] = z[0].to(DEV)
    for worth, want in ((1, [1.0 / 1.05, 0.05 / 1.05, 0, 0, 0, 0]), (2, [0, 0, 0.25 / 0.49, 0.24 / 0.49, 0, 0])):
        share = torch.empty(1, 6, device=DEV)
        o.moe_route(h, router, 6, 2, None, share, score="softmax", groups=3, keep=1, group_worth=worth, renormalize=True)
        assert torch.allclose(share[0].cpu(), torch.tensor(want), atol=1e-5)
    plain_share = torch.empty(1, 6, device=DEV)
    o.moe_route(h, router, 6, 2, None, plain_share, score="softmax", scale=2.0)
    assert torch.allclose(plain_share[0].cpu(), torch.tensor([0.8, 0, 0.5, 0, 0, 0]), atol=1e-5)       # not renormalised
    # choice scores below zero inside an open group beat larger ones of a closed group and are no worse for their sign
    share = torch.empty(1, 6, device=DEV)
    o.moe_route(h, router, 6, 2, None, share, score="softmax", correction=torch.tensor([0.0, -2.0, -1.0, -1.0, -1.0, -1.0], device=DEV),
                groups=3, keep=1, group_worth=1, renormalize=True)
    assert torch.allclose(share[0].cpu(), torch.tensor([0.4 / 0.42, 0.02 / 0.42, 0, 0, 0, 0]), atol=1e-5)


@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("experts,identity,top,ff,groups,keep", [(4, 2, 2, 24, 3, 2), (3, 0, 2, 9, 1, 1), (2, 4, 3, 16, 2, 1)])
def test_a_layer_of_experts_some_of_which_are_the_identity(experts, identity, top, ff, groups, keep, dtype):
    from tokenizer_b200.parts.base import ResidualStream
    width, n, limit = 40, 21, 0.8
    store = {f"p.e{e}.{name}": rnd(*shape, seed=100 + 3 * e + i, scale=0.4).cpu().bfloat16()
             for e in range(experts) for i, (name, shape) in enumerate((("gate", (ff, width)), ("up", (ff, width)), ("down", (width, ff))))}
    store["p.router"] = rnd(experts + identity, width, seed=90, scale=0.4).cpu()
    store["p.correction"] = rnd(experts + identity, seed=91, scale=0.1).cpu()
    part = part_of("feed_forward", "routed_mlp", {
        "hidden_size": width, "experts": experts, "top": top, "expert_inner": ff, "identity": identity, "score": "softmax",
        "correction": True, "groups": groups, "group_keep": keep, "group_worth": 1, "renormalize": True,
        "activation": "clamped_swish", "limit": limit, "alpha": 1.702}, store, dtype)
    h = rnd(n, width, seed=92, dtype=dtype)
    w = {k: v.double() for k, v in store.items()}
    mlp = {"expert": {"limit": limit}, "router": {"experts": experts, "top": top, "groups": {"count": groups, "keep": keep}}}
    want = plain.routed_feed_forward(h.double().cpu(), w, "p.", mlp)
    stream = ResidualStream(torch.zeros(n, width, device=DEV))
    stream.add(part.forward(h))
    close(stream.flush(), want, dtype, "the layer's output")
    if identity:
        without = plain.routed_feed_forward(h.double().cpu(), w, "p.", mlp) - want
        assert float(without.abs().max()) == 0.0
        z = plain.linear(h.double().cpu(), w["p.router"])
        through = [sum(s for e, s in plain.route(z[t], w["p.correction"], top, groups, keep).items() if e >= experts) for t in range(n)]
        assert max(through) > 0.2 and min(through) < 1.0


# ---- whole models -----------------------------------------------------------------------------------
LENGTHS = {"a": [1, 2, 23, 100, 131, 49], "b": [5, 19, 97, 201, 260, 100], "c": [3, 40, 130, 64, 1, 90],
           "d": [4, 31, 77, 150, 9, 60]}


def close_calls(raw, w, ids, below=0.02):
    """The positions of `ids` at which some layer of experts decides between two choice scores closer than `below`
    of a score's usual size (an expert in or out, a group in or out), from the plain implementation: there the
    rounding of bfloat16 anywhere upstream decides which expert is used, so the comparisons in bfloat16 leave these
    positions out; in float32 nothing is left out."""
    found, inner, row = set(), plain.route, [0]

    def spy(z, correction, top, groups, keep):
        s = torch.softmax(z, dim=-1) + correction
        size = z.shape[0] // groups
        worth = torch.stack([s[g * size:(g + 1) * size].max() for g in range(groups)]).sort(descending=True)
        tight = keep < groups and float(worth.values[keep - 1] - worth.values[keep]) < below
        inside = torch.cat([s[g * size:(g + 1) * size] for g in worth.indices[:keep].tolist()]).sort(descending=True).values
        tight = tight or (top < inside.shape[0] and float(inside[top - 1] - inside[top]) < below)
        if tight:
            found.add(row[0] % len(ids))
        row[0] += 1
        return inner(z, correction, top, groups, keep)
    plain.route = spy
    try:
        plain.forward(raw, w, list(ids))
    finally:
        plain.route = inner
    return found


_CLOSE_CALLS = {}     # id of a fixture's reference logits -> {request: positions with a close call}


@pytest.fixture(scope="module", params=sorted(TINY))
def model(request, tmp_path_factory):
    folder, cfg, page = make_folder(tmp_path_factory, request.param)
    requests = {f"r{i}": random_ids(n, cfg.vocab, 300 + i) for i, n in enumerate(LENGTHS[request.param])}
    want = reference_logits(folder, requests)
    raw, w = plain.load_folder(folder)
    _CLOSE_CALLS[id(want)] = {name: close_calls(raw, w, ids) for name, ids in requests.items()}
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
    logits of these tiny models at a few parts in a hundred, while a key, a window's edge, a state or an
    expert's weight that is wrong moves a position's logits by their own size.  Positions at which the choice of
    experts is a close call are left out; a token that chose another expert still sits in the cache of the tokens
    behind it, so two positions in a hundred may lie beyond the bound."""
    if dtype == "float32":
        return ru.compare(got, want, dtype, what)
    rel, where = [], []
    skip = _CLOSE_CALLS.get(id(want), {})
    for name in sorted(got):
        for position in sorted(got[name]):
            if position in skip.get(name, ()):
                continue
            row, ref = got[name][position], want[name][position]
            assert np.isfinite(row).all(), f"{what}: {name}[{position}] not finite"
            d, c = row - ref, ref - ref.mean()
            rel.append(float(np.sqrt(((d - d.mean()) ** 2).mean()) / np.sqrt((c ** 2).mean())))
            where.append((name, position))
    rel = np.array(rel)
    far = int((rel > 0.25).sum())
    worst = int(rel.argmax())
    assert far <= max(1, 0.02 * len(rel)), \
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
    and pages between the kept first tokens and the window are given back."""
    folder, cfg, page, requests, want = model
    steps = ru.steps_decode_tail(requests, 60)
    budget = max(ru.rounded64(len(v)) for v in requests.values())
    got = ru.collect(steps, replay(folder, dtype, steps, budget, page))
    compare(got, want, dtype, "decode tail")


def test_every_token_alone_from_the_first(model):
    """A sequence fed one token a step from its very first: the kept first tokens arrive one by one."""
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


def test_sizes_that_tiny_models_make_equal_or_one(tmp_path_factory):
    """One head, one lane of most things, one expert; models of one kind of mixer alone (no keys kept at all, no
    matrices kept at all); a loop over every layer; no feed-forward anywhere."""
    from tiny_kazepel import attention, config, delta, moe
    from tokenizer_b200 import write_random_model
    ones = config([attention(1, 1, 16, 16, 0.25, size=2, keep=1, rot=(10.0, 2, (1.0, 16, 2.0, 1.0)), mlp=moe(1, 1, 8, 1.0)),
                   delta(1, 1, 8, 1, 2, mlp=moe(1, 1, 1, 1.0, groups=(2, 1), identity=1))],
                  vocab=40, width=16, eps=1e-6, logit_scale=1.0, loop=(0, 2, 2))
    matrices = config([delta(4, 1, 32, 32, 4, mlp=moe(3, 1, 8, 0.5)), delta(2, 2, 64, 36, 3)], vocab=90, width=48, eps=1e-6)
    keys = config([attention(8, 8, 16, 16, 0.3, size=9, keep=40, rot=(100.0, 16, (4.0, 64, 8.0, 1.0))),
                   attention(2, 1, 32, 80, 0.2, size=30, keep=0), attention(2, 1, 32, 32, 0.2, size=24, keep=8, rot=(100.0, 12, None)),
                   attention(2, 1, 32, 32, 0.2, size=24, keep=9), attention(2, 1, 32, 32, 0.2, size=25, keep=9)],
                  vocab=60, width=40, eps=1e-6, logit_scale=2.0, loop=(0, 5, 1))
    for at, cfg in enumerate((ones, matrices, keys)):
        folder, page = str(tmp_path_factory.mktemp(f"kazepel_more{at}")), 16
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
    """More rows than the one-kernel step makes its low-rank products for itself, against each request alone."""
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
    if dtype != "float32":      # a token chosen where the experts' choice is a close call says nothing in bfloat16
        for position in close_calls(cfg, w, list(prompt) + list(tokens)):
            if len(prompt) - 1 <= position < len(prompt) - 1 + len(tokens):
                gap[position - (len(prompt) - 1)] = 0.0
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
    decoded tokens, pages behind them are given back, the first tokens' stay."""
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
