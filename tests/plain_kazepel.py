"""A plain, slow restatement of the Kazepel decoder on the CPU, one function per mechanism, token by
token where a mechanism is a recurrence.  It reads config.json and the weight file itself and shares
nothing with the engine: it is what the engine is compared with.

Everything is computed in float64 unless `dtype` says otherwise, so that it stands between the engine's
two precisions as the exact answer.
"""
import json
import math
import os

import torch


def load_folder(folder, dtype=torch.float64):
    from safetensors.torch import load_file
    with open(os.path.join(folder, "config.json")) as fh:
        cfg = json.load(fh)
    weights = {k: (v.to(dtype) if v.is_floating_point() else v)
               for k, v in load_file(os.path.join(folder, "model.safetensors")).items()}
    return cfg, weights


# ---- mechanisms ---------------------------------------------------------------------------
def linear(x, w):
    return x @ w.t()


def sigmoid(x):
    return 1.0 / (1.0 + torch.exp(-x))


def silu(x):
    return x * sigmoid(x)


def softplus(x):
    return torch.where(x > 30, x, torch.log1p(torch.exp(torch.clamp(x, max=30))))


def dynamic_tanh(x, alpha, gain, bias):
    """tanh(alpha x) gain + bias, element by element: no statistics of the row."""
    return torch.tanh(alpha * x) * gain + bias


def short_convolution(x, taps):
    """Causal convolution over time, channel by channel, from zeros.  x [T, C], taps [C, n] with the last
    column weighing the current token."""
    n = taps.shape[1]
    full = torch.cat([torch.zeros(n - 1, x.shape[1], dtype=x.dtype), x], dim=0)
    out = torch.zeros_like(x)
    for j in range(n):
        out = out + full[j:j + x.shape[0]] * taps[:, j]
    return out


def unit_vectors(x):
    """Every vector of the last axis divided by sqrt(sum of squares + 1e-6)."""
    return x / torch.sqrt((x * x).sum(dim=-1, keepdim=True) + 1e-6)


def channel_delta_rule(q, k, v, beta, decay, state=None):
    """One head.  q, k, decay [T, dim], v [T, vdim], beta [T].  Per token every ROW of S is multiplied by
    its own decay, then u = beta (v - S^T k), S <- S + k u^T, o = S^T q.  Returns o [T, vdim] and the last S."""
    S = torch.zeros(q.shape[1], v.shape[1], dtype=q.dtype) if state is None else state.clone()
    rows = []
    for t in range(q.shape[0]):
        S = decay[t][:, None] * S
        u = beta[t] * (v[t] - S.t() @ k[t])
        S = S + torch.outer(k[t], u)
        rows.append(S.t() @ q[t])
    return torch.stack(rows), S


def delta_mixer(h, w, prefix, m, eps):
    """The delta rule with one decay a key channel over a whole sequence from its start.  h [T, width]."""
    heads, groups, dim, vdim = m["heads"], m["kv_heads"], m["dim"], m["vdim"]
    T = h.shape[0]
    q = short_convolution(linear(h, w[prefix + "q"]), w[prefix + "q.conv"])
    k = short_convolution(linear(h, w[prefix + "k"]), w[prefix + "k.conv"])
    v = short_convolution(linear(h, w[prefix + "v"]), w[prefix + "v.conv"])
    q = unit_vectors(silu(q).view(T, groups, dim)) * dim ** -0.5
    k = unit_vectors(silu(k).view(T, groups, dim))
    v = silu(v).view(T, heads, vdim)
    beta = sigmoid(linear(h, w[prefix + "b"]))
    pre = linear(linear(h, w[prefix + "a1"]), w[prefix + "a2"]) + w[prefix + "dt_bias"]
    decay = torch.exp(-torch.exp(w[prefix + "A_log"])[None, :, None] * softplus(pre).view(T, heads, dim))
    gate = sigmoid(linear(linear(h, w[prefix + "g1"]), w[prefix + "g2"])).view(T, heads, vdim)
    outs = []
    for head in range(heads):
        g = head // (heads // groups)
        o, _ = channel_delta_rule(q[:, g], k[:, g], v[:, head], beta[:, head], decay[:, head])
        o = o / torch.sqrt((o * o).mean(dim=-1, keepdim=True) + eps) * w[prefix + "norm"]
        outs.append(o * gate[:, head])
    return linear(torch.cat(outs, dim=1), w[prefix + "o"])


def yarn_frequencies(base, dims, scaling):
    """(frequencies of the dims / 2 pairs, the factor on cosine and sine).  A frequency is divided by the
    factor where the ramp is 1 and kept where it is 0; the ramp rises between the pair that turns `fast`
    times over the original length and the one that turns `slow` times."""
    freqs = [base ** (-2.0 * i / dims) for i in range(dims // 2)]
    if scaling is None:
        return freqs, 1.0
    factor, original = float(scaling["factor"]), float(scaling["original"])

    def pair_that_turns(times):
        return dims * math.log(original / (2.0 * math.pi * times)) / (2.0 * math.log(base))

    lo = max(math.floor(pair_that_turns(float(scaling["fast"]))), 0)
    hi = min(math.ceil(pair_that_turns(float(scaling["slow"]))), dims - 1)
    out = []
    for i, f in enumerate(freqs):
        ramp = min(max((i - lo) / max(hi - lo, 0.001), 0.0), 1.0)
        out.append(f / factor * ramp + f * (1.0 - ramp))
    return out, 0.1 * math.log(factor) + 1.0


def rotate_halves(x, positions, freqs, magnitude):
    """Rotation of the first 2 n lanes of the last axis (n frequencies), lane i paired with lane i + n,
    cosine and sine multiplied by `magnitude`; the other lanes pass.  x [T, heads, lanes]."""
    out = x.clone()
    n = len(freqs)
    for i, f in enumerate(freqs):
        angle = positions.to(x.dtype) * f
        c, s = torch.cos(angle)[:, None] * magnitude, torch.sin(angle)[:, None] * magnitude
        a, b = x[..., i], x[..., i + n]
        out[..., i] = a * c - b * s
        out[..., i + n] = b * c + a * s
    return out


def seen_keys(T, mask):
    """[T, T] bool: position i sees j <= i with i - j < size or j < keep_first (no mask: every j <= i)."""
    i, j = torch.arange(T)[:, None], torch.arange(T)[None, :]
    seen = j <= i
    if mask is not None:
        seen = seen & ((i - j < int(mask["size"])) | (j < int(mask.get("keep_first", 0))))
    return seen


def softmax_one(scores):
    """exp(s) / (1 + sum exp(s)) over the last axis (hidden scores are -inf)."""
    top = torch.clamp(scores.max(dim=-1, keepdim=True).values, min=0.0)
    e = torch.exp(scores - top)
    return e / (torch.exp(-top) + e.sum(dim=-1, keepdim=True))


def windowed_attention(h, w, prefix, m):
    heads, groups, dim, vdim = m["heads"], m["kv_heads"], m["dim"], m["vdim"]
    T = h.shape[0]
    positions = torch.arange(T)
    q = linear(h, w[prefix + "q"]).view(T, heads, dim)
    k = linear(h, w[prefix + "k"]).view(T, groups, dim)
    v = linear(h, w[prefix + "v"]).view(T, groups, vdim)
    if m.get("rot") is not None:
        freqs, magnitude = yarn_frequencies(float(m["rot"]["base"]), int(m["rot"]["dims"]), m["rot"].get("scaling"))
        q = rotate_halves(q, positions, freqs, magnitude)
        k = rotate_halves(k, positions, freqs, magnitude)
    seen = seen_keys(T, m.get("mask"))
    outs = []
    for head in range(heads):
        g = head // (heads // groups)
        score = (q[:, head] @ k[:, g].t()) * float(m["scale"])
        outs.append(softmax_one(score.masked_fill(~seen, -math.inf)) @ v[:, g])
    return linear(torch.cat(outs, dim=1), w[prefix + "o"])


def clamped_expert(h, w, prefix, limit):
    g = torch.clamp(linear(h, w[prefix + "gate"]), max=limit)
    u = torch.clamp(linear(h, w[prefix + "up"]), min=-limit, max=limit)
    return linear(g * sigmoid(1.702 * g) * (u + 1.0), w[prefix + "down"])


def route(z, correction, top, groups, keep):
    """One token's router outputs z -> {expert: weight}.  Scores are the softmax over all outputs; the choice
    is made on scores + correction inside the `keep` groups of neighbours whose largest choice score is
    largest; the weights are the chosen scores without the correction, brought to a sum of one."""
    s = torch.softmax(z, dim=-1)
    choice = s + correction
    size = z.shape[0] // groups
    worth = [float(choice[g * size:(g + 1) * size].max()) for g in range(groups)]
    best = sorted(range(groups), key=lambda g: (-worth[g], g))[:keep]
    candidates = [e for g in best for e in range(g * size, (g + 1) * size)]
    chosen = sorted(candidates, key=lambda e: (-float(choice[e]), e))[:top]
    total = sum(float(s[e]) for e in chosen) + 1e-20
    return {e: float(s[e]) / total for e in chosen}


def routed_feed_forward(h, w, prefix, mlp):
    """The last `identity` router outputs stand for the input itself."""
    router = mlp["router"]
    experts, top = int(router["experts"]), int(router["top"])
    groups = router.get("groups") or {"count": 1, "keep": 1}
    z = linear(h, w[prefix + "router"])
    out = torch.zeros_like(h)
    for t in range(h.shape[0]):
        shares = route(z[t], w[prefix + "correction"], top, int(groups["count"]), int(groups["keep"]))
        for e, share in shares.items():
            if e >= experts:
                out[t] = out[t] + share * h[t]
            else:
                out[t] = out[t] + share * clamped_expert(h[t:t + 1], w, f"{prefix}e{e}.", float(mlp["expert"]["limit"]))[0]
    return out


# ---- the model ----------------------------------------------------------------------------
def run_order(cfg):
    """[(layer, pass number or None)]: the layers before the loop, the looped layers `times` times, the
    rest; the pass number stands at a pass's first layer."""
    n = len(cfg["layers"])
    loop = cfg.get("loop")
    if not loop or int(loop["stop"]) <= int(loop["start"]):
        return [(i, None) for i in range(n)]
    start, stop, times = int(loop["start"]), int(loop["stop"]), int(loop["times"])
    order = [(i, None) for i in range(start)]
    for t in range(times):
        order += [(i, t if i == start else None) for i in range(start, stop)]
    return order + [(i, None) for i in range(stop, n)]


def enter_pass(x, x0, w_in, step):
    """What a pass of the looped layers starts from: W_in on the stream and the embedding's output side by
    side, plus the pass's vector."""
    return linear(torch.cat([x, x0], dim=1), w_in) + step


def forward(cfg, w, ids, keep=None):
    """Logits [T, vocab] of a whole sequence from its start.  `keep` (a list) receives the residual stream
    after every layer run."""
    eps = float(cfg["norm"]["eps"])

    def norm(x, name):
        return dynamic_tanh(x, w[name + ".alpha"], w[name], w[name + ".b"])

    x0 = w["embed"][torch.tensor(list(ids), dtype=torch.long)]
    x = x0.clone()
    for index, turn in run_order(cfg):
        layer, p = cfg["layers"][index], f"l{index}."
        if turn is not None:
            x = enter_pass(x, x0, w["loop.in"], w["loop.step"][turn])
        h = norm(x, p + "norm1")
        if layer["type"] == "channel_delta":
            x = x + delta_mixer(h, w, p + "mix.", layer["mixer"], eps)
        elif layer["type"] == "attention":
            x = x + windowed_attention(h, w, p + "mix.", layer["mixer"])
        else:
            raise ValueError(f"unknown layer type {layer['type']!r}")
        if layer.get("mlp") is not None:
            x = x + routed_feed_forward(norm(x, p + "norm2"), w, p + "mlp.", layer["mlp"])
        if keep is not None:
            keep.append(x.clone())
    return linear(norm(x, "final.norm"), w["embed"]) * float(cfg.get("logit_scale", 1.0))


def greedy_generate(cfg, w, prompt, n_new):
    ids, out = list(prompt), []
    for _ in range(n_new):
        out.append(int(torch.argmax(forward(cfg, w, ids)[-1])))
        ids.append(out[-1])
    return out
