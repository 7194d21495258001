"""A plain, slow restatement of the Kerudra decoder on the CPU, one function per mechanism, token by token
where a mechanism is a recurrence.  It reads config.json and the weight file itself and shares nothing with the
engine: it is what the engine is compared with.

Everything is computed in float64 unless `dtype` says otherwise, so that it stands between the engine's two
precisions as the exact answer.
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


def log_sigmoid(x):
    return torch.minimum(x, torch.zeros_like(x)) - torch.log1p(torch.exp(-x.abs()))


def rms(x, eps):
    """Every vector of the last axis divided by its root mean square, eps inside the root."""
    return x / torch.sqrt((x * x).mean(dim=-1, keepdim=True) + eps)


def rotate(x, positions, base, dims, layout):
    """Rotation of the first `dims` lanes of the last axis at the rows' positions; the other lanes pass.  Layout
    "half" pairs lane i with lane i + dims / 2, "interleaved" lane 2i with lane 2i + 1.  x [T, heads, lanes]."""
    out = x.clone()
    for i in range(dims // 2):
        angle = positions.to(x.dtype) * float(base) ** (-2.0 * i / dims)
        c, s = torch.cos(angle)[:, None], torch.sin(angle)[:, None]
        first, second = (i, i + dims // 2) if layout == "half" else (2 * i, 2 * i + 1)
        a, b = x[..., first], x[..., second]
        out[..., first] = a * c - b * s
        out[..., second] = b * c + a * s
    return out


def seen_keys(T, size=None):
    """[T, T] bool: position i sees j <= i with i - j < size (None: every j <= i)."""
    i, j = torch.arange(T)[:, None], torch.arange(T)[None, :]
    seen = j <= i
    return seen if size is None else seen & (i - j < int(size))


def softmax_rows(scores, seen):
    return torch.softmax(scores.masked_fill(~seen, -math.inf), dim=-1)


def shared_key_value_attention(h, w, prefix, m):
    """Grouped-query attention whose values are the keys as projected (bias added, not rotated)."""
    heads, groups, dim = m["heads"], m["kv_heads"], m["dim"]
    T = h.shape[0]
    positions = torch.arange(T)
    q = (linear(h, w[prefix + "q"]) + w[prefix + "q.b"]).view(T, heads, dim)
    k = (linear(h, w[prefix + "k"]) + w[prefix + "k.b"]).view(T, groups, dim)
    v = k
    if m.get("rot") is not None:
        q = rotate(q, positions, m["rot"]["base"], m["rot"]["dims"], "half")
        k = rotate(k, positions, m["rot"]["base"], m["rot"]["dims"], "half")
    seen = seen_keys(T)
    outs = []
    for head in range(heads):
        g = head // (heads // groups)
        outs.append(softmax_rows((q[:, head] @ k[:, g].t()) * float(m["scale"]), seen) @ v[:, g])
    return linear(torch.cat(outs, dim=1), w[prefix + "o"])


def latent_attention(h, w, prefix, m, eps):
    """Attention whose keys and values are expanded, head by head, from one normed latent a token; a rotated key
    part is shared by the heads; the heads' outputs pass a gate that reads h."""
    heads, dim, rot_dim, vdim, rank = m["heads"], m["dim"], m["rot_dim"], m["vdim"], m["kv_rank"]
    T = h.shape[0]
    positions = torch.arange(T)
    base, dims = m["rot"]["base"], m["rot"]["dims"]
    q = linear(h, w[prefix + "q"]).view(T, heads, dim + rot_dim)
    down = linear(h, w[prefix + "dkv"])
    c = rms(down[:, :rank], eps) * w[prefix + "dkv.norm"]
    shared = rotate(down[:, None, rank:], positions, base, dims, "interleaved")[:, 0]
    q_rot = rotate(q[..., dim:], positions, base, dims, "interleaved")
    keys = linear(c, w[prefix + "uk"]).view(T, heads, dim)
    values = linear(c, w[prefix + "uv"]).view(T, heads, vdim)
    seen = seen_keys(T, m["mask"]["size"] if m.get("mask") is not None else None)
    outs = []
    for head in range(heads):
        score = (q[:, head, :dim] @ keys[:, head].t() + q_rot[:, head] @ shared.t()) * float(m["scale"])
        outs.append(softmax_rows(score, seen) @ values[:, head])
    gate = sigmoid(linear(h, w[prefix + "g"]))
    return linear(torch.cat(outs, dim=1) * gate, w[prefix + "o"])


def matrix_memory(q, k, v, log_in, log_forget, state=None):
    """One head.  q, k [T, dim], v [T, vdim], the logarithms of the two gates [T].  The matrix S and the vector n are
    kept divided by exp of a running maximum, which starts at 0.  Returns o [T, vdim] and (S, n, maximum)."""
    if state is None:
        S = torch.zeros(q.shape[1], v.shape[1], dtype=q.dtype)
        n = torch.zeros(q.shape[1], dtype=q.dtype)
        top = torch.zeros((), dtype=q.dtype)
    else:
        S, n, top = (part.clone() for part in state)
    rows = []
    for t in range(q.shape[0]):
        new = torch.maximum(log_forget[t] + top, log_in[t])
        keep, add = torch.exp(log_forget[t] + top - new), torch.exp(log_in[t] - new)
        S = keep * S + add * torch.outer(k[t], v[t])
        n = keep * n + add * k[t]
        top = new
        rows.append((S.t() @ q[t]) / (torch.maximum((n @ q[t]).abs(), torch.exp(-top)) + 1e-6))
    return torch.stack(rows), (S, n, top)


def capped_gates(h, w, prefix, cap):
    """(log input gate, log forget gate), both [T, heads]."""
    squash = lambda z: cap * torch.tanh(z / cap)
    return (squash(linear(h, w[prefix + "i"]) + w[prefix + "i.b"]),
            log_sigmoid(squash(linear(h, w[prefix + "f"]) + w[prefix + "f.b"])))


def memory_mixer(h, w, prefix, m, eps):
    """The matrix memory over a whole sequence from its start.  h [T, width]."""
    heads, dim, vdim = m["heads"], m["dim"], m["vdim"]
    T = h.shape[0]
    q = (linear(h, w[prefix + "q"]) * dim ** -0.5).view(T, heads, dim)
    k = linear(h, w[prefix + "k"]).view(T, heads, dim)
    v = linear(h, w[prefix + "v"]).view(T, heads, vdim)
    log_in, log_forget = capped_gates(h, w, prefix, float(m["gate_cap"]))
    outs = [rms(matrix_memory(q[:, a], k[:, a], v[:, a], log_in[:, a], log_forget[:, a])[0], eps) for a in range(heads)]
    y = torch.cat(outs, dim=1) * w[prefix + "norm"] * sigmoid(linear(h, w[prefix + "g"]))
    return linear(y, w[prefix + "o"])


def squared_relu_feed_forward(h, w, prefix):
    return linear(torch.clamp(linear(h, w[prefix + "up"]), min=0.0) ** 2, w[prefix + "down"])


# ---- the streams ------------------------------------------------------------------------
def combine(xs, weights):
    """What a sublayer reads: the streams' weighted sum.  xs [streams, T, width]."""
    return sum(weights[s] * xs[s] for s in range(xs.shape[0]))


def mix_and_add(xs, mix, out, y, m):
    """Every stream anew from all the old ones and the sublayer's output: stream t is sum_s mix[s, t] x_s + m out[t] y."""
    n = xs.shape[0]
    return torch.stack([sum(mix[s, t] * xs[s] for s in range(n)) + m * out[t] * y for t in range(n)])


# ---- the model ----------------------------------------------------------------------------
def run_order(cfg):
    """Layer indices: those before the loop, the looped ones `times` times, the rest."""
    n = len(cfg["layers"])
    loop = cfg.get("loop")
    if not loop:
        return list(range(n))
    start, stop = int(loop["start"]), int(loop["stop"])
    return list(range(start)) + list(range(start, stop)) * int(loop["times"]) + list(range(stop, n))


def mixer(layer, h, w, prefix, eps):
    kind = layer["type"]
    if kind == "attention":
        return shared_key_value_attention(h, w, prefix, layer["mixer"])
    if kind == "latent_attention":
        return latent_attention(h, w, prefix, layer["mixer"], eps)
    if kind == "mlstm":
        return memory_mixer(h, w, prefix, layer["mixer"], eps)
    raise ValueError(f"unknown layer type {kind!r}")


def forward(cfg, w, ids, keep=None):
    """Logits [T, vocab] of a whole sequence from its start.  `keep` (a list) receives the streams' sum after every
    layer run."""
    eps, m = float(cfg["norm"]["eps"]), float(cfg.get("residual_mult", 1.0))
    x = w["embed"][torch.tensor(list(ids), dtype=torch.long)] * float((cfg.get("embedding") or {}).get("scale", 1.0))
    xs = torch.stack([x] * int(cfg["streams"]))
    for index in run_order(cfg):
        layer, p = cfg["layers"][index], f"l{index}."
        u = combine(xs, w[p + "hc1.in"])
        y = mixer(layer, rms(u, eps) * w[p + "norm1"], w, p + "mix.", eps)
        xs = mix_and_add(xs, w[p + "hc1.mix"], w[p + "hc1.out"], y, m)
        if layer.get("mlp") is not None:
            u = combine(xs, w[p + "hc2.in"])
            y = squared_relu_feed_forward(rms(u, eps) * w[p + "norm2"], w, p + "mlp.")
            xs = mix_and_add(xs, w[p + "hc2.mix"], w[p + "hc2.out"], y, m)
        if keep is not None:
            keep.append(xs.sum(dim=0))
    return linear(rms(xs.sum(dim=0), eps) * w["final.norm"], w["embed"]) * float(cfg.get("logit_scale", 1.0))


def greedy_generate(cfg, w, prompt, n_new):
    ids, out = list(prompt), []
    for _ in range(n_new):
        out.append(int(torch.argmax(forward(cfg, w, ids)[-1])))
        ids.append(out[-1])
    return out
