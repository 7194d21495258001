"""Attention whose keys and values are expanded from a small latent per token, so that the
latent is all the cache keeps.

Per token, from the mixer's input h:
  query latent   cq = rms_norm(Wdq h) * g_q;   queries q = Wuq cq, head by head
                 [dim lanes without position | rot_dim lanes that carry the position]
  kv latent      c = rms_norm((Wdkv h)[:kv_rank]) * g_c;   the last rot_dim rows of Wdkv h are one
                 positional key part shared by all heads (not normed)
  per head       key = [Wuk_h c | rotated shared part], value = Wuv_h c,
                 score = q . key * scale, softmax (with a window and / or a sink), output Wo on the
                 concatenated heads.
The cache row of a token is [c | rotated shared part | zeros up to a multiple of 16 lanes].

How it is computed.  Nothing lies between Wuq and the score but the rotation of the positional
lanes, and nothing between the weighted sum of values and Wo, so the expansions are folded into
the projections once, at load time, in float64:
  score_h = (Wuk_h^T Wuq_h[:dim]) cq . c + rot(q_h[dim:]) . rot(shared)
  output  = sum_h (Wo[:, h] Wuv_h) (sum_j p_hj c_j)
The attention is then attention of `heads` query heads over ONE cached head of kv_rank + rot_dim
lanes whose values are the leading kv_rank lanes of the same rows: the framework's paged kernels
take it with the cache pool passed as keys and as values (the value lanes behind kv_rank meet
zero columns of the folded output projection).  Per token this costs heads * kv_rank * (q_rank +
hidden) multiply-adds for the two folded products, against heads * (dim * (q_rank + kv_rank) +
vdim * (kv_rank + hidden)) unfolded: less or about as much while the latent is not much wider than
a head.

Two parameters change the form.  `q_rank` None: there is no query latent, q = Wq h (tensor `.q`); the folded queries then
are columns of the input product, and one kernel rotates them, norms the latent and writes the cache row.
`output_gate`: the concatenated heads are multiplied by sigmoid(Wg h) (tensor `.g`, more columns of the input product) in
front of Wo.  A gate lies between the values and Wo, so these two stay apart: the weighted latents are expanded to the
heads' values by a small product a head whose epilogue applies the gate (`latent_values`).
"""
from __future__ import annotations

import torch

from ..config.spec import ConfigError
from ..kernels import ops
from ..weights.store import TensorSpec
from .attention import PagedAttention
from .base import CacheNeed, KVNeed, build_part, register_part
from .linear import Linear
from .recurrent import SideProjection, stacked_rows

ROW_MULTIPLE = 16       # cache rows are padded to whole 16 lanes (the tensor-core kernels' step)


class LatentAttention(PagedAttention, SideProjection):
    @staticmethod
    def tensors(spec):
        p, x = spec.params, spec.prefix
        hidden, heads = p["hidden_size"], p["heads"]
        rot = p.get("rot_dim", 0)
        if p["q_rank"] is None:
            out = [TensorSpec(x + ".q", (heads * (p["dim"] + rot), hidden))]
        else:
            out = [TensorSpec(x + ".dq", (p["q_rank"], hidden)),
                   TensorSpec(x + ".dq.norm", (p["q_rank"],), "one_plus_normal"),
                   TensorSpec(x + ".uq", (heads * (p["dim"] + rot), p["q_rank"]))]
        out += [TensorSpec(x + ".dkv", (p["kv_rank"] + rot, hidden)),
               TensorSpec(x + ".dkv.norm", (p["kv_rank"],), "one_plus_normal"),
               TensorSpec(x + ".uk", (heads * p["dim"], p["kv_rank"])),
               TensorSpec(x + ".uv", (heads * p["vdim"], p["kv_rank"]))]
        if p.get("sink"):
            out.append(TensorSpec(x + ".sink", (heads,), "normal", 1.0))
        if p.get("output_gate"):
            out.append(TensorSpec(x + ".g", (heads * p["vdim"], hidden)))
        out.append(TensorSpec(x + ".o", (hidden, heads * p["vdim"])))
        return out

    def __init__(self, spec, store, runtime):
        p, x = spec.params, spec.prefix
        self.runtime = runtime
        self.hidden, self.heads = int(p["hidden_size"]), int(p["heads"])
        self.dim, self.vdim = int(p["dim"]), int(p["vdim"])
        self.q_rank, self.kv_rank = int(p["q_rank"]) if p["q_rank"] is not None else None, int(p["kv_rank"])
        self.gated = bool(p.get("output_gate"))
        self.rot_dim = int(p.get("rot_dim", 0))
        self.eps = float(p["eps"])
        self.scale = float(p["scale"])
        self.window = p.get("window")          # None: every earlier key; n: the n keys before the query too
        if self.window is not None and int(self.window) < 0:
            raise ConfigError("a window reaches back a number of keys that is not negative")
        self.position = None
        self.rot_dims = 0
        if self.rot_dim:
            if p.get("position") is None:
                raise ConfigError("latent attention with positional lanes needs a position encoding")
            self.position = build_part("position", p["position"], store, runtime)
            self.rot_dims = self.position.dims
            if self.rot_dims > self.rot_dim:
                raise ConfigError(f"{self.rot_dims} rotated lanes do not fit {self.rot_dim} positional lanes")
        # what the paged kernels see: `heads` query heads over one cached head of `row` lanes
        self.nh, self.nkv = self.heads, 1
        self.row = -(-(self.kv_rank + self.rot_dim) // ROW_MULTIPLE) * ROW_MULTIPLE
        self.d = self.row
        self.sink = runtime.vector(store.get(x + ".sink")) if p.get("sink") else None
        self.c_gain = runtime.vector(store.get(x + ".dkv.norm"))
        # the input product, block by block: the latents, and behind them (in whole 8s) queries and gate where they
        # come straight from the mixer's input
        latents = [store.get(x + ".dkv")]
        if self.q_rank is None:
            queries = self._fold_queries(store.get(x + ".q"), store.get(x + ".uk"), self.hidden)
        else:
            self.q_gain = runtime.vector(store.get(x + ".dq.norm"))
            latents = [store.get(x + ".dq")] + latents
            self.q_proj = Linear(runtime.matrix(self._fold_queries(store.get(x + ".uq"), store.get(x + ".uk"), self.q_rank)))
        self._own = latents
        if self.q_rank is None or self.gated:
            self._own = [stacked_rows([w.to(torch.float32) for w in latents])]
        self.q_at = self.g_at = sum(w.shape[0] for w in self._own)
        if self.q_rank is None:
            self._own.append(queries)
            self.g_at += self.heads * self.row
        if self.gated:
            self._own.append(stacked_rows([store.get(x + ".g").to(torch.float32)]))
        self.inputs = self._stack(runtime, list(self._own), [None] * len(self._own), None)
        if self.gated:
            self.values = self._value_weights(store.get(x + ".uv"))
            self.out = Linear(runtime.matrix(store.get(x + ".o")))
        else:
            self.out = Linear(runtime.matrix(self._fold_output(store.get(x + ".uv"), store.get(x + ".o"))))

    def _value_weights(self, uv):
        """A head's values from a weighted cache row, as `latent_values` wants them: zero beyond the latent's lanes."""
        values = torch.zeros((self.heads, self.vdim, self.row), dtype=torch.float32, device=uv.device)
        values[:, :, :self.kv_rank] = uv.to(torch.float32).view(self.heads, self.vdim, self.kv_rank)
        return self.runtime.matrix(values if self.runtime.dtype == torch.bfloat16 else values.transpose(1, 2))

    def _fold_queries(self, uq, uk, inner):
        """Queries straight into the cache row's lanes, [heads * row, inner], from Wuq [heads * (dim + rot), inner] and
        Wuk: float64 products rounded once to float32."""
        H, dim, rank, rot, row, f64 = self.heads, self.dim, self.kv_rank, self.rot_dim, self.row, torch.float64
        uq = uq.to(f64).view(H, dim + rot, inner)
        uk = uk.to(f64).view(H, dim, rank)
        q_folded = torch.zeros((H, row, inner), dtype=f64, device=uq.device)
        q_folded[:, :rank] = torch.matmul(uk.transpose(1, 2), uq[:, :dim])
        q_folded[:, rank:rank + rot] = uq[:, dim:]
        return q_folded.view(H * row, inner).to(torch.float32)

    def _fold_output(self, uv, o):
        """The output projection straight from the weighted latents [hidden, heads * row], a float64 product rounded
        once."""
        H, vdim, rank, f64 = self.heads, self.vdim, self.kv_rank, torch.float64
        uv, o = uv.to(f64).view(H, vdim, rank), o.to(f64).view(self.hidden, H, vdim)
        o_folded = torch.zeros((self.hidden, H, self.row), dtype=f64, device=uv.device)
        o_folded[:, :, :rank] = torch.einsum("ohv,hvr->ohr", o, uv)
        return o_folded.view(self.hidden, H * self.row).to(torch.float32)

    def take_side(self, weight, bias):
        self.inputs = self._stack(self.runtime, list(self._own), [None] * len(self._own), (weight, bias))

    def cache_need(self):
        return CacheNeed(kv=KVNeed(1, self.row, self.window, planes=1))

    def streamed_weights(self):
        return [self.inputs.weight] + ([self.q_proj.weight] if self.q_rank is not None else []) + \
            ([self.values] if self.gated else []) + [self.out.weight]

    def _queries(self, product, ctx, group, cache):
        """The heads' queries in the cache row's lanes, rotated; the token's cache row is written on the way."""
        n, slots = ctx.n_tokens, group.slots if cache.writes else None
        if self.q_rank is None:
            q = self.runtime.empty(n, self.heads * self.row)
            ops.latent_rotate_store(product, 0, self.q_at, self.heads, self.kv_rank, self.rot_dim, self.rot_dims, self.row,
                                    self.c_gain, self.eps, self.position.inv_freq64 if self.position is not None else None,
                                    ctx.pos, ctx.row_req, slots, q, cache.k_pool)
            return q
        cq = self.runtime.empty(n, self.q_rank)
        freq = self.position.inv_freq if self.position is not None else None
        ops.latent_prepare(product, 0, self.q_rank, self.q_rank, self.kv_rank, self.rot_dim, self.rot_dims,
                           self.q_gain, self.c_gain, self.eps, freq, ctx.pos, ctx.row_req, slots, cq, cache.k_pool)
        q = self.q_proj.forward(cq)
        if self.rot_dims:
            ops.rotate_interleaved(q, self.heads, self.kv_rank, self.rot_dims, freq, ctx.pos, ctx.row_req)
        return q

    def forward(self, h, ctx, cache):
        group = ctx.groups[cache.group]
        product = self.inputs.forward(h, out_dtype=torch.float32)
        q = self._queries(product, ctx, group, cache)
        mixed = self.runtime.empty(ctx.n_tokens, self.heads * self.row)
        self.attend(q, mixed, ctx, group, cache)
        if self.gated:
            y = self.runtime.empty(ctx.n_tokens, self.heads * self.vdim)
            ops.latent_values(mixed, self.values, product, self.g_at, self.heads, self.vdim, self.row, y)
            mixed = y
        self._keep_side(product)
        return self.out.forward(mixed, partials_ok=True)


register_part("mixer", "latent_attention", LatentAttention)
