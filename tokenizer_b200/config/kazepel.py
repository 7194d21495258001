"""Typed configuration of the Kazepel decoder: a small decoder-only model whose layers, listed one by one in
config.json, are pre-norm residual ones with a norm that computes no statistics, tanh(alpha x) * w + b.  A
layer's mixer is the delta rule with one decay a key channel (a linear recurrence over a matrix state per
head) or grouped-query attention with the half layout of the rotation under yarn's scaling, a sliding window that
keeps the sequence's first tokens, and one added to the softmax's denominator.  A feed-forward is made of routed
experts with a clamped activation, some of which are the identity; the router scores by the softmax over
all its outputs, chooses on corrected scores inside the best groups of neighbours and weighs by the chosen scores
brought to a sum of one.  A run of layers may be passed through several times with the same weights; every
pass starts from a projection of the stream and the embedding's output side by side, plus a vector of the pass.
Logits come from the embedding table, times a constant.

config.json keys: `architecture` ("Kazepel"), `vocab`, `width`, `norm.eps`, `logit_scale` (optional),
`loop` {start, stop, times} (optional: layers start .. stop - 1 run `times` times; each pass has caches and
states of its own), and `layers`: a list of {`type`, `mixer`, `mlp`}.
  type "channel_delta": mixer {heads, kv_heads, dim, vdim, conv}
  type "attention":     mixer {heads, kv_heads, dim, vdim, scale, mask {size, keep_first} (optional), rot {base,
                        dims, scaling {factor, original, fast, slow} (optional)} (optional)}
  mlp: null, or {kind "moe", expert {ff, limit}, router {experts, top, groups {count, keep} (optional),
       identity (optional)}}
Tensors: `embed`, `loop.in`, `loop.step`, `l<i>.norm1`, `.norm2`, `final.norm` (each with `.b` and `.alpha`),
`l<i>.mix.*`, `l<i>.mlp.*`.  Every size is read here or from the weight file (the ranks of the delta rule's
bottlenecks); none stands in the parts.
"""
from __future__ import annotations

import copy
from typing import Any, Dict, List, Optional

from .registry import register_architecture
from .spec import ConfigError, LayerCall, LayerSpec, ModelSpec, PartSpec, as_float, as_int, require_keys

ARCHITECTURE = "Kazepel"
# the slope inside the sigmoid of the experts' activation: the design fixes it
EXPERT_ALPHA = 1.702
# The design has no longest position (angles are computed, not tabulated); what the engine uses
# as its bound on a request's length.
POSITIONS = 1 << 20


def _object(raw: Dict[str, Any], key: str, what: str) -> Dict[str, Any]:
    value = raw.get(key)
    if not isinstance(value, dict):
        raise ConfigError(f"{what}: {key} must be an object")
    return value


class KazepelConfig:
    def __init__(self, raw: Dict[str, Any]):
        self.raw = raw
        self.vocab = as_int(raw, "vocab", 1)
        self.width = as_int(raw, "width", 1)
        self.eps = as_float(_object(raw, "norm", ARCHITECTURE), "eps")
        if self.eps < 0:
            raise ConfigError("norm.eps must not be negative")
        self.logit_scale = as_float(raw, "logit_scale") if raw.get("logit_scale") is not None else 1.0
        self.layers: List[Dict[str, Any]] = raw["layers"]
        if not isinstance(self.layers, list) or not self.layers:
            raise ConfigError("config.json layers must be a list with at least one layer")
        for index, layer in enumerate(self.layers):
            self._check_layer(index, layer)
        self.loop: Optional[Dict[str, int]] = None
        if raw.get("loop") is not None:
            loop = _object(raw, "loop", ARCHITECTURE)
            require_keys(loop, ["start", "stop", "times"], ARCHITECTURE + " loop")
            start, stop, times = as_int(loop, "start", 0), as_int(loop, "stop", 0), as_int(loop, "times", 1)
            if stop > len(self.layers) or start > stop:
                raise ConfigError(f"loop {start} .. {stop} does not lie inside the {len(self.layers)} layers")
            if stop > start:
                self.loop = {"start": start, "stop": stop, "times": times}

    # ---- checks ------------------------------------------------------------------------------
    @staticmethod
    def _check_heads(m: Dict[str, Any], keys: List[str], what: str) -> None:
        require_keys(m, keys, what)
        for key in keys:
            as_int(m, key, 1)
        if m["heads"] % m["kv_heads"]:
            raise ConfigError(f"{what}: {m['heads']} heads do not divide into {m['kv_heads']} kv_heads")

    @classmethod
    def _check_attention(cls, m: Dict[str, Any], what: str) -> None:
        cls._check_heads(m, ["heads", "kv_heads", "dim", "vdim"], what)
        require_keys(m, ["scale"], what)
        as_float(m, "scale")
        if m.get("mask") is not None:
            mask = _object(m, "mask", what)
            require_keys(mask, ["size"], what + " mask")
            as_int(mask, "size", 1)
            if mask.get("keep_first") is not None:
                as_int(mask, "keep_first", 0)
        if m.get("rot") is None:
            return
        rot = _object(m, "rot", what)
        require_keys(rot, ["base", "dims"], what + " rot")
        dims = as_int(rot, "dims", 2)
        if dims % 2 or dims > m["dim"] or as_float(rot, "base") <= 0:
            raise ConfigError(f"{what}: rot.dims must be even and at most dim, rot.base positive")
        if rot.get("scaling") is None:
            return
        scaling = _object(rot, "scaling", what + " rot")
        keys = ["factor", "original", "fast", "slow"]
        require_keys(scaling, keys, what + " rot.scaling")
        if any(as_float(scaling, key) <= 0 for key in keys) or as_float(rot, "base") == 1.0:
            raise ConfigError(f"{what}: the numbers of rot.scaling must be positive, and rot.base not 1")

    @staticmethod
    def _check_mlp(mlp: Any, what: str) -> None:
        if mlp is None:
            return
        if not isinstance(mlp, dict) or mlp.get("kind") != "moe":
            raise ConfigError(f"{what}: mlp is null or an object of kind moe")
        expert = _object(mlp, "expert", what + " mlp")
        require_keys(expert, ["ff", "limit"], what + " mlp.expert")
        as_int(expert, "ff", 1)
        as_float(expert, "limit")
        router = _object(mlp, "router", what + " mlp")
        require_keys(router, ["experts", "top"], what + " mlp.router")
        outputs = as_int(router, "experts", 1) + (as_int(router, "identity", 0) if router.get("identity") is not None else 0)
        top, count, keep = as_int(router, "top", 1), 1, 1
        if router.get("groups") is not None:
            groups = _object(router, "groups", what + " mlp.router")
            require_keys(groups, ["count", "keep"], what + " mlp.router.groups")
            count, keep = as_int(groups, "count", 1), as_int(groups, "keep", 1)
        if outputs % count or keep > count or keep * (outputs // count) < top:
            raise ConfigError(f"{what}: {outputs} experts in {count} groups of which {keep} are kept cannot give a "
                              f"token {top} experts")

    @classmethod
    def _check_layer(cls, index: int, layer: Dict[str, Any]) -> None:
        what = f"{ARCHITECTURE} layer {index}"
        if not isinstance(layer, dict):
            raise ConfigError(f"{what} must be an object")
        require_keys(layer, ["type", "mixer"], what)
        m = _object(layer, "mixer", what)
        if layer["type"] == "channel_delta":
            cls._check_heads(m, ["heads", "kv_heads", "dim", "vdim", "conv"], what + " mixer")
        elif layer["type"] == "attention":
            cls._check_attention(m, what + " mixer")
        else:
            raise ConfigError(f"{what}: unknown type {layer['type']!r} (known: attention, channel_delta)")
        cls._check_mlp(layer.get("mlp"), what)

    @classmethod
    def from_dict(cls, raw: Dict[str, Any]) -> "KazepelConfig":
        require_keys(raw, ["vocab", "width", "layers", "norm"], ARCHITECTURE)
        return cls(copy.deepcopy(raw))

    def to_dict(self) -> Dict[str, Any]:
        out = copy.deepcopy(self.raw)
        out.pop("architectures", None)
        out["architecture"] = ARCHITECTURE
        return out

    # ---- the model as data -------------------------------------------------------------------
    def _mixer(self, index: int, layer: Dict[str, Any]) -> PartSpec:
        m, prefix = layer["mixer"], f"l{index}.mix"
        common = {"hidden_size": self.width, "heads": m["heads"], "kv_heads": m["kv_heads"], "dim": m["dim"],
                  "vdim": m["vdim"]}
        if layer["type"] == "channel_delta":
            return PartSpec("channel_delta_net", dict(common, conv=m["conv"], eps=self.eps), prefix)
        mask, rot, position = m.get("mask"), m.get("rot"), None
        if rot is not None:
            scaling = None
            if rot.get("scaling") is not None:
                s = rot["scaling"]
                scaling = {"kind": "yarn", "factor": float(s["factor"]), "original": float(s["original"]),
                           "fast": float(s["fast"]), "slow": float(s["slow"])}
            position = PartSpec("rope_half", {"base": float(rot["base"]), "dims": int(rot["dims"]), "scaling": scaling})
        # a window of n keys: the position itself and the n - 1 before it
        return PartSpec("gqa_rotary", dict(
            common, scale=float(m["scale"]), bias=False, position=position, unit_sink=True, chunk=None,
            window=int(mask["size"]) - 1 if mask is not None else None,
            keep_first=int(mask.get("keep_first") or 0) if mask is not None else 0), prefix)

    def _feed_forward(self, index: int, mlp: Dict[str, Any]) -> PartSpec:
        router = mlp["router"]
        groups = router.get("groups") or {"count": 1, "keep": 1}
        return PartSpec("routed_mlp", {
            "hidden_size": self.width, "experts": router["experts"], "top": router["top"],
            "expert_inner": mlp["expert"]["ff"], "identity": router.get("identity") or 0, "score": "softmax",
            "correction": True, "groups": groups["count"], "group_keep": groups["keep"], "group_worth": 1,
            "renormalize": True, "activation": "clamped_swish", "limit": float(mlp["expert"]["limit"]),
            "alpha": EXPERT_ALPHA}, f"l{index}.mlp")

    def _norm(self, name: str, scale: float = 1.0) -> PartSpec:
        params = {"size": self.width, "tensor": name}
        if scale != 1.0:
            params["scale"] = scale
        return PartSpec("dynamic_tanh", params, name)

    def run_order(self) -> List[LayerCall]:
        """The calls of the layers: those before the loop, the looped ones `times` times (each call with a cache
        and state of its own), the rest.  A pass's first call carries what the pass starts from."""
        n = len(self.layers)
        if self.loop is None:
            return [LayerCall(i) for i in range(n)]
        start, stop, times = self.loop["start"], self.loop["stop"], self.loop["times"]
        order = [LayerCall(i) for i in range(start)]
        for t in range(times):
            entry = PartSpec("pass_projection", {"projection": "loop.in", "tensor": "loop.step", "passes": times,
                                                 "hidden_size": self.width, "index": t}, "loop")
            order += [LayerCall(i, before=entry if i == start else None) for i in range(start, stop)]
        return order + [LayerCall(i) for i in range(stop, n)]

    def model_spec(self) -> ModelSpec:
        layers = []
        for index, layer in enumerate(self.layers):
            p = f"l{index}"
            parts = dict(mixer=self._mixer(index, layer), mixer_norm=self._norm(p + ".norm1"))
            if layer.get("mlp") is None:
                layers.append(LayerSpec("pre_norm_mixer_only", **parts))
                continue
            layers.append(LayerSpec("pre_norm_residual", feed_forward=self._feed_forward(index, layer["mlp"]),
                                    feed_forward_norm=self._norm(p + ".norm2"), **parts))
        spec = ModelSpec(
            architecture=ARCHITECTURE, vocab_size=self.vocab, hidden_size=self.width, max_positions=POSITIONS,
            embedding=PartSpec("token_embedding", {"vocab_size": self.vocab, "hidden_size": self.width,
                                                   "tensor": "embed"}, "embed"),
            layers=tuple(layers), order=tuple(self.run_order()),
            # logits = (embed x) * logit_scale: the final norm's output carries the constant
            final_norm=self._norm("final.norm", self.logit_scale),
            head=PartSpec("lm_head", {"vocab_size": self.vocab, "hidden_size": self.width, "tied_to": "embed"}, "head"))
        spec.validate()
        return spec


register_architecture(ARCHITECTURE, KazepelConfig)
