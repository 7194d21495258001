"""Typed configuration of the Kerudra decoder: a small decoder-only model whose layers, listed one by one in
config.json, run on several residual streams side by side: a sublayer reads the norm of a weighted sum of the streams,
and its output, times a constant, is added to all of them while they are mixed.  A layer's mixer is attention over a
cached latent (queries from the mixer's input, a window, a rotated key part that the heads share, a gate on the heads'
outputs), grouped-query attention whose values are its keys as projected (the half layout of the rotation, biases), or a
matrix memory with exponential gates.  The feed-forward is dense with the square of relu.  A run of layers may be passed
through several times with the same weights.  Logits come from the embedding table, times a constant.

config.json keys: `architecture` ("Kerudra"), `vocab`, `width`, `norm.eps`, `streams`, `residual_mult` (optional),
`embedding.scale` (optional), `logit_scale` (optional), `loop` {start, stop, times} (optional: layers start .. stop - 1 run
`times` times; each pass has caches and states of its own), and `layers`: a list of {`type`, `mixer`, `mlp`}.
  type "latent_attention": mixer {heads, dim, rot_dim, vdim, kv_rank, scale, rot {base, dims}, mask {size} (optional)}
  type "attention":        mixer {heads, kv_heads, dim, vdim, scale, rot {base, dims} (optional)}
  type "mlstm":            mixer {heads, dim, vdim, gate_cap}
  mlp: null, or {kind "dense", ff}
Tensors: `embed`, `l<i>.norm1`, `.norm2`, `final.norm`, `l<i>.hc1.*`, `.hc2.*`, `l<i>.mix.*`, `l<i>.mlp.*`.  Every size is
read here; none stands in the parts.
"""
from __future__ import annotations

import copy
from typing import Any, Dict, List, Optional

from .registry import register_architecture
from .spec import ConfigError, LayerCall, LayerSpec, ModelSpec, PartSpec, as_float, as_int, require_keys

ARCHITECTURE = "Kerudra"
# The design has no longest position (angles are computed, not tabulated); what the engine uses
# as its bound on a request's length.
POSITIONS = 1 << 20


def _object(raw: Dict[str, Any], key: str, what: str) -> Dict[str, Any]:
    value = raw.get(key)
    if not isinstance(value, dict):
        raise ConfigError(f"{what}: {key} must be an object")
    return value


def _optional_float(raw: Dict[str, Any], key: str) -> float:
    return as_float(raw, key) if raw.get(key) is not None else 1.0


class KerudraConfig:
    def __init__(self, raw: Dict[str, Any]):
        self.raw = raw
        self.vocab = as_int(raw, "vocab", 1)
        self.width = as_int(raw, "width", 1)
        self.streams = as_int(raw, "streams", 1)
        self.eps = as_float(_object(raw, "norm", ARCHITECTURE), "eps")
        if self.eps < 0:
            raise ConfigError("norm.eps must not be negative")
        self.residual_mult = _optional_float(raw, "residual_mult")
        self.logit_scale = _optional_float(raw, "logit_scale")
        self.embedding_scale = 1.0
        if raw.get("embedding") is not None:
            self.embedding_scale = _optional_float(_object(raw, "embedding", ARCHITECTURE), "scale")
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
            self.loop = {"start": start, "stop": stop, "times": times}

    # ---- checks ------------------------------------------------------------------------------
    @staticmethod
    def _check_sizes(m: Dict[str, Any], keys: List[str], what: str) -> None:
        require_keys(m, keys, what)
        for key in keys:
            as_int(m, key, 1)

    @staticmethod
    def _check_rotation(m: Dict[str, Any], most: int, what: str) -> None:
        rot = _object(m, "rot", what)
        require_keys(rot, ["base", "dims"], what + " rot")
        dims = as_int(rot, "dims", 2)
        if dims % 2 or dims > most or as_float(rot, "base") <= 0:
            raise ConfigError(f"{what}: rot.dims must be even and at most {most}, rot.base positive")

    @classmethod
    def _check_layer(cls, index: int, layer: Dict[str, Any]) -> None:
        what = f"{ARCHITECTURE} layer {index}"
        if not isinstance(layer, dict):
            raise ConfigError(f"{what} must be an object")
        require_keys(layer, ["type", "mixer"], what)
        m, kind = _object(layer, "mixer", what), layer["type"]
        if kind == "mlstm":
            cls._check_sizes(m, ["heads", "dim", "vdim"], what + " mixer")
            require_keys(m, ["gate_cap"], what + " mixer")
            if as_float(m, "gate_cap") <= 0:
                raise ConfigError(f"{what}: gate_cap must be positive")
        elif kind == "attention":
            cls._check_sizes(m, ["heads", "kv_heads", "dim", "vdim"], what + " mixer")
            require_keys(m, ["scale"], what + " mixer")
            as_float(m, "scale")
            if m["heads"] % m["kv_heads"]:
                raise ConfigError(f"{what}: {m['heads']} heads do not divide into {m['kv_heads']} kv_heads")
            if m["vdim"] != m["dim"]:
                raise ConfigError(f"{what}: the values are the keys, so vdim is dim; found {m['vdim']} and {m['dim']}")
            if m.get("rot") is not None:
                cls._check_rotation(m, m["dim"], what + " mixer")
        elif kind == "latent_attention":
            cls._check_sizes(m, ["heads", "dim", "rot_dim", "vdim", "kv_rank"], what + " mixer")
            require_keys(m, ["scale", "rot"], what + " mixer")
            as_float(m, "scale")
            cls._check_rotation(m, m["rot_dim"], what + " mixer")
            if m.get("mask") is not None:
                mask = _object(m, "mask", what)
                require_keys(mask, ["size"], what + " mask")
                as_int(mask, "size", 1)
        else:
            raise ConfigError(f"{what}: unknown type {kind!r} (known: attention, latent_attention, mlstm)")
        mlp = layer.get("mlp")
        if mlp is not None:
            if not isinstance(mlp, dict) or mlp.get("kind") != "dense":
                raise ConfigError(f"{what}: mlp is null or an object of kind dense")
            require_keys(mlp, ["ff"], what + " mlp")
            as_int(mlp, "ff", 1)

    @classmethod
    def from_dict(cls, raw: Dict[str, Any]) -> "KerudraConfig":
        require_keys(raw, ["vocab", "width", "layers", "norm", "streams"], ARCHITECTURE)
        return cls(copy.deepcopy(raw))

    def to_dict(self) -> Dict[str, Any]:
        out = copy.deepcopy(self.raw)
        out.pop("architectures", None)
        out["architecture"] = ARCHITECTURE
        return out

    # ---- the model as data -------------------------------------------------------------------
    def _mixer(self, index: int, layer: Dict[str, Any]) -> PartSpec:
        m, prefix, kind = layer["mixer"], f"l{index}.mix", layer["type"]
        common = {"hidden_size": self.width, "heads": m["heads"], "dim": m["dim"], "vdim": m["vdim"]}
        if kind == "mlstm":
            return PartSpec("matrix_memory", dict(common, gate_cap=float(m["gate_cap"]), eps=self.eps), prefix)
        rot, position = m.get("rot"), None
        if rot is not None:
            position = PartSpec("rope_interleaved" if kind == "latent_attention" else "rope_half",
                                {"base": float(rot["base"]), "dims": int(rot["dims"])})
        if kind == "attention":
            return PartSpec("gqa_rotary", dict(common, kv_heads=m["kv_heads"], scale=float(m["scale"]), bias=True,
                                               position=position, values_are_keys=True, window=None, chunk=None), prefix)
        # a window of n keys: the position itself and the n - 1 before it
        return PartSpec("latent_attention", dict(
            common, q_rank=None, kv_rank=m["kv_rank"], rot_dim=m["rot_dim"], scale=float(m["scale"]), eps=self.eps,
            window=int(m["mask"]["size"]) - 1 if m.get("mask") is not None else None, sink=False, position=position,
            output_gate=True), prefix)

    def _norm(self, name: str, **more) -> PartSpec:
        return PartSpec("rms_norm", dict({"size": self.width, "eps": self.eps, "tensor": name}, **more), name)

    def run_order(self) -> List[LayerCall]:
        """The calls of the layers: those before the loop, the looped ones `times` times (each call with a cache and
        state of its own), the rest."""
        n = len(self.layers)
        if self.loop is None:
            return [LayerCall(i) for i in range(n)]
        start, stop, times = self.loop["start"], self.loop["stop"], self.loop["times"]
        indices = list(range(start)) + list(range(start, stop)) * times + list(range(stop, n))
        return [LayerCall(i) for i in indices]

    def model_spec(self) -> ModelSpec:
        layers = []
        for index, layer in enumerate(self.layers):
            p = f"l{index}"
            link = {"streams": self.streams, "mult": self.residual_mult}
            parts = dict(mixer=self._mixer(index, layer), mixer_norm=self._norm(p + ".norm1"),
                         mixer_connection=PartSpec("stream_connection", dict(link), p + ".hc1"))
            if layer.get("mlp") is None:
                layers.append(LayerSpec("connected_streams_mixer_only", **parts))
                continue
            layers.append(LayerSpec(
                "connected_streams", feed_forward=PartSpec("dense_mlp", {
                    "hidden_size": self.width, "inner_size": layer["mlp"]["ff"], "activation": "relu_squared"}, p + ".mlp"),
                feed_forward_norm=self._norm(p + ".norm2"),
                feed_forward_connection=PartSpec("stream_connection", dict(link), p + ".hc2"), **parts))
        spec = ModelSpec(
            architecture=ARCHITECTURE, vocab_size=self.vocab, hidden_size=self.width, max_positions=POSITIONS,
            embedding=PartSpec("token_embedding", {"vocab_size": self.vocab, "hidden_size": self.width, "tensor": "embed",
                                                   "scale": self.embedding_scale}, "embed"),
            layers=tuple(layers), order=tuple(self.run_order()),
            # logits = (embed norm(x)) * logit_scale: the constant rides in the final norm's gain
            final_norm=self._norm("final.norm", gain_scale=self.logit_scale),
            head=PartSpec("lm_head", {"vocab_size": self.vocab, "hidden_size": self.width, "tied_to": "embed"}, "head"),
            streams=self.streams)
        spec.validate()
        return spec


register_architecture(ARCHITECTURE, KerudraConfig)
