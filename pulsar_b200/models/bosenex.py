"""Bosenex: a pre-norm decoder whose ``config.json`` lists its layers one by one.

A layer is  x += mixer(norm1(x)); x += ff(norm2(x))  (block kind ``prenorm``; the second sublayer only where ``mlp`` is given).
The typed configuration below reads every key, checks it, and states the model as data for the generic decoder:

  * type "mlstm" -> mixer kind ``matrix_memory``: a matrix, a normaliser and a running maximum per head with exponential gates;
    queries multiplied by dim^-1/2, a sigmoid gate on every element of the normed heads;
  * type "parallel" -> mixer kind ``side_by_side`` with two members whose outputs are normed over the width with a weight each and
    join as half their sum: ``left`` is the general form of kind ``attention`` (grouped heads, rotate-half layout on a head's
    first ``rot.dims`` dimensions, capped scores, a sliding window, a learned sink per head in the softmax's denominator, one
    sigmoid gate per head), ``right`` is kind ``state_space_dual`` (one decay per head, a short convolution, a gate in front of a
    norm over equal parts);
  * ``mlp.kind`` "dense" -> feed-forward kind ``swiglu`` with activation relu; "moe" -> kind ``moe``: the ``router.top`` largest of
    biased logits, weights the softmax over those alone, clamped gated experts with the design's sigmoid slope, plus an optional
    shared expert of the same form (``clamped_glu``) that is added;
  * ``mlp`` null -> the layer has its mixer only.

Tensor names: ``embed``, ``l<i>.norm1|norm2``, ``l<i>.mix.*`` (``l<i>.mix.left.*`` / ``l<i>.mix.right.*`` for a parallel layer),
``l<i>.mlp.*``, ``final.norm``, ``head``.
"""
from __future__ import annotations

import copy
from dataclasses import dataclass
from typing import Any, Dict, List, Optional, Tuple

from ..config.model_config import ConfigError, require
from ..config.registry import register_architecture
from ..config.specs import BlockSpec, FeedForwardSpec, LayerCall, MixerSpec, ModelSpec, NormSpec, PositionSpec

GATE_SLOPE = 1.702              # an expert's g * sigmoid(1.702 g)
UP_SHIFT = 1.0                  # ... times (u + 1)
MEMORY_DENOM_EPS = 1e-6         # added to the matrix memory's denominator
MEMBER_SCALE = 0.5              # a parallel layer's two outputs join as half their sum

_MEMORY_NAMES = (("q", "q"), ("k", "k"), ("v", "v"), ("g", "g"), ("i", "i"), ("f", "f"), ("i_bias", "i.b"), ("f_bias", "f.b"),
                 ("norm", "norm"), ("o", "o"))
_LEFT_NAMES = (("q", "q"), ("k", "k"), ("v", "v"), ("o", "o"), ("gate", "g"), ("sinks", "sink"))
_RIGHT_NAMES = (("in", "in"), ("conv", "conv"), ("conv_bias", "conv.b"), ("dt_bias", "dt_bias"), ("a_log", "A_log"), ("d", "D"),
                ("norm", "norm"), ("o", "o"))
_FF_NAMES = (("gate", "gate"), ("up", "up"), ("down", "down"))
_MOE_NAMES = (("router", "router"),) + _FF_NAMES


def _sub(raw: Dict[str, Any], key: str, where: str) -> Dict[str, Any]:
    value = raw.get(key)
    if not isinstance(value, dict):
        raise ConfigError(f"config.json: {where}'{key}' must be an object")
    return value


def _positive(raw: Dict[str, Any], key: str, where: str) -> int:
    try:
        value = require(raw, key, int)
    except ConfigError as e:
        raise ConfigError(f"{e} (in {where})") from None
    if value <= 0:
        raise ConfigError(f"config.json: {where}'{key}' must be positive, found {value}")
    return value


def _number(raw: Dict[str, Any], key: str, where: str, positive: bool = False) -> float:
    try:
        value = require(raw, key, float)
    except ConfigError as e:
        raise ConfigError(f"{e} (in {where})") from None
    if positive and not (value > 0.0):
        raise ConfigError(f"config.json: {where}'{key}' must be positive, found {value}")
    return value


@dataclass(frozen=True)
class BosenexConfig:
    vocab: int
    width: int
    norm_eps: float
    embedding_scale: float
    logit_scale: float
    layers: Tuple[Dict[str, Any], ...]          # as config.json lists them, checked
    architecture: str = "Bosenex"

    @classmethod
    def from_dict(cls, raw: Dict[str, Any]) -> "BosenexConfig":
        layers = raw.get("layers")
        if not isinstance(layers, list) or not layers:
            raise ConfigError("config.json: 'layers' must list at least one layer")
        scale = 1.0
        if raw.get("embedding") is not None:
            scale = _number(_sub(raw, "embedding", ""), "scale", "embedding.")
        cfg = cls(vocab=_positive(raw, "vocab", ""), width=_positive(raw, "width", ""),
                  norm_eps=_number(_sub(raw, "norm", ""), "eps", "norm.", positive=True), embedding_scale=scale,
                  logit_scale=_number(raw, "logit_scale", "") if raw.get("logit_scale") is not None else 1.0,
                  layers=tuple(copy.deepcopy(layers)))
        for i, layer in enumerate(cfg.layers):
            if not isinstance(layer, dict):
                raise ConfigError(f"config.json: layers[{i}] must be an object")
            cfg._check_mixer(layer, f"layers[{i}].")
            cfg._check_feed_forward(layer.get("mlp"), f"layers[{i}].mlp.")
        return cfg

    @staticmethod
    def _check_mixer(layer: Dict[str, Any], where: str) -> None:
        kind = layer.get("type")
        m = _sub(layer, "mixer", where)
        wm = where + "mixer."
        if kind == "mlstm":
            for key in ("heads", "dim", "vdim"):
                _positive(m, key, wm)
            _number(m, "gate_cap", wm, positive=True)
            return
        if kind != "parallel":
            raise ConfigError(f"config.json: {where}type '{kind}' is not one of mlstm, parallel")
        left, right = _sub(m, "left", wm), _sub(m, "right", wm)
        wl, wr = wm + "left.", wm + "right."
        for key in ("heads", "kv_heads", "dim", "vdim"):
            _positive(left, key, wl)
        if left["heads"] % left["kv_heads"]:
            raise ConfigError(f"config.json: {wl}heads ({left['heads']}) is not a multiple of kv_heads ({left['kv_heads']})")
        _number(left, "scale", wl, positive=True)
        if left.get("softcap") is not None:
            _number(left, "softcap", wl, positive=True)
        if left.get("mask") is not None:
            _positive(_sub(left, "mask", wl), "size", wl + "mask.")
        if left.get("rot") is not None:
            rot = _sub(left, "rot", wl)
            dims = _positive(rot, "dims", wl + "rot.")
            if dims % 2 or dims > left["dim"]:
                raise ConfigError(f"config.json: {wl}rot.dims ({dims}) must be even and at most {left['dim']}")
            _number(rot, "base", wl + "rot.", positive=True)
        for key in ("heads", "vdim", "state", "groups", "conv", "norm_groups"):
            _positive(right, key, wr)
        if right["heads"] % right["groups"]:
            raise ConfigError(f"config.json: {wr}heads ({right['heads']}) is not a multiple of groups ({right['groups']})")
        if right["heads"] * right["vdim"] % right["norm_groups"]:
            raise ConfigError(f"config.json: {wr}norm_groups ({right['norm_groups']}) does not divide heads * vdim "
                              f"({right['heads'] * right['vdim']})")

    @staticmethod
    def _check_feed_forward(mlp: Optional[Dict[str, Any]], where: str) -> None:
        if mlp is None:
            return
        kind = mlp.get("kind") if isinstance(mlp, dict) else None
        if kind == "dense":
            _positive(mlp, "ff", where)
            return
        if kind != "moe":
            raise ConfigError(f"config.json: {where}kind must be 'dense' or 'moe' (or mlp null)")
        router = _sub(mlp, "router", where)
        experts, top = _positive(router, "experts", where + "router."), _positive(router, "top", where + "router.")
        if top > experts:
            raise ConfigError(f"config.json: {where}router.top ({top}) exceeds router.experts ({experts})")
        for key in ("expert",) + (("shared",) if mlp.get("shared") is not None else ()):
            unit = _sub(mlp, key, where)
            _positive(unit, "ff", f"{where}{key}.")
            _number(unit, "limit", f"{where}{key}.", positive=True)

    def to_dict(self) -> Dict[str, Any]:
        return {"architecture": self.architecture, "vocab": self.vocab, "width": self.width, "norm": {"eps": self.norm_eps},
                "embedding": {"scale": self.embedding_scale}, "logit_scale": self.logit_scale, "layers": copy.deepcopy(list(self.layers))}

    # ------------------------------------------------------------------ the model as data
    def _mixer_spec(self, layer: Dict[str, Any]) -> MixerSpec:
        m = layer["mixer"]
        if layer["type"] == "mlstm":
            return MixerSpec(kind="matrix_memory", hidden=self.width, n_heads=int(m["heads"]), head_dim=int(m["dim"]),
                             v_head_dim=int(m["vdim"]), norm_eps=self.norm_eps, tensor_names=_MEMORY_NAMES,
                             extra=(("gate_cap", float(m["gate_cap"])), ("q_scale", int(m["dim"]) ** -0.5),
                                    ("denom_eps", MEMORY_DENOM_EPS)))
        left, right = m["left"], m["right"]
        mask, rot = left.get("mask"), left.get("rot")
        position = None
        if rot is not None:
            position = PositionSpec(kind="rope", head_dim=int(left["dim"]), rotary_dim=int(rot["dims"]), theta=float(rot["base"]))
        left_spec = MixerSpec(kind="attention", hidden=self.width, n_heads=int(left["heads"]), n_kv_heads=int(left["kv_heads"]),
                              head_dim=int(left["dim"]), v_head_dim=int(left["vdim"]), scale=float(left["scale"]),
                              window=None if mask is None else int(mask["size"]), position=position,
                              softcap=None if left.get("softcap") is None else float(left["softcap"]), sinks=True, gate_per_head=True,
                              tensor_names=_LEFT_NAMES)
        right_spec = MixerSpec(kind="state_space_dual", hidden=self.width, n_heads=int(right["heads"]), v_head_dim=int(right["vdim"]),
                               norm_eps=self.norm_eps, tensor_names=_RIGHT_NAMES,
                               extra=tuple((key, int(right[key])) for key in ("state", "groups", "conv", "norm_groups")))
        return MixerSpec(kind="side_by_side", hidden=self.width, norm_eps=self.norm_eps,
                         extra=(("members", (("left.", left_spec, MEMBER_SCALE), ("right.", right_spec, MEMBER_SCALE))),
                                ("norm_names", ("left.out", "right.out"))))

    def _feed_forward_spec(self, mlp: Optional[Dict[str, Any]]) -> Optional[FeedForwardSpec]:
        if mlp is None:
            return None
        if mlp["kind"] == "dense":
            return FeedForwardSpec("swiglu", self.width, int(mlp["ff"]), "relu", extra=(("tensor_names", _FF_NAMES),))
        expert, router, shared = mlp["expert"], mlp["router"], mlp.get("shared")
        shared_spec = None
        if shared is not None:
            shared_spec = FeedForwardSpec("clamped_glu", self.width, int(shared["ff"]), extra=(
                ("limit", float(shared["limit"])), ("alpha", GATE_SLOPE), ("tensor_names", _FF_NAMES)))
        return FeedForwardSpec("moe", self.width, int(expert["ff"]),
                               extra=(("limit", float(expert["limit"])), ("alpha", GATE_SLOPE), ("shift", UP_SHIFT),
                                      ("experts", int(router["experts"])), ("top", int(router["top"])), ("router_scale", 1.0),
                                      ("scoring", "softmax"), ("renormalize", True), ("renorm_eps", 0.0),
                                      ("router_bias", "router.b"), ("shared", shared_spec), ("shared_prefix", "shared."),
                                      ("tensor_names", _MOE_NAMES)))

    def model_spec(self) -> ModelSpec:
        norm = NormSpec("rmsnorm", self.width, self.norm_eps, suffix="")
        blocks: List[BlockSpec] = []
        order: List[LayerCall] = []
        entry = 0
        for i, layer in enumerate(self.layers):
            ff = self._feed_forward_spec(layer.get("mlp"))
            blocks.append(BlockSpec(kind="prenorm", mixer=self._mixer_spec(layer), feed_forward=ff, mixer_norm=norm,
                                    feed_forward_norm=norm if ff is not None else None, weight_prefix=f"l{i}.",
                                    names=(("mixer", "mix."), ("feed_forward", "mlp."), ("mixer_norm", "norm1"),
                                           ("feed_forward_norm", "norm2"))))
            members = (entry + 1,) if layer["type"] == "parallel" else ()
            order.append(LayerCall(i, entry, members=members))
            entry += 1 + len(members)
        return ModelSpec(architecture=self.architecture, vocab_size=self.vocab, hidden=self.width, blocks=tuple(blocks),
                         run_order=tuple(order), final_norm=norm, embed_name="embed", final_norm_name="final.norm", head_name="head",
                         tie_word_embeddings=False, init_std=0.05, embedding_multiplier=self.embedding_scale,
                         logit_scale=self.logit_scale)


@register_architecture("Bosenex")
def bosenex_config(raw: dict) -> BosenexConfig:
    return BosenexConfig.from_dict(raw)
