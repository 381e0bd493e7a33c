"""Rikolix: a decoder whose ``config.json`` lists its layers one by one, each normed before and behind its sublayers.

A layer is  x += norm1b(mixer(norm1(x))); x += norm2b(ff(norm2(x)))  (block kind ``sandwich``; the second sublayer only where
``mlp`` is given).  Every such norm's tensor holds the weight's distance from one.  The typed configuration below reads every
key, checks it, and states the model as data for the generic decoder:

  * type "latent_attention" -> mixer kind ``latent_attention``: queries out of a normed latent of ``q_rank`` numbers, keys and
    values expanded per head from a normed latent of ``kv_rank`` numbers, one rotated key part of ``rot_dim`` for all heads
    (neighbouring pairs turn); with ``kv_from`` the layer reads the rows that an earlier layer cached and has no latent of its own;
  * type "attention" -> the general form of mixer kind ``attention``: grouped heads, q and k normed over their whole
    projections, rotation of neighbouring pairs over the first ``rot.dims`` dimensions, values turned by their positions over
    all their dimensions (the same base) and outputs turned back, weights sigmoid(score + bias[head]) without normalisation;
  * ``mlp.kind`` "dense" -> feed-forward kind ``mlp`` with the squared ReLU;
  * ``mlp.kind`` "moe" -> feed-forward kind ``moe``: ungated squared-ReLU experts, softmax scores, a correction per router
    output that joins the choice alone, a choice within the best groups of neighbours, ``router.identity`` outputs that return
    the input, weights not renormalised;
  * ``mlp`` null -> the layer has its mixer only.

Tensor names: ``embed``, ``l<i>.norm1|norm1b|norm2|norm2b``, ``l<i>.mix.*``, ``l<i>.mlp.*``, ``final.norm``, ``head``.
"""
from __future__ import annotations

import copy
from dataclasses import dataclass
from typing import Any, Dict, List, Optional, Tuple

from ..config.model_config import ConfigError, require
from ..config.registry import register_architecture
from ..config.specs import BlockSpec, FeedForwardSpec, LayerCall, MixerSpec, ModelSpec, NormSpec, PositionSpec

_LATENT_NAMES = (("q_down", "dq"), ("q_norm", "dq.norm"), ("q", "uq"), ("down", "dkv"), ("latent_norm", "dkv.norm"), ("up_k", "uk"),
                 ("up_v", "uv"), ("o", "o"))
_ATTENTION_NAMES = (("q", "q"), ("k", "k"), ("v", "v"), ("o", "o"), ("q_norm", "q.norm"), ("k_norm", "k.norm"), ("score_bias", "pb"))
_FF_NAMES = (("up", "up"), ("down", "down"))
_MOE_NAMES = (("router", "router"), ("up", "up"), ("down", "down"))


def _sub(raw: Dict[str, Any], key: str, where: str) -> Dict[str, Any]:
    value = raw.get(key)
    if not isinstance(value, dict):
        raise ConfigError(f"config.json: {where}'{key}' must be an object")
    return value


def _whole(raw: Dict[str, Any], key: str, where: str, least: int = 1) -> int:
    try:
        value = require(raw, key, int)
    except ConfigError as e:
        raise ConfigError(f"{e} (in {where})") from None
    if value < least:
        raise ConfigError(f"config.json: {where}'{key}' must be at least {least}, found {value}")
    return value


def _number(raw: Dict[str, Any], key: str, where: str) -> float:
    try:
        return require(raw, key, float)
    except ConfigError as e:
        raise ConfigError(f"{e} (in {where})") from None


def _check_rot(m: Dict[str, Any], within: int, where: str) -> None:
    rot = _sub(m, "rot", where)
    w = where + "rot."
    dims = _whole(rot, "dims", w)
    if dims % 2 or dims > within:
        raise ConfigError(f"config.json: {w}dims ({dims}) must be even and at most {within}")
    if not (_number(rot, "base", w) > 0.0):
        raise ConfigError(f"config.json: {w}base must be positive")


@dataclass(frozen=True)
class RikolixConfig:
    vocab: int
    width: int
    norm_eps: float
    embedding_scale: float
    layers: Tuple[Dict[str, Any], ...]          # as config.json lists them, checked
    architecture: str = "Rikolix"

    @classmethod
    def from_dict(cls, raw: Dict[str, Any]) -> "RikolixConfig":
        layers = raw.get("layers")
        if not isinstance(layers, list) or not layers:
            raise ConfigError("config.json: 'layers' must list at least one layer")
        embedding = raw.get("embedding")
        cfg = cls(vocab=_whole(raw, "vocab", ""), width=_whole(raw, "width", ""),
                  norm_eps=_number(_sub(raw, "norm", ""), "eps", "norm."),
                  embedding_scale=1.0 if embedding is None else _number(_sub(raw, "embedding", ""), "scale", "embedding."),
                  layers=tuple(copy.deepcopy(layers)))
        cfg.validate()
        return cfg

    def validate(self) -> None:
        if not (self.norm_eps > 0.0):
            raise ConfigError("config.json: norm.eps must be positive")
        for i, layer in enumerate(self.layers):
            where = f"layers[{i}]."
            if not isinstance(layer, dict):
                raise ConfigError(f"config.json: layers[{i}] must be an object")
            m, wm = _sub(layer, "mixer", where), where + "mixer."
            if layer.get("type") == "latent_attention":
                for key in ("heads", "dim", "rot_dim", "vdim", "q_rank", "kv_rank"):
                    _whole(m, key, wm)
                _check_rot(m, int(m["rot_dim"]), wm)
                self._check_borrowed(i, m, wm)
            elif layer.get("type") == "attention":
                for key in ("heads", "kv_heads", "dim", "vdim"):
                    _whole(m, key, wm)
                if m["heads"] % m["kv_heads"]:
                    raise ConfigError(f"config.json: {wm}heads ({m['heads']}) is not a multiple of kv_heads ({m['kv_heads']})")
                if m["vdim"] % 2:
                    raise ConfigError(f"config.json: {wm}vdim ({m['vdim']}) must be even: the values turn in pairs")
                _check_rot(m, int(m["dim"]), wm)
            else:
                raise ConfigError(f"config.json: {where}type '{layer.get('type')}' is not one of latent_attention, attention")
            _number(m, "scale", wm)
            if layer.get("mlp") is not None:
                self._check_mlp(layer["mlp"], where + "mlp.")

    def _check_borrowed(self, i: int, m: Dict[str, Any], wm: str) -> None:
        src = m.get("kv_from")
        if src is None:
            return
        if isinstance(src, bool) or not isinstance(src, int) or not (0 <= src < i):
            raise ConfigError(f"config.json: {wm}kv_from must name an earlier layer")
        other = self.layers[src]
        om = other.get("mixer", {})
        if other.get("type") != "latent_attention" or om.get("kv_from") is not None:
            raise ConfigError(f"config.json: {wm}kv_from = {src}: that layer has no latent of its own")
        if any(om.get(k) != m.get(k) for k in ("kv_rank", "rot_dim", "rot")):
            raise ConfigError(f"config.json: {wm}kv_from = {src}: kv_rank, rot_dim and rot must be equal")

    @staticmethod
    def _check_mlp(mlp: Any, wf: str) -> None:
        if not isinstance(mlp, dict) or mlp.get("kind") not in ("dense", "moe"):
            raise ConfigError(f"config.json: {wf}kind must be 'dense' or 'moe' (or mlp null)")
        if mlp["kind"] == "dense":
            _whole(mlp, "ff", wf)
            return
        _whole(_sub(mlp, "expert", wf), "ff", wf + "expert.")
        router, wr = _sub(mlp, "router", wf), wf + "router."
        outputs = _whole(router, "experts", wr) + (_whole(router, "identity", wr, 0) if router.get("identity") is not None else 0)
        top, offered = _whole(router, "top", wr), outputs
        if router.get("groups") is not None:
            groups, wg = _sub(router, "groups", wr), wr + "groups."
            count, keep = _whole(groups, "count", wg), _whole(groups, "keep", wg)
            if outputs % count or keep > count:
                raise ConfigError(f"config.json: {wg}count ({count}) must divide the router's {outputs} outputs, keep ({keep}) not exceed it")
            offered = keep * (outputs // count)
        if top > offered:
            raise ConfigError(f"config.json: {wr}top ({top}) exceeds the {offered} outputs it chooses from")

    def to_dict(self) -> Dict[str, Any]:
        return {"architecture": self.architecture, "vocab": self.vocab, "width": self.width, "norm": {"eps": self.norm_eps},
                "embedding": {"scale": self.embedding_scale}, "layers": copy.deepcopy(list(self.layers))}

    # ------------------------------------------------------------------ the model as data
    def _mixer_spec(self, layer: Dict[str, Any]) -> MixerSpec:
        m = layer["mixer"]
        base, dims = float(m["rot"]["base"]), int(m["rot"]["dims"])
        if layer["type"] == "latent_attention":
            return MixerSpec(kind="latent_attention", hidden=self.width, n_heads=int(m["heads"]), n_kv_heads=1,
                             head_dim=int(m["dim"]), v_head_dim=int(m["vdim"]), scale=float(m["scale"]),
                             position=PositionSpec("rope", int(m["rot_dim"]), dims, base), own_kv=m.get("kv_from") is None,
                             tensor_names=_LATENT_NAMES,
                             extra=(("q_rank", int(m["q_rank"])), ("kv_rank", int(m["kv_rank"])), ("rot_dim", int(m["rot_dim"])),
                                    ("latent_norm_eps", self.norm_eps)))
        dim, vdim = int(m["dim"]), int(m["vdim"])
        return MixerSpec(kind="attention", hidden=self.width, n_heads=int(m["heads"]), n_kv_heads=int(m["kv_heads"]), head_dim=dim,
                         v_head_dim=vdim, scale=float(m["scale"]), qk_norm_eps=self.norm_eps, qk_norm_whole=True,
                         position=PositionSpec("rope", dim, dims, base), rotate_neighbours=True,
                         value_position=PositionSpec("rope", vdim, vdim, base), sigmoid_weights=True, score_bias=True,
                         tensor_names=_ATTENTION_NAMES)

    def _feed_forward_spec(self, mlp: Optional[Dict[str, Any]]) -> Optional[FeedForwardSpec]:
        if mlp is None:
            return None
        if mlp["kind"] == "dense":
            return FeedForwardSpec("mlp", self.width, int(mlp["ff"]), "relu2", extra=(("tensor_names", _FF_NAMES),))
        router = mlp["router"]
        groups = router.get("groups")
        return FeedForwardSpec("moe", self.width, int(mlp["expert"]["ff"]), "relu2",
                               extra=(("gated", False), ("experts", int(router["experts"])), ("top", int(router["top"])),
                                      ("identity", int(router.get("identity") or 0)), ("correction", "correction"),
                                      ("groups", None if groups is None else (int(groups["count"]), int(groups["keep"]))),
                                      ("scoring", "softmax"), ("router_scale", 1.0), ("renormalize", False),
                                      ("tensor_names", _MOE_NAMES)))

    def model_spec(self) -> ModelSpec:
        norm = NormSpec("rmsnorm", self.width, self.norm_eps, suffix="", about_one=True)
        blocks: List[BlockSpec] = []
        order: List[LayerCall] = []
        entry_of: Dict[int, int] = {}
        for i, layer in enumerate(self.layers):
            ff = self._feed_forward_spec(layer.get("mlp"))
            blocks.append(BlockSpec(
                kind="sandwich", mixer=self._mixer_spec(layer), feed_forward=ff, mixer_norm=norm,
                feed_forward_norm=norm if ff is not None else None, weight_prefix=f"l{i}.",
                names=(("mixer", "mix."), ("feed_forward", "mlp."), ("mixer_norm", "norm1"), ("mixer_post_norm", "norm1b"),
                       ("feed_forward_norm", "norm2"), ("feed_forward_post_norm", "norm2b")),
                mixer_post_norm=norm, feed_forward_post_norm=norm if ff is not None else None))
            src = layer["mixer"].get("kv_from") if layer["type"] == "latent_attention" else None
            if src is None:
                entry_of[i] = len(entry_of)
                order.append(LayerCall(i, entry_of[i]))
            else:                                      # reads the rows that layer cached this step and before
                order.append(LayerCall(i, entry_of[src]))
        return ModelSpec(architecture=self.architecture, vocab_size=self.vocab, hidden=self.width, blocks=tuple(blocks),
                         run_order=tuple(order), final_norm=norm, embed_name="embed", final_norm_name="final.norm", head_name="head",
                         tie_word_embeddings=False, init_std=0.05, embedding_multiplier=self.embedding_scale)


@register_architecture("Rikolix")
def rikolix_config(raw: dict) -> RikolixConfig:
    return RikolixConfig.from_dict(raw)
