"""Configuration of the Pununex decoder: a list of layers, each with one of two mixers (``parallel``: windowed softmax
attention beside a gated delta rule, both reading the same rows; ``delta``: a gated delta rule alone) and a dense or routed
feed-forward; the norm's eps and, where the model has one, the hash of the bigram embedding.

Every size and constant comes from ``config.json``; what a part needs is checked here, so that a folder with a missing or
mistyped key is refused before any weight is read.  Optional keys switch a mechanism off when they are absent: no
``embedding.bigram``, no ``mask`` (every earlier position is seen), no ``mask.keep_first``, no ``softcap``, no
``router.groups``, no ``router.identity``, no ``mlp.shared``, ``mlp`` null.  The ranks of the delta rule's two small products
(``decay_rank``, ``gate_rank``) are taken from a checkpoint's tensors where there is one.
"""
from __future__ import annotations

import copy
from dataclasses import dataclass, field
from typing import Any, Dict, List, Optional, Tuple

from .base import ConfigError, ModelConfig, eos_ids, optional
from .fegarax import DEFAULT_MAX_POSITIONS, _int, _num, _obj

MIXER_TYPES = ("parallel", "delta")
MLP_KINDS = ("dense", "moe")
#: inner width of a small product of two matrices where neither config.json nor a checkpoint says
DEFAULT_RANK = 64


def _heads(m: Dict[str, Any], where: str, keys) -> Dict[str, Any]:
    out = {k: _int(m, k, where) for k in ("heads", "kv_heads", "dim", "vdim") + tuple(keys)}
    if out["heads"] % out["kv_heads"] != 0:
        raise ConfigError(f"config.json: {where}{out['heads']} heads cannot share {out['kv_heads']} kv heads evenly")
    return out


def _attention(m: Dict[str, Any], where: str) -> Dict[str, Any]:
    out = _heads(m, where, ())
    out["scale"] = _num(m, "scale", where)
    out["softcap"] = _num(m, "softcap", where, True) if m.get("softcap") is not None else None
    mask = _obj(m, "mask", where, needed=False)
    out["mask"] = None
    if mask is not None:
        out["mask"] = {"size": _int(mask, "size", where + "mask: "),
                       "keep_first": _int(mask, "keep_first", where + "mask: ", 0) if mask.get("keep_first") is not None else 0}
    return out


def _delta(m: Dict[str, Any], where: str, low_rank: bool) -> Dict[str, Any]:
    out = _heads(m, where, ("conv",))
    if low_rank:
        for key in ("decay_rank", "gate_rank"):
            out[key] = _int(m, key, where) if m.get(key) is not None else DEFAULT_RANK
    return out


def _mixer(kind: str, m: Dict[str, Any], where: str) -> Dict[str, Any]:
    if kind == "delta":
        return _delta(m, where, False)
    return {"left": _attention(_obj(m, "left", where), where + "left: "), "right": _delta(_obj(m, "right", where), where + "right: ", True),
            "left_scale": _num(m, "left_scale", where), "right_scale": _num(m, "right_scale", where)}


def _router(raw: Dict[str, Any], where: str) -> Dict[str, Any]:
    out: Dict[str, Any] = {"experts": _int(raw, "experts", where), "top": _int(raw, "top", where),
                           "identity": _int(raw, "identity", where, 0) if raw.get("identity") is not None else 0,
                           "scale": _num(raw, "scale", where) if raw.get("scale") is not None else 1.0}
    outputs = out["experts"] + out["identity"]
    groups = _obj(raw, "groups", where, needed=False)
    out["groups"] = None
    choice = outputs
    if groups is not None:
        g = {k: _int(groups, k, where + "groups: ") for k in ("count", "keep")}
        if outputs % g["count"] != 0 or g["keep"] > g["count"]:
            raise ConfigError(f"config.json: {where}{outputs} router outputs do not form {g['count']} equal groups of which {g['keep']} are kept")
        out["groups"] = g
        choice = outputs // g["count"] * g["keep"]
    if out["top"] > choice:
        raise ConfigError(f"config.json: {where}`top` {out['top']} exceeds the {choice} router outputs that can be chosen")
    return out


def _mlp(mlp: Any, where: str) -> Optional[Dict[str, Any]]:
    if mlp is None:
        return None
    if not isinstance(mlp, dict):
        raise ConfigError(f"config.json: {where}`mlp` must be an object or null")
    kind = mlp.get("kind")
    if kind not in MLP_KINDS:
        raise ConfigError(f"config.json: {where}`mlp.kind` {kind!r} is not one of {list(MLP_KINDS)}")
    if kind == "dense":
        return {"kind": "dense", "ff": _int(mlp, "ff", where + "mlp: ")}
    shared = _obj(mlp, "shared", where + "mlp: ", needed=False)
    return {"kind": "moe", "expert": {"ff": _int(_obj(mlp, "expert", where + "mlp: "), "ff", where + "mlp.expert: ")},
            "router": _router(_obj(mlp, "router", where + "mlp: "), where + "mlp.router: "),
            "shared": {"ff": _int(shared, "ff", where + "mlp.shared: ")} if shared is not None else None}


def _without_none(value: Any) -> Any:
    return {k: _without_none(v) for k, v in value.items() if v is not None} if isinstance(value, dict) else value


@dataclass
class PununexLayer:
    type: str
    mixer: Dict[str, Any]
    mlp: Optional[Dict[str, Any]]

    @classmethod
    def parse(cls, raw: Any, index: int) -> "PununexLayer":
        where = f"layers[{index}]: "
        if not isinstance(raw, dict):
            raise ConfigError(f"config.json: {where}must be an object")
        kind = raw.get("type")
        if kind not in MIXER_TYPES:
            raise ConfigError(f"config.json: {where}`type` {kind!r} is not one of {list(MIXER_TYPES)}")
        return cls(kind, _mixer(kind, _obj(raw, "mixer", where), where), _mlp(raw.get("mlp"), where))

    def to_json_dict(self) -> Dict[str, Any]:
        return {"type": self.type, "mixer": _without_none(self.mixer), "mlp": _without_none(self.mlp)}


@dataclass
class PununexConfig(ModelConfig):
    layers: List[PununexLayer] = field(default_factory=list)
    norm_eps: float = 0.0
    #: {"buckets", "mul_prev", "mul_cur"} or None
    bigram: Optional[Dict[str, int]] = None

    ARCHITECTURE = "Pununex"
    MODEL_TYPE = "pununex"

    @classmethod
    def from_dict(cls, raw: Dict[str, Any], generation: Optional[Dict[str, Any]] = None) -> "PununexConfig":
        layers_raw = raw.get("layers")
        if not isinstance(layers_raw, list) or not layers_raw:
            raise ConfigError("config.json: `layers` must be a non-empty list")
        layers = [PununexLayer.parse(layer, i) for i, layer in enumerate(layers_raw)]
        norm = _obj(raw, "norm", "")
        emb = _obj(raw, "embedding", "", needed=False)
        bigram = _obj(emb, "bigram", "embedding: ", needed=False) if emb is not None else None
        if bigram is not None:
            where = "embedding.bigram: "
            bigram = {"buckets": _int(bigram, "buckets", where), "mul_prev": _int(bigram, "mul_prev", where, 0),
                      "mul_cur": _int(bigram, "mul_cur", where, 0)}
        eos = eos_ids(raw.get("eos_token_id"))
        if generation is not None and generation.get("eos_token_id") is not None:
            eos = eos_ids(generation.get("eos_token_id"))
        return cls(architecture=cls.ARCHITECTURE, model_type=cls.MODEL_TYPE, vocab_size=_int(raw, "vocab", ""),
                   hidden_size=_int(raw, "width", ""), max_position_embeddings=optional(raw, "max_positions", int, DEFAULT_MAX_POSITIONS),
                   eos_token_ids=eos, raw=dict(raw), layers=layers, norm_eps=_num(norm, "eps", "norm: "), bigram=bigram)

    def with_tensor_shapes(self, shapes: Dict[str, Tuple[int, ...]]) -> "PununexConfig":
        """The ranks of the small products as the checkpoint's tensors have them."""
        cfg = copy.deepcopy(self)
        for i, layer in enumerate(cfg.layers):
            if layer.type != "parallel":
                continue
            for key, name in (("decay_rank", "a1"), ("gate_rank", "g1")):
                shape = shapes.get(f"l{i}.mix.right.{name}")
                if shape is not None and len(shape) == 2:
                    layer.mixer["right"][key] = int(shape[0])
        return cfg

    def to_json_dict(self) -> Dict[str, Any]:
        out: Dict[str, Any] = {"architecture": self.ARCHITECTURE, "vocab": self.vocab_size, "width": self.hidden_size, "norm": {"eps": self.norm_eps},
                               "layers": [layer.to_json_dict() for layer in self.layers]}
        if self.bigram is not None:
            out["embedding"] = {"bigram": dict(self.bigram)}
        if self.max_position_embeddings != DEFAULT_MAX_POSITIONS:
            out["max_positions"] = self.max_position_embeddings
        if self.eos_token_ids:
            out["eos_token_id"] = list(self.eos_token_ids)
        return out
