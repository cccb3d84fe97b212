"""Configuration of the Punolix decoder: a list of layers, each with one of two mixers (``attention``: differential attention;
``parallel``: attention inside chunks behind short convolutions beside gated linear attention, both reading the same rows) and a dense
feed-forward; a loop over a run of layers; the embedding's scale, what multiplies a layer's result and the norm's eps.

Every size and constant comes from ``config.json``; what a part needs is checked here, so that a folder with a missing or
mistyped key is refused before any weight is read.  Optional keys switch a mechanism off when they are absent: no ``loop`` (every
layer runs once), no ``softcap``, no ``mask`` (every earlier position is seen), no ``conv``, no ``rot.scaling`` (plain frequencies), ``mlp`` null, an
``embedding.scale`` and a ``residual_mult`` of 1.  The numbers between the two matrices of the decays (``decay_rank``) are taken from a checkpoint's
tensors where there is one.
"""
from __future__ import annotations

import copy
from dataclasses import dataclass, field
from typing import Any, Dict, List, Optional, Tuple

from .base import ConfigError, ModelConfig, eos_ids, optional
from .fegarax import DEFAULT_MAX_POSITIONS, _int, _num, _obj

MIXER_TYPES = ("attention", "parallel")
MLP_KINDS = ("dense",)
#: numbers between the decays' two matrices where neither config.json nor a checkpoint says
DEFAULT_DECAY_RANK = 16


def _rot(m: Dict[str, Any], where: str, dim: int) -> Dict[str, Any]:
    rot = _obj(m, "rot", where)
    where += "rot: "
    out: Dict[str, Any] = {"dims": _int(rot, "dims", where), "base": _num(rot, "base", where, True), "scaling": None}
    if out["dims"] % 2 != 0 or out["dims"] > dim:
        raise ConfigError(f"config.json: {where}`dims` {out['dims']} must be even and at most the head size {dim}")
    scaling = _obj(rot, "scaling", where, needed=False)
    if scaling is not None:
        where += "scaling: "
        out["scaling"] = {k: _num(scaling, k, where, True) for k in ("factor", "low", "high", "original")}
        if out["scaling"]["high"] <= out["scaling"]["low"]:
            raise ConfigError(f"config.json: {where}`high` must be above `low`")
    return out


def _heads(m: Dict[str, Any], where: str) -> Dict[str, Any]:
    out: Dict[str, Any] = {k: _int(m, k, where) for k in ("heads", "kv_heads", "dim", "vdim")}
    if out["heads"] % out["kv_heads"] != 0:
        raise ConfigError(f"config.json: {where}{out['heads']} heads cannot share {out['kv_heads']} kv heads evenly")
    out["scale"] = _num(m, "scale", where)
    out["rot"] = _rot(m, where, out["dim"])
    return out


def _differential(m: Dict[str, Any], where: str) -> Dict[str, Any]:
    out = _heads(m, where)
    out["softcap"] = _num(m, "softcap", where, True) if m.get("softcap") is not None else None
    out["diff"] = _num(m, "diff", where)
    return out


def _chunked(m: Dict[str, Any], where: str) -> Dict[str, Any]:
    out = _heads(m, where)
    out["conv"] = _int(m, "conv", where) if m.get("conv") is not None else None
    mask = _obj(m, "mask", where, needed=False)
    out["mask"] = {"size": _int(mask, "size", where + "mask: ")} if mask is not None else None
    return out


def _linear(m: Dict[str, Any], where: str) -> Dict[str, Any]:
    out: Dict[str, Any] = {k: _int(m, k, where) for k in ("heads", "dim", "vdim")}
    out["tau"] = _num(m, "tau", where, True)
    out["decay_rank"] = _int(m, "decay_rank", where) if m.get("decay_rank") is not None else DEFAULT_DECAY_RANK
    return out


def _mixer(kind: str, m: Dict[str, Any], where: str) -> Dict[str, Any]:
    if kind == "attention":
        return _differential(m, where)
    return {"left": _chunked(_obj(m, "left", where), where + "left: "), "right": _linear(_obj(m, "right", where), where + "right: "),
            "left_scale": _num(m, "left_scale", where), "right_scale": _num(m, "right_scale", where)}


def _mlp(mlp: Any, where: str) -> Optional[Dict[str, Any]]:
    if mlp is None:
        return None
    if not isinstance(mlp, dict):
        raise ConfigError(f"config.json: {where}`mlp` must be an object or null")
    if mlp.get("kind") not in MLP_KINDS:
        raise ConfigError(f"config.json: {where}`mlp.kind` {mlp.get('kind')!r} is not one of {list(MLP_KINDS)}")
    return {"kind": "dense", "ff": _int(mlp, "ff", where + "mlp: ")}


def _without_none(value: Any) -> Any:
    return {k: _without_none(v) for k, v in value.items() if v is not None} if isinstance(value, dict) else value


@dataclass
class PunolixLayer:
    type: str
    mixer: Dict[str, Any]
    mlp: Optional[Dict[str, Any]]

    @classmethod
    def parse(cls, raw: Any, index: int) -> "PunolixLayer":
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
class PunolixConfig(ModelConfig):
    layers: List[PunolixLayer] = field(default_factory=list)
    norm_eps: float = 0.0
    embedding_scale: float = 1.0
    residual_mult: float = 1.0
    #: {"start", "stop", "times"} or None
    loop: Optional[Dict[str, int]] = None

    ARCHITECTURE = "Punolix"
    MODEL_TYPE = "punolix"

    @classmethod
    def from_dict(cls, raw: Dict[str, Any], generation: Optional[Dict[str, Any]] = None) -> "PunolixConfig":
        layers_raw = raw.get("layers")
        if not isinstance(layers_raw, list) or not layers_raw:
            raise ConfigError("config.json: `layers` must be a non-empty list")
        layers = [PunolixLayer.parse(layer, i) for i, layer in enumerate(layers_raw)]
        norm = _obj(raw, "norm", "")
        emb = _obj(raw, "embedding", "", needed=False) or {}
        loop = _obj(raw, "loop", "", needed=False)
        if loop is not None:
            loop = {"start": _int(loop, "start", "loop: ", 0), "stop": _int(loop, "stop", "loop: "), "times": _int(loop, "times", "loop: ")}
            if not loop["start"] < loop["stop"] <= len(layers):
                raise ConfigError(f"config.json: loop: layers {loop['start']} .. {loop['stop'] - 1} of {len(layers)} cannot be run in a loop")
        eos = eos_ids(raw.get("eos_token_id"))
        if generation is not None and generation.get("eos_token_id") is not None:
            eos = eos_ids(generation.get("eos_token_id"))
        return cls(architecture=cls.ARCHITECTURE, model_type=cls.MODEL_TYPE, vocab_size=_int(raw, "vocab", ""),
                   hidden_size=_int(raw, "width", ""), max_position_embeddings=optional(raw, "max_positions", int, DEFAULT_MAX_POSITIONS),
                   eos_token_ids=eos, raw=dict(raw), layers=layers, norm_eps=_num(norm, "eps", "norm: "),
                   embedding_scale=_num(emb, "scale", "embedding: ") if emb.get("scale") is not None else 1.0,
                   residual_mult=_num(raw, "residual_mult", "") if raw.get("residual_mult") is not None else 1.0, loop=loop)

    @property
    def layer_runs(self) -> List[Tuple[int, Optional[int]]]:
        """The layers in the order they run, each with the pass of the loop that starts right before it (None: none does)."""
        n = len(self.layers)
        if self.loop is None:
            return [(i, None) for i in range(n)]
        start, stop, times = (self.loop[k] for k in ("start", "stop", "times"))
        runs: List[Tuple[int, Optional[int]]] = [(i, None) for i in range(start)]
        for p in range(times):
            runs += [(i, p if i == start else None) for i in range(start, stop)]
        return runs + [(i, None) for i in range(stop, n)]

    def with_tensor_shapes(self, shapes: Dict[str, Tuple[int, ...]]) -> "PunolixConfig":
        """The numbers between the decays' two matrices as the checkpoint's tensors have them."""
        cfg = copy.deepcopy(self)
        for i, layer in enumerate(cfg.layers):
            shape = shapes.get(f"l{i}.mix.right.a1") if layer.type == "parallel" else None
            if shape is not None and len(shape) == 2:
                layer.mixer["right"]["decay_rank"] = int(shape[0])
        return cfg

    def to_json_dict(self) -> Dict[str, Any]:
        out: Dict[str, Any] = {"architecture": self.ARCHITECTURE, "vocab": self.vocab_size, "width": self.hidden_size, "norm": {"eps": self.norm_eps},
                               "embedding": {"scale": self.embedding_scale}, "residual_mult": self.residual_mult,
                               "layers": [layer.to_json_dict() for layer in self.layers]}
        if self.loop is not None:
            out["loop"] = dict(self.loop)
        if self.max_position_embeddings != DEFAULT_MAX_POSITIONS:
            out["max_positions"] = self.max_position_embeddings
        if self.eos_token_ids:
            out["eos_token_id"] = list(self.eos_token_ids)
        return out
