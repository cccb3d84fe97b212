"""Pununex as data: layers over one residual stream whose sublayers read the stream itself and whose outputs are normed (layer
norm), scaled element by element and added to it; token embedding plus a bigram embedding.

* ``parallel``: two mixers side by side on the same rows, their results weighted and added: windowed softmax attention without
  a rotation (q and k normed per head, scores capped, the sequence's first positions always visible, a learned sink) and a gated
  delta rule with one decay per head and key channel.
* ``delta``: a gated delta rule with one decay per head.
* feed-forward: dense with a relu gate, or experts chosen by a router with a correction that only the choice sees, groups of
  which some are kept, and outputs that stand for the identity; plus a shared expert.

Tensor names: ``embed``, ``bigram``, ``l<i>.norm1`` / ``norm2`` (``.b`` their offsets), ``l<i>.ls1`` / ``ls2``, ``l<i>.mix.*``
(``.left.*``, ``.right.*``), ``l<i>.mlp.*``, ``final.norm``, ``head``.
"""
from __future__ import annotations

from typing import Dict, Optional, Tuple

from ..config.pununex import PununexConfig
from ..parts.spec import LayerSpec, ModelSpec, PartSpec, ScheduleEntry
from .registry import register_architecture

ATTENTION_NAMES = {"q": "q", "k": "k", "v": "v", "o": "o", "q_norm": "q.norm", "k_norm": "k.norm", "sink": "sink"}
EXPERT_NAMES = {"router": "router", "correction": "correction", "gate": "e{e}.gate", "up": "e{e}.up", "down": "e{e}.down",
                "shared_gate": "shared.gate", "shared_up": "shared.up", "shared_down": "shared.down"}


def _attention(m: dict, h: int, eps: float) -> PartSpec:
    mask = m["mask"] or {}
    return PartSpec("sink_attention", {
        "hidden": h, "heads": m["heads"], "kv_heads": m["kv_heads"], "head_dim": m["dim"], "v_head_dim": m["vdim"], "scale": m["scale"],
        "qk_norm": "head", "norm_eps": eps, "position": PartSpec("none", {}), "window": mask.get("size"), "keep_first": mask.get("keep_first", 0),
        "softcap": m["softcap"], "sink": "learned", "names": ATTENTION_NAMES})


def _delta(m: dict, h: int, eps: float) -> PartSpec:
    params = {"hidden": h, "heads": m["heads"], "kv_heads": m["kv_heads"], "dim": m["dim"], "vdim": m["vdim"], "taps": m["conv"], "norm_eps": eps}
    if "decay_rank" in m:
        params.update(decay="channel", decay_rank=m["decay_rank"], gate="sigmoid", gate_rank=m["gate_rank"])
    else:
        params.update(decay="head", gate="silu")
    return PartSpec("delta_rule", params)


def _mixer(kind: str, m: dict, h: int, eps: float) -> PartSpec:
    if kind == "delta":
        return _delta(m, h, eps)
    return PartSpec("parallel_mixers", {"hidden": h, "inner": {"left": _attention(m["left"], h, eps), "right": _delta(m["right"], h, eps)},
                                        "scales": {"left": m["left_scale"], "right": m["right_scale"]}})


def _feedforward(mlp: Optional[dict], h: int) -> Optional[PartSpec]:
    if mlp is None:
        return None
    if mlp["kind"] == "dense":
        return PartSpec("swiglu", {"hidden": h, "intermediate": mlp["ff"], "activation": "relu", "names": ("gate", "up", "down")})
    router, shared = mlp["router"], mlp["shared"]
    groups = router["groups"] or {"count": 1, "keep": 1}
    return PartSpec("routed_experts", {
        "hidden": h, "intermediate": mlp["expert"]["ff"], "experts": router["experts"], "top": router["top"], "score": "softmax",
        "renormalize": True, "weight_on": "output", "correction": True, "groups": groups["count"], "keep_groups": groups["keep"],
        "identity": router["identity"], "weight_scale": router["scale"],
        "shared_intermediate": shared["ff"] if shared is not None else None, "names": EXPERT_NAMES})


def resolve_shapes(cfg: PununexConfig, shapes: Dict[str, Tuple[int, ...]]) -> PununexConfig:
    """Sizes that only the checkpoint gives are taken from the shapes of its tensors, by name, before the model is built."""
    return cfg.with_tensor_shapes(shapes)


def build_spec(cfg: PununexConfig) -> ModelSpec:
    h = cfg.hidden_size
    norm = PartSpec("layernorm", {"dim": h, "eps": cfg.norm_eps, "names": ("", "b")})
    layers = [LayerSpec(block="postnorm", norm=norm, mixer=_mixer(layer.type, layer.mixer, h, cfg.norm_eps), feedforward=_feedforward(layer.mlp, h),
                        prefix=f"l{i}", names={"norm1": "norm1", "mixer": "mix", "norm2": "norm2", "feedforward": "mlp"},
                        block_params={"layer_scale": ("ls1", "ls2")})
              for i, layer in enumerate(cfg.layers)]
    embedding = {"vocab": cfg.vocab_size, "hidden": h, "name": "embed", "tensor": "embed"}
    if cfg.bigram is not None:
        embedding.update(bigram=dict(cfg.bigram), bigram_tensor="bigram")
    return ModelSpec(
        hidden_size=h,
        vocab_size=cfg.vocab_size,
        embedding=PartSpec("token_table", embedding),
        final_norm=PartSpec("layernorm", {"dim": h, "eps": cfg.norm_eps, "name": "final.norm", "names": ("", "b")}),
        head=PartSpec("linear", {"vocab": cfg.vocab_size, "hidden": h, "name": "head", "tied": False, "tensor": "head"}),
        layers=layers,
        schedule=[ScheduleEntry(i) for i in range(len(cfg.layers))],
    )


register_architecture(PununexConfig.ARCHITECTURE, PununexConfig.MODEL_TYPE, PununexConfig, build_spec, resolve_shapes)
