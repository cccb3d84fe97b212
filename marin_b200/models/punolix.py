"""Punolix as data: layers over one residual stream whose two sublayers read one norm side by side, their sum times a constant added to the
stream; a run of layers several times in a row with the same weights, a learned vector added where each pass starts and the embedding's
output again where each but the first does.

* ``attention``: differential attention (two softmax maps per head over the same values, the second weighted and subtracted), neighbouring
  pairs rotated, scores capped.
* ``parallel``: two mixers side by side, their results weighted and added: softmax attention inside chunks of the sequence (biased projections
  through short convolutions, q and k normed per head, half-split pairs rotated by band-scaled frequencies) and gated linear attention with one
  decay per head and key channel.
* feed-forward: dense with a gelu gate.

Tensor names: ``embed``, ``loop.step``, ``l<i>.norm1``, ``l<i>.mix.*`` (``.left.*``, ``.right.*``), ``l<i>.mlp.*``, ``final.norm``, ``head``.  Every run of a
looped layer is a schedule entry of its own and so has a cache and state of its own.
"""
from __future__ import annotations

from typing import Dict, Optional, Tuple

from ..config.punolix import PunolixConfig
from ..parts.spec import LayerSpec, ModelSpec, PartSpec, ScheduleEntry, TensorSpec
from .registry import register_architecture

ATTENTION_NAMES = {"q": "q", "k": "k", "v": "v", "o": "o", "q_bias": "q.b", "k_bias": "k.b", "v_bias": "v.b", "o_bias": "o.b", "q_norm": "q.norm", "k_norm": "k.norm",
                   "q_conv": "q.conv", "k_conv": "k.conv", "v_conv": "v.conv"}


def _position(m: dict, interleaved: bool) -> PartSpec:
    rot = m["rot"]
    params = {"head_dim": m["dim"], "theta": rot["base"], "rotary_dim": rot["dims"], "interleaved": interleaved}
    # (without bands the same table with a factor of 1: frequencies in float64, rounded once)
    params.update(rot["scaling"] or {"factor": 1.0, "low": 1.0, "high": 2.0, "original": 1.0})
    return PartSpec("rope_llama3", params)


def _heads(m: dict, h: int, eps: float, interleaved: bool) -> dict:
    return {"hidden": h, "heads": m["heads"], "kv_heads": m["kv_heads"], "head_dim": m["dim"], "v_head_dim": m["vdim"], "scale": m["scale"], "bias": True,
            "norm_eps": eps, "sink": False, "position": _position(m, interleaved), "names": ATTENTION_NAMES}


def _differential(m: dict, h: int, eps: float) -> PartSpec:
    return PartSpec("sink_attention", {**_heads(m, h, eps, True), "qk_norm": None, "softcap": m["softcap"], "differential": m["diff"]})


def _chunked(m: dict, h: int, eps: float) -> PartSpec:
    return PartSpec("sink_attention", {**_heads(m, h, eps, False), "qk_norm": "head", "taps": m["conv"], "out_bias": True,
                                       "chunk": m["mask"]["size"] if m["mask"] is not None else None})


def _linear(m: dict, h: int, eps: float) -> PartSpec:
    return PartSpec("gated_linear_attention", {"hidden": h, "heads": m["heads"], "dim": m["dim"], "vdim": m["vdim"], "tau": m["tau"],
                                               "decay_rank": m["decay_rank"], "norm_eps": eps})


def _mixer(kind: str, m: dict, h: int, eps: float) -> PartSpec:
    if kind == "attention":
        return _differential(m, h, eps)
    return PartSpec("parallel_mixers", {"hidden": h, "inner": {"left": _chunked(m["left"], h, eps), "right": _linear(m["right"], h, eps)},
                                        "scales": {"left": m["left_scale"], "right": m["right_scale"]}})


def _feedforward(mlp: Optional[dict], h: int) -> Optional[PartSpec]:
    if mlp is None:
        return None
    return PartSpec("swiglu", {"hidden": h, "intermediate": mlp["ff"], "activation": "gelu_tanh", "names": ("gate", "up", "down")})


def resolve_shapes(cfg: PunolixConfig, shapes: Dict[str, Tuple[int, ...]]) -> PunolixConfig:
    """Sizes that only the checkpoint gives are taken from the shapes of its tensors, by name, before the model is built."""
    return cfg.with_tensor_shapes(shapes)


def build_spec(cfg: PunolixConfig) -> ModelSpec:
    h = cfg.hidden_size
    norm = PartSpec("rmsnorm", {"dim": h, "eps": cfg.norm_eps, "tensor": ""})
    layers = [LayerSpec(block="parallel_prenorm", norm=norm, mixer=_mixer(layer.type, layer.mixer, h, cfg.norm_eps), feedforward=_feedforward(layer.mlp, h),
                        prefix=f"l{i}", names={"norm1": "norm1", "mixer": "mix", "feedforward": "mlp"}, block_params={"residual_mult": cfg.residual_mult})
              for i, layer in enumerate(cfg.layers)]
    return ModelSpec(
        hidden_size=h,
        vocab_size=cfg.vocab_size,
        embedding=PartSpec("token_table", {"vocab": cfg.vocab_size, "hidden": h, "name": "embed", "tensor": "embed", "scale": cfg.embedding_scale}),
        final_norm=PartSpec("rmsnorm", {"dim": h, "eps": cfg.norm_eps, "name": "final.norm", "tensor": ""}),
        head=PartSpec("linear", {"vocab": cfg.vocab_size, "hidden": h, "name": "head", "tied": False, "tensor": "head"}),
        layers=layers,
        schedule=[ScheduleEntry(i, enters=p) for i, p in cfg.layer_runs],
        pass_vectors=TensorSpec("loop.step", (cfg.loop["times"], h), "bias") if cfg.loop is not None else None,
    )


register_architecture(PunolixConfig.ARCHITECTURE, PunolixConfig.MODEL_TYPE, PunolixConfig, build_spec, resolve_shapes)
