"""Small Pununex configurations and random weights for the tests, written with the ``safetensors`` library (not with the
engine's own writer).  Weights are drawn so that every mechanism matters: sinks from weak to strong, decays from long memory to a
token's, scores that reach their cap, choice corrections that overrule scores.  Values are rounded to bfloat16 so that a 32-bit
engine and the plain implementation read the same numbers.
"""
from __future__ import annotations

import json
import math
import os
from typing import Dict

import torch


def _attn(heads, kv, dim, vdim, scale, size=None, keep=None, softcap=None):
    m = {"heads": heads, "kv_heads": kv, "dim": dim, "vdim": vdim, "scale": scale}
    if size:
        m["mask"] = {"size": size}
        if keep is not None:
            m["mask"]["keep_first"] = keep
    if softcap:
        m["softcap"] = softcap
    return m


def _delta(heads, kv, dim, vdim, conv):
    return {"heads": heads, "kv_heads": kv, "dim": dim, "vdim": vdim, "conv": conv}


def _parallel(left, right, ls, rs):
    return {"left": left, "right": right, "left_scale": ls, "right_scale": rs}


def _moe(ff, experts, top, identity=None, groups=None, scale=1.0, shared=None):
    router = {"experts": experts, "top": top, "scale": scale}
    if identity is not None:
        router["identity"] = identity
    if groups:
        router["groups"] = {"count": groups[0], "keep": groups[1]}
    mlp = {"kind": "moe", "expert": {"ff": ff}, "router": router}
    if shared:
        mlp["shared"] = {"ff": shared}
    return mlp


def _dense(ff):
    return {"kind": "dense", "ff": ff}


# Sizes that fit no tensor-core kernel: three heads of 12 over one kv head, a window of 9 that also keeps four positions
# (inside one page of four, and the window's own pages are given back), delta heads of 10 x 14 that share two q/k heads,
# three taps; two of five experts and one identity output in three groups of two.
CONFIG_A = {"architecture": "Pununex", "vocab": 83, "width": 44, "norm": {"eps": 1e-5}, "embedding": {"bigram": {"buckets": 31, "mul_prev": 5, "mul_cur": 3}},
            "layers": [{"type": "delta", "mixer": _delta(4, 2, 10, 14, 3), "mlp": _dense(60)},
                       {"type": "parallel", "mixer": _parallel(_attn(3, 1, 12, 10, 0.3, size=9, keep=4, softcap=4.0), _delta(2, 1, 6, 9, 3), 0.7, -0.9),
                        "mlp": _moe(28, 5, 2, identity=1, groups=(3, 2), scale=1.5, shared=36)},
                       {"type": "parallel", "mixer": _parallel(_attn(4, 2, 10, 16, 0.25, size=5, keep=11, softcap=9.0), _delta(3, 3, 8, 12, 2), 1.2, 0.4),
                        "mlp": _dense(40)}]}
# Sizes the tensor-core kernels are made for: heads of 64 with values as wide, delta heads of 64 x 64 and 32 x 48, experts in
# whole steps of 64; a window of 70 with 20 kept positions over pages of sixteen; three identity outputs among twelve.
CONFIG_B = {"architecture": "Pununex", "vocab": 170, "width": 128, "norm": {"eps": 1e-6}, "embedding": {"bigram": {"buckets": 97, "mul_prev": 13, "mul_cur": 11}},
            "layers": [{"type": "parallel", "mixer": _parallel(_attn(8, 2, 64, 64, 0.125, size=70, keep=20, softcap=20.0), _delta(4, 2, 64, 64, 4), 0.8, 0.5),
                        "mlp": _moe(64, 9, 3, identity=3, groups=(4, 2), scale=2.5, shared=128)},
                       {"type": "delta", "mixer": _delta(6, 3, 32, 48, 4), "mlp": _dense(256)},
                       {"type": "parallel", "mixer": _parallel(_attn(4, 4, 48, 32, 0.15, size=33, keep=3, softcap=50.0), _delta(2, 2, 128, 32, 5), 0.5, 1.1),
                        "mlp": _moe(128, 6, 1, identity=2, groups=(2, 1), scale=1.0, shared=64)}]}
# Edges of the parameter space: no bigram embedding, no feed-forward, no mask, no cap, a window of one position, more kept
# positions than the window is long, nothing kept, a convolution of a single tap, no identity outputs, no groups, all groups kept,
# no shared expert, every expert chosen, key heads much smaller and larger than the value heads.
CONFIG_C = {"architecture": "Pununex", "vocab": 70, "width": 64, "norm": {"eps": 1e-6},
            "layers": [{"type": "parallel", "mixer": _parallel(_attn(2, 2, 16, 16, 0.25), _delta(2, 1, 32, 128, 1), 1.0, 1.0), "mlp": None},
                       {"type": "parallel", "mixer": _parallel(_attn(4, 1, 32, 48, 0.2, size=1, keep=2), _delta(1, 1, 128, 9, 2), 0.3, 0.9),
                        "mlp": _moe(32, 4, 4)},
                       {"type": "delta", "mixer": _delta(2, 2, 16, 16, 7), "mlp": _moe(64, 4, 2, groups=(2, 2), scale=0.5)},
                       {"type": "parallel", "mixer": _parallel(_attn(2, 1, 16, 32, 0.3, size=24, softcap=3.0), _delta(3, 1, 16, 48, 4), 0.6, 0.6),
                        "mlp": _moe(64, 2, 2, identity=2, shared=32)}]}
CONFIGS = {"A": CONFIG_A, "B": CONFIG_B, "C": CONFIG_C}
PAGE = {"A": 4, "B": 16, "C": 8}


def random_weights(raw: dict, seed: int) -> Dict[str, torch.Tensor]:
    g = torch.Generator().manual_seed(seed)
    width, vocab = raw["width"], raw["vocab"]

    def normal(*shape, std=1.0, mean=0.0):
        return torch.randn(shape, generator=g) * std + mean

    def matrix(rows, cols, gain=1.0):
        return normal(rows, cols, std=gain / math.sqrt(cols))

    def norm(name):
        w[name], w[name + ".b"] = normal(width, std=0.2, mean=1.0), normal(width, std=0.2)

    def attention(p, m):
        H, G, d, dv = m["heads"], m["kv_heads"], m["dim"], m["vdim"]
        w[p + ".q"], w[p + ".k"], w[p + ".v"] = matrix(H * d, width), matrix(G * d, width), matrix(G * dv, width)
        w[p + ".q.norm"], w[p + ".k.norm"] = normal(d, std=0.3, mean=1.4), normal(d, std=0.3, mean=1.4)
        w[p + ".sink"] = normal(H, std=2.0)
        w[p + ".o"] = matrix(width, H * dv, 1.5)

    def delta(p, m, low_rank):
        H, G, d, dv, taps = m["heads"], m["kv_heads"], m["dim"], m["vdim"], m["conv"]
        for key, rows in (("q", G * d), ("k", G * d), ("v", H * dv)):
            w[f"{p}.{key}"], w[f"{p}.{key}.conv"] = matrix(rows, width, 1.5), normal(rows, taps, std=0.7)
        w[p + ".b"], w[p + ".norm"], w[p + ".o"] = matrix(H, width, 1.5), normal(dv, std=0.2, mean=1.0), matrix(width, H * dv, 1.5)
        w[p + ".A_log"] = torch.rand(H, generator=g) * 4.5 - 3.5                # rates from 0.03 (long memory) to 2.7
        if low_rank:
            # (two ranks that differ, neither a multiple of 8 in every configuration)
            ra, rg = m.get("decay_rank", 12 + width % 7), m.get("gate_rank", 16)
            w[p + ".a1"], w[p + ".a2"], w[p + ".dt_bias"] = matrix(ra, width), matrix(H * d, ra), normal(H * d, std=1.0, mean=-1.0)
            w[p + ".g1"], w[p + ".g2"] = matrix(rg, width), matrix(H * dv, rg, 2.0)
        else:
            w[p + ".a"], w[p + ".dt_bias"], w[p + ".g"] = matrix(H, width), normal(H, std=1.0, mean=-1.0), matrix(H * dv, width)

    w: Dict[str, torch.Tensor] = {"embed": normal(vocab, width), "head": matrix(vocab, width, 1.5)}
    norm("final.norm")
    bigram = (raw.get("embedding") or {}).get("bigram")
    if bigram is not None:
        w["bigram"] = normal(bigram["buckets"] + 1, width)
    for i, layer in enumerate(raw["layers"]):
        p, m = f"l{i}", layer["mixer"]
        norm(p + ".norm1")
        w[p + ".ls1"] = normal(width, std=0.2, mean=0.9)
        if layer["type"] == "delta":
            delta(p + ".mix", m, False)
        else:
            attention(p + ".mix.left", m["left"])
            delta(p + ".mix.right", m["right"], True)
        mlp = layer.get("mlp")
        if mlp is None:
            continue
        norm(p + ".norm2")
        w[p + ".ls2"] = normal(width, std=0.2, mean=0.9)
        experts = [("", mlp["ff"])] if mlp["kind"] == "dense" else [(f".e{e}", mlp["expert"]["ff"]) for e in range(mlp["router"]["experts"])]
        if mlp.get("shared"):
            experts.append((".shared", mlp["shared"]["ff"]))
        for name, ff in experts:
            w[f"{p}.mlp{name}.gate"], w[f"{p}.mlp{name}.up"], w[f"{p}.mlp{name}.down"] = matrix(ff, width), matrix(ff, width), matrix(width, ff, 1.5)
        if mlp["kind"] == "moe":
            n = mlp["router"]["experts"] + mlp["router"].get("identity", 0)
            # (all corrections below zero: what a group that is not kept counts as must not be 0)
            w[p + ".mlp.router"], w[p + ".mlp.correction"] = matrix(n, width, 0.7), normal(n, std=0.3, mean=-1.5)
    return {k: v.to(torch.bfloat16) for k, v in w.items()}


def write_model(path: str, raw: dict, weights: Dict[str, torch.Tensor]) -> str:
    from safetensors.torch import save_file

    os.makedirs(path, exist_ok=True)
    with open(os.path.join(path, "config.json"), "w") as fh:
        json.dump(raw, fh)
    save_file({k: v.contiguous() for k, v in weights.items()}, os.path.join(path, "model.safetensors"))
    return path


def make_model_dir(path: str, name: str, seed: int = 3) -> str:
    return write_model(path, CONFIGS[name], random_weights(CONFIGS[name], seed))
