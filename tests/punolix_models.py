"""Small Punolix configurations and random weights for the tests, written with the ``safetensors`` library (not with the engine's own
writer).  Weights are drawn so that every mechanism matters: second maps that take away a good part of the first, biases as large as what they
are added to, scores that reach their cap, convolutions that mix tokens, decays from long memory to a token's.  Values are rounded to
bfloat16 so that a 32-bit engine and the plain implementation read the same numbers.
"""
from __future__ import annotations

import json
import math
import os
from typing import Dict

import torch


def _rot(dims, base, scaling=None):
    rot = {"dims": dims, "base": base}
    if scaling:
        rot["scaling"] = dict(zip(("factor", "low", "high", "original"), scaling))
    return rot


def _diff(heads, kv, dim, vdim, scale, rot, diff, softcap=None):
    m = {"heads": heads, "kv_heads": kv, "dim": dim, "vdim": vdim, "scale": scale, "rot": rot, "diff": diff}
    if softcap:
        m["softcap"] = softcap
    return m


def _left(heads, kv, dim, vdim, scale, rot, conv=None, chunk=None):
    m = {"heads": heads, "kv_heads": kv, "dim": dim, "vdim": vdim, "scale": scale, "rot": rot}
    if conv:
        m["conv"] = conv
    if chunk:
        m["mask"] = {"size": chunk}
    return m


def _right(heads, dim, vdim, tau):
    return {"heads": heads, "dim": dim, "vdim": vdim, "tau": tau}


def _parallel(left, right, ls, rs):
    return {"left": left, "right": right, "left_scale": ls, "right_scale": rs}


def _layer(kind, mixer, ff):
    return {"type": kind, "mixer": mixer, "mlp": {"kind": "dense", "ff": ff} if ff else None}


# Sizes that fit no tensor-core kernel: maps of 6 over one kv head, a chunk of 11 over pages of four, three taps, heads of 6 x 9; a loop of two
# layers that starts at the first one.
CONFIG_A = {"architecture": "Punolix", "vocab": 83, "width": 44, "norm": {"eps": 1e-5}, "embedding": {"scale": 3.0}, "residual_mult": 0.7,
            "loop": {"start": 0, "stop": 2, "times": 3},
            "layers": [_layer("attention", _diff(3, 1, 6, 10, 0.5, _rot(4, 500.0), 0.25, softcap=6.0), 60),
                       _layer("parallel", _parallel(_left(4, 2, 12, 10, 0.3, _rot(8, 900.0, (3.0, 1.0, 4.0, 60)), conv=3, chunk=11), _right(3, 6, 9, 8.0), 0.7, -0.9), 52),
                       _layer("attention", _diff(4, 4, 10, 7, 0.4, _rot(10, 2000.0), 0.5, softcap=3.0), None)]}
# Sizes the tensor-core kernels are made for: two maps of 64 over values of 128, of 32 over 128 and of 64 over 64; chunks of 70 with keys of 128 over
# values of 64; heads of 64 x 64 and 32 x 48; the loop leaves out the first and the last layer.
CONFIG_B = {"architecture": "Punolix", "vocab": 170, "width": 128, "norm": {"eps": 1e-6}, "embedding": {"scale": 8.0}, "residual_mult": 0.5,
            "loop": {"start": 1, "stop": 3, "times": 2},
            "layers": [_layer("attention", _diff(8, 2, 64, 128, 0.125, _rot(64, 10000.0), 0.3, softcap=20.0), 256),
                       _layer("parallel", _parallel(_left(8, 2, 128, 64, 0.09, _rot(64, 50000.0, (8.0, 1.0, 4.0, 128)), conv=4, chunk=70), _right(4, 64, 64, 16.0), 0.8, 0.6), 192),
                       _layer("attention", _diff(3, 3, 32, 128, 0.18, _rot(16, 3000.0), 0.6), 128),
                       _layer("parallel", _parallel(_left(4, 4, 64, 64, 0.125, _rot(64, 10000.0), conv=2, chunk=33), _right(2, 32, 48, 4.0), 0.5, 1.1), None),
                       _layer("attention", _diff(4, 1, 64, 64, 0.125, _rot(32, 10000.0), 0.1, softcap=8.0), 64)]}
# Edges of the parameter space: a loop of a single layer in a single pass, no residual multiplier, no embedding scale, no cap, chunks of one
# position, no chunks, no convolution, one tap, seven taps, a single rotated pair, a decay that is not slowed, heads of 16 x 256 and 128 x 12.
CONFIG_C = {"architecture": "Punolix", "vocab": 70, "width": 64, "norm": {"eps": 1e-6}, "loop": {"start": 2, "stop": 3, "times": 1},
            "layers": [_layer("parallel", _parallel(_left(2, 2, 16, 16, 0.25, _rot(2, 100.0), conv=1), _right(2, 16, 256, 1.0), 1.0, 1.0), None),
                       _layer("attention", _diff(2, 2, 16, 16, 0.3, _rot(16, 100.0), 0.8), 48),
                       _layer("parallel", _parallel(_left(4, 1, 32, 48, 0.2, _rot(32, 1000.0, (2.0, 0.5, 3.0, 32)), chunk=1), _right(1, 128, 12, 32.0), 0.3, 0.9), 40),
                       _layer("parallel", _parallel(_left(6, 3, 48, 32, 0.15, _rot(24, 1000.0), conv=7, chunk=24), _right(3, 48, 80, 5.0), -0.6, 0.6), 96),
                       _layer("attention", _diff(8, 1, 48, 80, 0.15, _rot(40, 5000.0), -0.2, softcap=2.0), 32)]}
CONFIGS = {"A": CONFIG_A, "B": CONFIG_B, "C": CONFIG_C}
PAGE = {"A": 4, "B": 16, "C": 8}
#: numbers between the decays' two matrices (in no key: the tensors' shapes give them)
RANK = {44: 5, 128: 16, 64: 24}


def attention_tensors(normal, matrix, w, p, m):
    """q, k, v with biases and the four vectors of lambda for differential attention."""
    H, G, d, dv, width = m["heads"], m["kv_heads"], m["dim"], m["vdim"], matrix.cols
    for key, rows in (("q", 2 * H * d), ("k", 2 * G * d), ("v", G * dv)):
        w[f"{p}.{key}"], w[f"{p}.{key}.b"] = matrix(rows, width, 1.3), normal(rows, std=0.4)
    for key in ("lq1", "lk1", "lq2", "lk2"):
        w[f"{p}.{key}"] = normal(d, std=0.5 / d ** 0.5)
    w[p + ".o"] = matrix(width, H * dv, 1.5)


def left_tensors(normal, matrix, w, p, m):
    H, G, d, dv, width = m["heads"], m["kv_heads"], m["dim"], m["vdim"], matrix.cols
    for key, rows in (("q", H * d), ("k", G * d), ("v", G * dv)):
        w[f"{p}.{key}"], w[f"{p}.{key}.b"] = matrix(rows, width), normal(rows, std=0.4)
        if m.get("conv"):
            w[f"{p}.{key}.conv"] = normal(rows, m["conv"], std=0.7)
    w[p + ".q.norm"], w[p + ".k.norm"] = normal(d, std=0.3, mean=1.4), normal(d, std=0.3, mean=1.4)
    w[p + ".o"], w[p + ".o.b"] = matrix(width, H * dv, 1.5), normal(width, std=0.5)


def right_tensors(normal, matrix, w, p, m, rank):
    H, d, dv, width = m["heads"], m["dim"], m["vdim"], matrix.cols
    for key, rows in (("q", H * d), ("k", H * d), ("v", H * dv), ("g", H * dv)):
        w[f"{p}.{key}"] = matrix(rows, width, 1.3)
    w[p + ".a1"], w[p + ".a2"], w[p + ".a2.b"] = matrix(rank, width), matrix(H * d, rank, 1.5), normal(H * d, std=2.0, mean=1.0)
    w[p + ".norm"], w[p + ".o"] = normal(dv, std=0.2, mean=1.0), matrix(width, H * dv, 1.5)


class Draw:
    """Random matrices of a generator; ``cols`` is the model's width."""

    def __init__(self, seed: int, cols: int):
        self.g, self.cols = torch.Generator().manual_seed(seed), cols

    def normal(self, *shape, std=1.0, mean=0.0):
        return torch.randn(shape, generator=self.g) * std + mean

    def __call__(self, rows, cols, gain=1.0):
        return self.normal(rows, cols, std=gain / math.sqrt(cols))


def random_weights(raw: dict, seed: int) -> Dict[str, torch.Tensor]:
    width, vocab = raw["width"], raw["vocab"]
    matrix = Draw(seed, width)
    normal = matrix.normal
    scale = (raw.get("embedding") or {}).get("scale", 1.0)
    w: Dict[str, torch.Tensor] = {"embed": normal(vocab, width, std=1.0 / scale), "head": matrix(vocab, width, 1.5), "final.norm": normal(width, std=0.2, mean=1.0)}
    if raw.get("loop") is not None:
        w["loop.step"] = normal(raw["loop"]["times"], width, std=0.5)
    for i, layer in enumerate(raw["layers"]):
        p, m = f"l{i}", layer["mixer"]
        w[p + ".norm1"] = normal(width, std=0.2, mean=1.0)
        if layer["type"] == "attention":
            attention_tensors(normal, matrix, w, p + ".mix", m)
        else:
            left_tensors(normal, matrix, w, p + ".mix.left", m["left"])
            right_tensors(normal, matrix, w, p + ".mix.right", m["right"], RANK.get(width, 16))
        if layer.get("mlp") is not None:
            ff = layer["mlp"]["ff"]
            w[p + ".mlp.gate"], w[p + ".mlp.up"], w[p + ".mlp.down"] = matrix(ff, width, 1.3), matrix(ff, width), matrix(width, ff, 1.5)
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
