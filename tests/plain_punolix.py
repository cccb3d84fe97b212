"""A plain, slow implementation of Punolix in float64: one function per mechanism, whole sequences only, no cache, no batch.  It
shares nothing with the package; the GPU tests compare the engine with it.

``config`` is the dictionary of a model's ``config.json``; ``tensors`` maps tensor names to float64 tensors.  Matrices are stored
``[out, in]``.
"""
from __future__ import annotations

import math
import os
from typing import Dict, List, Optional

import torch

F = torch.float64


def rms(x: torch.Tensor, eps: float) -> torch.Tensor:
    return torch.sqrt((x * x).mean(-1, keepdim=True) + eps)


def silu(x: torch.Tensor) -> torch.Tensor:
    return x * torch.sigmoid(x)


def gelu_tanh(z: torch.Tensor) -> torch.Tensor:
    return 0.5 * z * (1.0 + torch.tanh(math.sqrt(2.0 / math.pi) * (z + 0.044715 * z ** 3)))


def frequencies(rot: dict) -> List[float]:
    """The angle per position of every rotated pair; with ``scaling``, slow pairs (by wavelength) turn more slowly."""
    out = []
    s = rot.get("scaling")
    for i in range(rot["dims"] // 2):
        f = rot["base"] ** (-2.0 * i / rot["dims"])
        if s is not None:
            length = 2.0 * math.pi / f
            if length > s["original"] / s["low"]:
                f = f / s["factor"]
            elif length >= s["original"] / s["high"]:
                share = (s["original"] / length - s["low"]) / (s["high"] - s["low"])
                f = (1.0 - share) * f / s["factor"] + share * f
        out.append(f)
    return out


def rotate(x: torch.Tensor, rot: dict, interleaved: bool) -> torch.Tensor:
    """``x`` ``[T, heads, dim]``: the first ``dims`` elements in pairs, neighbours or half the width apart."""
    T, n = x.shape[0], rot["dims"]
    angle = torch.arange(T, dtype=F)[:, None] * torch.tensor(frequencies(rot), dtype=F)[None, :]
    c, s = torch.cos(angle)[:, None, :], torch.sin(angle)[:, None, :]
    out = x.clone()
    first, second = (slice(0, n, 2), slice(1, n, 2)) if interleaved else (slice(0, n // 2), slice(n // 2, n))
    u, v = x[..., first], x[..., second]
    out[..., first], out[..., second] = u * c - v * s, v * c + u * s
    return out


def softmax_attention(q: torch.Tensor, k: torch.Tensor, v: torch.Tensor, scale: float, cap: Optional[float] = None,
                      chunk: Optional[int] = None) -> torch.Tensor:
    """``q`` ``[T, H, d]``, ``k`` ``[T, G, d]``, ``v`` ``[T, G, dv]``: causal, grouped; scores capped by a tanh; only the own chunk."""
    T, H, G = q.shape[0], q.shape[1], k.shape[1]
    i, j = torch.arange(T)[:, None], torch.arange(T)[None, :]
    seen = j <= i
    if chunk:
        seen = seen & (i // chunk == j // chunk)
    out = torch.zeros(T, H, v.shape[2], dtype=F)
    for a in range(H):
        c = a // (H // G)
        s = (q[:, a] @ k[:, c].T) * scale
        if cap:
            s = cap * torch.tanh(s / cap)
        out[:, a] = torch.softmax(torch.where(seen, s, torch.full_like(s, -float("inf"))), dim=1) @ v[:, c]
    return out


def lam_of(t: Dict[str, torch.Tensor], name: str, diff: float) -> float:
    return float(torch.exp((t[f"{name}.lq1"] * t[f"{name}.lk1"]).sum()) - torch.exp((t[f"{name}.lq2"] * t[f"{name}.lk2"]).sum()) + diff)


def differential_attention(h: torch.Tensor, t: Dict[str, torch.Tensor], name: str, m: dict, eps: float) -> torch.Tensor:
    """Two softmax maps per head over the same values, the second weighted and subtracted; the difference is divided by its root
    mean square per head and multiplied by ``1 - diff``."""
    T = h.shape[0]
    H, G, d, dv = m["heads"], m["kv_heads"], m["dim"], m["vdim"]
    q = (h @ t[f"{name}.q"].T + t[f"{name}.q.b"]).reshape(T, H, 2, d)
    k = (h @ t[f"{name}.k"].T + t[f"{name}.k.b"]).reshape(T, G, 2, d)
    v = (h @ t[f"{name}.v"].T + t[f"{name}.v.b"]).reshape(T, G, dv)
    a1, a2 = (softmax_attention(rotate(q[:, :, n], m["rot"], True), rotate(k[:, :, n], m["rot"], True), v, m["scale"], m.get("softcap")) for n in (0, 1))
    o = a1 - lam_of(t, name, m["diff"]) * a2
    o = o / rms(o, eps) * (1.0 - m["diff"])
    return o.reshape(T, H * dv) @ t[f"{name}.o"].T


def short_convolution(x: torch.Tensor, w: torch.Tensor) -> torch.Tensor:
    """Per channel, over the last ``taps`` rows (zeros before the first), the last column on the current row."""
    taps = w.shape[1]
    padded = torch.cat([torch.zeros(taps - 1, x.shape[1], dtype=F), x], dim=0)
    out = torch.zeros_like(x)
    for j in range(taps):
        out += padded[j:j + x.shape[0]] * w[:, j]
    return out


def chunked_attention(h: torch.Tensor, t: Dict[str, torch.Tensor], name: str, m: dict, eps: float) -> torch.Tensor:
    """Grouped-query attention inside chunks of the sequence; biased projections through a short convolution, q and k normed per
    head, rotated; the output projection has a bias."""
    T = h.shape[0]
    H, G, d, dv = m["heads"], m["kv_heads"], m["dim"], m["vdim"]
    q, k, v = (h @ t[f"{name}.{p}"].T + t[f"{name}.{p}.b"] for p in "qkv")
    if m.get("conv"):
        q, k, v = (short_convolution(x, t[f"{name}.{p}.conv"]) for p, x in zip("qkv", (q, k, v)))
    q, k = q.reshape(T, H, d), k.reshape(T, G, d)
    q = rotate(q / rms(q, eps) * t[f"{name}.q.norm"], m["rot"], False)
    k = rotate(k / rms(k, eps) * t[f"{name}.k.norm"], m["rot"], False)
    o = softmax_attention(q, k, v.reshape(T, G, dv), m["scale"], None, (m.get("mask") or {}).get("size"))
    return o.reshape(T, H * dv) @ t[f"{name}.o"].T + t[f"{name}.o.b"]


def linear_recurrence(q, k, v, decay, start: Optional[torch.Tensor] = None, ends: Optional[list] = None) -> torch.Tensor:
    """``q``, ``k``, ``decay`` ``[T, heads, dim]``, ``v`` ``[T, heads, vdim]``: ``S <- diag(decay) S + k v^T``, ``o = S^T q`` per head."""
    T, H, d = q.shape
    S = torch.zeros(H, d, v.shape[2], dtype=F) if start is None else start.clone()
    out = torch.zeros(T, H, v.shape[2], dtype=F)
    for i in range(T):
        S = decay[i][:, :, None] * S + k[i][:, :, None] * v[i][:, None, :]
        out[i] = torch.einsum("hdv,hd->hv", S, q[i])
    if ends is not None:
        ends.append(S)
    return out


def gated_linear_attention(h: torch.Tensor, t: Dict[str, torch.Tensor], name: str, m: dict, eps: float) -> torch.Tensor:
    T = h.shape[0]
    H, d, dv = m["heads"], m["dim"], m["vdim"]
    q = (h @ t[f"{name}.q"].T).reshape(T, H, d) * d ** -0.5
    k = (h @ t[f"{name}.k"].T).reshape(T, H, d)
    v = (h @ t[f"{name}.v"].T).reshape(T, H, dv)
    z = (h @ t[f"{name}.a1"].T) @ t[f"{name}.a2"].T + t[f"{name}.a2.b"]
    o = linear_recurrence(q, k, v, (torch.sigmoid(z) ** (1.0 / m["tau"])).reshape(T, H, d))
    o = (o / rms(o, eps) * t[f"{name}.norm"]).reshape(T, H * dv) * silu(h @ t[f"{name}.g"].T)
    return o @ t[f"{name}.o"].T


def mixer(layer: dict, h: torch.Tensor, t: Dict[str, torch.Tensor], name: str, eps: float) -> torch.Tensor:
    m = layer["mixer"]
    if layer["type"] == "attention":
        return differential_attention(h, t, name, m, eps)
    return (m["left_scale"] * chunked_attention(h, t, f"{name}.left", m["left"], eps)
            + m["right_scale"] * gated_linear_attention(h, t, f"{name}.right", m["right"], eps))


def feed_forward(h: torch.Tensor, t: Dict[str, torch.Tensor], name: str) -> torch.Tensor:
    return (gelu_tanh(h @ t[f"{name}.gate"].T) * (h @ t[f"{name}.up"].T)) @ t[f"{name}.down"].T


def parallel_layer(layer: dict, x: torch.Tensor, t: Dict[str, torch.Tensor], name: str, eps: float, mult: float) -> torch.Tensor:
    """One norm, both sublayers read it, their sum times ``mult`` is added."""
    h = x / rms(x, eps) * t[f"{name}.norm1"]
    y = mixer(layer, h, t, f"{name}.mix", eps)
    if layer.get("mlp") is not None:
        y = y + feed_forward(h, t, f"{name}.mlp")
    return x + mult * y


def layer_runs(config: dict) -> List[tuple]:
    """The layers in the order they run: ``(layer, pass of the loop that starts right before it, or None)``."""
    n, loop = len(config["layers"]), config.get("loop")
    if loop is None:
        return [(i, None) for i in range(n)]
    runs = [(i, None) for i in range(loop["start"])]
    for p in range(loop["times"]):
        runs += [(i, p if i == loop["start"] else None) for i in range(loop["start"], loop["stop"])]
    return runs + [(i, None) for i in range(loop["stop"], n)]


def read_weights(path: str) -> Dict[str, torch.Tensor]:
    from safetensors.torch import load_file

    return {k: v.to(F) for k, v in load_file(os.path.join(path, "model.safetensors")).items()}


def forward(config: dict, tensors: Dict[str, torch.Tensor], tokens: List[int], residuals: Optional[list] = None) -> torch.Tensor:
    """Logits ``[T, vocab]`` of one sequence from its first position; ``residuals`` collects the stream after every layer run."""
    eps, t = config["norm"]["eps"], tensors
    first = t["embed"][torch.tensor(tokens)] * (config.get("embedding") or {}).get("scale", 1.0)
    x = first.clone()
    for i, entered in layer_runs(config):
        if entered is not None:
            if entered > 0:
                x = x + first
            x = x + t["loop.step"][entered]
        x = parallel_layer(config["layers"][i], x, t, f"l{i}", eps, config.get("residual_mult", 1.0))
        if residuals is not None:
            residuals.append(x.clone())
    return (x / rms(x, eps) * t["final.norm"]) @ t["head"].T
