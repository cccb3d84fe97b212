"""A plain, slow implementation of Pununex in float64: one function per mechanism, whole sequences only, no cache, no
batch.  It shares nothing with the package; the GPU tests compare the engine with it.

``config`` is the dictionary of a model's ``config.json``; ``tensors`` maps tensor names to float64 tensors.  Matrices are
stored ``[out, in]``.
"""
from __future__ import annotations

import os
from typing import Dict, List, Optional

import torch

F = torch.float64


def rms_norm(x: torch.Tensor, w: torch.Tensor, eps: float) -> torch.Tensor:
    return x / torch.sqrt((x * x).mean(-1, keepdim=True) + eps) * w


def layer_norm(x: torch.Tensor, w: torch.Tensor, b: torch.Tensor, eps: float) -> torch.Tensor:
    centred = x - x.mean(-1, keepdim=True)
    return centred / torch.sqrt((centred * centred).mean(-1, keepdim=True) + eps) * w + b


def silu(x: torch.Tensor) -> torch.Tensor:
    return x * torch.sigmoid(x)


def softplus(x: torch.Tensor) -> torch.Tensor:
    return torch.clamp(x, min=0.0) + torch.log1p(torch.exp(-x.abs()))


def embedding(tokens: List[int], t: Dict[str, torch.Tensor], bigram: Optional[dict]) -> torch.Tensor:
    """The token's row, plus a row of a second table chosen by a hash of the token before it and itself (the table's last row
    for the first token of a sequence)."""
    x = t["embed"][torch.tensor(tokens)].clone()
    if bigram is not None:
        for i, token in enumerate(tokens):
            row = bigram["buckets"] if i == 0 else (tokens[i - 1] * bigram["mul_prev"] + token * bigram["mul_cur"]) % bigram["buckets"]
            x[i] += t["bigram"][row]
    return x


def sink_window_attention(h: torch.Tensor, t: Dict[str, torch.Tensor], name: str, m: dict, eps: float) -> torch.Tensor:
    """Grouped-query softmax attention without a rotation: RMS norm of q and k per head, scores capped by a tanh, a window
    that also keeps the sequence's first positions, a learned number per head in the denominator."""
    T = h.shape[0]
    H, G, d, dv = m["heads"], m["kv_heads"], m["dim"], m["vdim"]
    q = rms_norm((h @ t[f"{name}.q"].T).reshape(T, H, d), t[f"{name}.q.norm"], eps)
    k = rms_norm((h @ t[f"{name}.k"].T).reshape(T, G, d), t[f"{name}.k.norm"], eps)
    v = (h @ t[f"{name}.v"].T).reshape(T, G, dv)
    mask = m.get("mask") or {}
    size, keep, cap = mask.get("size"), mask.get("keep_first", 0), m.get("softcap")
    i, j = torch.arange(T)[:, None], torch.arange(T)[None, :]
    seen = j <= i
    if size:
        seen = seen & ((i - j < size) | (j < keep))
    out = torch.zeros(T, H, dv, dtype=F)
    for a in range(H):
        c = a // (H // G)
        s = (q[:, a] @ k[:, c].T) * m["scale"]
        if cap:
            s = cap * torch.tanh(s / cap)
        s = torch.where(seen, s, torch.full_like(s, -float("inf")))
        sink = t[f"{name}.sink"][a]
        top = torch.maximum(s.max(dim=1, keepdim=True).values, sink)
        e = torch.exp(s - top)
        out[:, a] = (e / (e.sum(1, keepdim=True) + torch.exp(sink - top))) @ v[:, c]
    return out.reshape(T, H * dv) @ t[f"{name}.o"].T


def short_convolution(x: torch.Tensor, w: torch.Tensor) -> torch.Tensor:
    """Per channel, over the last ``taps`` rows (zeros before the first), the last column on the current row; then silu."""
    taps = w.shape[1]
    padded = torch.cat([torch.zeros(taps - 1, x.shape[1], dtype=F), x], dim=0)
    out = torch.zeros_like(x)
    for j in range(taps):
        out += padded[j:j + x.shape[0]] * w[:, j]
    return silu(out)


def unit(x: torch.Tensor) -> torch.Tensor:
    return x / torch.sqrt((x * x).sum(-1, keepdim=True) + 1e-6)


def delta_rule(q, k, v, beta, decay, start: Optional[torch.Tensor] = None, ends: Optional[list] = None) -> torch.Tensor:
    """``q``, ``k``, ``decay`` ``[T, heads, dim]``, ``v`` ``[T, heads, vdim]``, ``beta`` ``[T, heads]``: token by token per head
    ``S <- decay S`` (row by row), ``u = beta (v - S^T k)``, ``S <- S + k u^T``, ``o = S^T q``.  ``ends`` collects the last state."""
    T, H, d = q.shape
    S = torch.zeros(H, d, v.shape[2], dtype=F) if start is None else start.clone()
    out = torch.zeros(T, H, v.shape[2], dtype=F)
    for i in range(T):
        S = decay[i][:, :, None] * S
        u = beta[i][:, None] * (v[i] - torch.einsum("hdv,hd->hv", S, k[i]))
        S = S + k[i][:, :, None] * u[:, None, :]
        out[i] = torch.einsum("hdv,hd->hv", S, q[i])
    if ends is not None:
        ends.append(S)
    return out


def delta_mixer(h: torch.Tensor, t: Dict[str, torch.Tensor], name: str, m: dict, eps: float, per_channel: bool) -> torch.Tensor:
    """A gated delta rule behind short convolutions.  ``per_channel``: one decay per head and key channel and a sigmoid gate,
    both out of small products of two matrices; else one decay per head and a silu gate."""
    T = h.shape[0]
    H, G, d, dv = m["heads"], m["kv_heads"], m["dim"], m["vdim"]
    q, k, v = (short_convolution(h @ t[f"{name}.{p}"].T, t[f"{name}.{p}.conv"]) for p in "qkv")
    of = torch.arange(H) // (H // G)
    q = (unit(q.reshape(T, G, d)) * d ** -0.5)[:, of]
    k = unit(k.reshape(T, G, d))[:, of]
    beta = torch.sigmoid(h @ t[f"{name}.b"].T)
    rate = torch.exp(t[f"{name}.A_log"])
    if per_channel:
        a = (h @ t[f"{name}.a1"].T) @ t[f"{name}.a2"].T + t[f"{name}.dt_bias"]
        decay = torch.exp(-rate[None, :, None] * softplus(a).reshape(T, H, d))
        gate = torch.sigmoid((h @ t[f"{name}.g1"].T) @ t[f"{name}.g2"].T)
    else:
        a = h @ t[f"{name}.a"].T + t[f"{name}.dt_bias"]
        decay = torch.exp(-rate * softplus(a))[:, :, None].expand(T, H, d)
        gate = silu(h @ t[f"{name}.g"].T)
    o = delta_rule(q, k, v.reshape(T, H, dv), beta, decay)
    o = rms_norm(o, t[f"{name}.norm"], eps) * gate.reshape(T, H, dv)
    return o.reshape(T, H * dv) @ t[f"{name}.o"].T


def mixer(layer: dict, h: torch.Tensor, t: Dict[str, torch.Tensor], name: str, eps: float) -> torch.Tensor:
    m = layer["mixer"]
    if layer["type"] == "delta":
        return delta_mixer(h, t, name, m, eps, False)
    return (m["left_scale"] * sink_window_attention(h, t, f"{name}.left", m["left"], eps)
            + m["right_scale"] * delta_mixer(h, t, f"{name}.right", m["right"], eps, True))


def gated_mlp(h: torch.Tensor, gate: torch.Tensor, up: torch.Tensor, down: torch.Tensor, act) -> torch.Tensor:
    return (act(h @ gate.T) * (h @ up.T)) @ down.T


def relu(x: torch.Tensor) -> torch.Tensor:
    return torch.clamp(x, min=0.0)


def route(h: torch.Tensor, t: Dict[str, torch.Tensor], name: str, router: dict):
    """Per row: the chosen outputs of the router (real experts first, then identity experts), their weights, and how far the
    choice is from falling otherwise (the smaller of the gap between the last kept and the first dropped group and the gap
    between the last chosen and the first passed-over output among the kept groups)."""
    top, groups = router["top"], router.get("groups") or {"count": 1, "keep": 1}
    s = torch.softmax(h @ t[f"{name}.router"].T, dim=-1)
    choice = s + t[f"{name}.correction"] if f"{name}.correction" in t else s
    T, E = s.shape
    per = E // groups["count"]
    chosen, weights, margins = [], [], []
    for i in range(T):
        best = choice[i].reshape(groups["count"], per).max(dim=1).values
        order = torch.sort(best, descending=True, stable=True)
        kept = order.indices[:groups["keep"]].tolist()
        gap = float("inf")
        if groups["keep"] < groups["count"]:
            gap = float(order.values[groups["keep"] - 1] - order.values[groups["keep"]])
        allowed = [g * per + k for g in sorted(kept) for k in range(per)]
        ranked = sorted(allowed, key=lambda e: (-float(choice[i, e]), e))
        if top < len(ranked):
            gap = min(gap, float(choice[i, ranked[top - 1]] - choice[i, ranked[top]]))
        picked = ranked[:top]
        w = s[i, picked]
        chosen.append(picked)
        weights.append(w / (w.sum() + 1e-20) * router["scale"])
        margins.append(gap)
    return chosen, weights, torch.tensor(margins, dtype=F)


def routed_mlp(h: torch.Tensor, t: Dict[str, torch.Tensor], name: str, mlp: dict, margins: Optional[list] = None) -> torch.Tensor:
    chosen, weights, gaps = route(h, t, name, mlp["router"])
    if margins is not None:
        margins.append(gaps)
    E = mlp["router"]["experts"]
    out = torch.zeros_like(h)
    for i, (picked, w) in enumerate(zip(chosen, weights)):
        for e, wt in zip(picked, w):
            y = h[i] if e >= E else gated_mlp(h[i:i + 1], t[f"{name}.e{e}.gate"], t[f"{name}.e{e}.up"], t[f"{name}.e{e}.down"], silu)[0]
            out[i] += wt * y
    if mlp.get("shared") is not None:
        out = out + gated_mlp(h, t[f"{name}.shared.gate"], t[f"{name}.shared.up"], t[f"{name}.shared.down"], silu)
    return out


def feed_forward(h: torch.Tensor, t: Dict[str, torch.Tensor], name: str, mlp: dict, margins: Optional[list] = None) -> torch.Tensor:
    if mlp["kind"] == "dense":
        return gated_mlp(h, t[f"{name}.gate"], t[f"{name}.up"], t[f"{name}.down"], relu)
    return routed_mlp(h, t, name, mlp, margins)


def read_weights(path: str) -> Dict[str, torch.Tensor]:
    from safetensors.torch import load_file

    return {k: v.to(F) for k, v in load_file(os.path.join(path, "model.safetensors")).items()}


def forward(config: dict, tensors: Dict[str, torch.Tensor], tokens: List[int], residuals: Optional[list] = None,
            margins: Optional[list] = None) -> torch.Tensor:
    """Logits ``[T, vocab]`` of one sequence from its first position; ``residuals`` collects the stream after every layer,
    ``margins`` every routed layer's margins (see ``route``)."""
    eps, t = config["norm"]["eps"], tensors
    x = embedding(tokens, t, (config.get("embedding") or {}).get("bigram"))
    for i, layer in enumerate(config["layers"]):
        p = f"l{i}"
        x = x + layer_norm(mixer(layer, x, t, f"{p}.mix", eps), t[f"{p}.norm1"], t[f"{p}.norm1.b"], eps) * t[f"{p}.ls1"]
        if layer.get("mlp") is not None:
            x = x + layer_norm(feed_forward(x, t, f"{p}.mlp", layer["mlp"], margins), t[f"{p}.norm2"], t[f"{p}.norm2.b"], eps) * t[f"{p}.ls2"]
        if residuals is not None:
            residuals.append(x.clone())
    return layer_norm(x, t["final.norm"], t["final.norm.b"], eps) @ t["head"].T
