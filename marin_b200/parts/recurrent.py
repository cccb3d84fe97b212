"""Mixers whose memory is a fixed-size state per request instead of a cache that grows: a matrix per head that every
token updates (``StateNeed``), kept in float32 in the request's state slot.

Both walk the tokens a request brings to a step in order, from the state the steps before left (zeros at admission), so
a prompt may be cut anywhere and single decoded tokens take the same path.  Which tokens belong to which request and
which slot they use is read on the device (``ctx.cu_tokens``, ``cache.slots``): single-token steps may be captured.
"""
from __future__ import annotations

from typing import Dict, List, Optional, Sequence

import torch

from ..kernels import ops
from .base import Runtime, element_size
from .mixer import Mixer, StateNeed
from .registry import register_mixer
from .spec import TensorSpec


@register_mixer("linear_attention")
class LinearAttention(Mixer):
    """Linear attention with a fixed decay per head and an output gate.

    ``q = silu(W_q x)``, ``k = silu(W_k x)`` (``heads`` x ``dim``), ``v = silu(W_v x)`` (``heads`` x ``vdim``); per head
    ``S_t = decay_h S_(t-1) + k_t v_t^T`` and ``o_t = S_t^T q_t`` (no other scale).  The heads side by side are divided by
    their common root mean square (``norm_eps`` under the root), times the weight ``norm``, times ``sigmoid(W_g x)``, and go
    through ``W_o`` into the residual.  ``decay``: one number per head.
    """

    NAMES = {"q": "q", "k": "k", "v": "v", "g": "g", "o": "o", "norm": "norm"}

    def __init__(self, hidden: int, heads: int, dim: int, vdim: int, decay: Sequence[float], name: str, norm_eps: float = 1e-6,
                 names=None):
        self.hidden, self.heads, self.dim, self.vdim = int(hidden), int(heads), int(dim), int(vdim)
        self.decay_values = [float(d) for d in decay]
        if len(self.decay_values) != self.heads:
            raise ValueError(f"{len(self.decay_values)} decays for {self.heads} heads")
        self.name, self.norm_eps = name, float(norm_eps)
        self.names = dict(self.NAMES, **(names or {}))
        self.qk, self.hv = self.heads * self.dim, self.heads * self.vdim
        self.w_in = self.w_o = self.norm_w = self.decay = None

    def _n(self, key: str) -> str:
        return f"{self.name}.{self.names[key]}"

    def cache_need(self):
        return StateNeed((self.heads, self.dim, self.vdim), torch.float32)

    def tensor_specs(self) -> List[TensorSpec]:
        h = self.hidden
        return [TensorSpec(self._n("q"), (self.qk, h)), TensorSpec(self._n("k"), (self.qk, h)), TensorSpec(self._n("v"), (self.hv, h)),
                TensorSpec(self._n("g"), (self.hv, h)), TensorSpec(self._n("o"), (h, self.hv)), TensorSpec(self._n("norm"), (self.hv,), "norm")]

    def load(self, tensors: Dict[str, torch.Tensor], rt: Runtime) -> None:
        # one matrix for the four projections of x: q | k | v | g
        self.w_in = rt.matrix(torch.cat([tensors.pop(self._n(p)) for p in "qkvg"], dim=0))
        self.w_o = rt.matrix(tensors.pop(self._n("o")))
        self.norm_w = rt.f32(tensors.pop(self._n("norm")))
        self.decay = torch.tensor(self.decay_values, dtype=torch.float32, device=rt.device)
        self.rt = rt

    def flops(self, tokens: int, pairs: int = 0) -> float:
        return super().flops(tokens, pairs) + 4.0 * tokens * self.heads * self.dim * self.vdim

    def kernel_jobs(self, dtype) -> Dict[str, tuple]:
        return ops.linear_attention_jobs(dtype, self.dim, self.vdim)

    def forward(self, x, ctx, cache, residual: torch.Tensor):
        T = x.shape[0]
        ws = ctx.workspace
        qk, hv = self.qk, self.hv
        ops.stage_name = "q|k|v|g"
        proj = ws.get("lin_proj", (T, 2 * qk + 2 * hv), x.dtype)
        ops.gemm(x, self.w_in, proj)
        ops.stage_name = "recurrence"
        o = ws.get("lin_o", (T, hv), torch.float32)
        # prompt portions 64 tokens at a time on the tensor cores; single tokens (and sizes that kernel is not made for, and
        # the 32-bit path) token by token
        chunked = (ctx.max_query_len > 1 and ops.use_chunked_linear_attention
                   and ops.linear_attention_chunked_supported(x.dtype, self.dim, self.vdim))
        run = ops.linear_attention_chunked if chunked else ops.linear_attention_scan
        run(proj[:, :qk], proj[:, qk:2 * qk], proj[:, 2 * qk:2 * qk + hv], self.decay, cache.state, ctx, cache.slots, o,
            self.heads, self.dim, self.vdim)
        ops.stage_name = "norm, gate"
        gated = ws.get("lin_gated", (T, hv), x.dtype)
        ops.gated_rmsnorm(o, self.norm_w, proj[:, 2 * qk + hv:], "sigmoid", self.norm_eps, gated)
        ops.stage_name = "o"
        ops.gemm(gated, self.w_o, residual, accumulate=True)
        return None


@register_mixer("wkv")
class WKV(Mixer):
    """Time mixing with a decay that depends on the token (RWKV-style).

    With ``x'`` the row before in the sequence (zeros before the first token) each of r, k, v, g, w reads its own mix
    ``x + (x' - x) * mu_s``.  ``r, k, v = W_r, W_k, W_v`` of their mixes (``heads`` x ``dim``), ``gate = silu(W_g mix_g)``,
    ``decay = exp(-exp(W_w2 tanh(W_w1 mix_w) + w0))`` per head and key channel.  Per head
    ``o_t = (S_(t-1) + diag(u) k_t v_t^T)^T r_t`` (the bonus ``u`` for the current token only), then
    ``S_t = diag(decay_t) S_(t-1) + k_t v_t^T``.  Each head's ``o`` is divided by its root mean square (``norm_eps`` under the
    root); heads side by side, times ``norm``, times the gate, through ``W_o`` into the residual.  The state of a request is
    the matrices of all heads and the last row of ``x`` it has seen.
    """

    NAMES = {"r": "r", "k": "k", "v": "v", "g": "g", "o": "o", "w1": "w1", "w2": "w2", "w0": "w0", "u": "u", "norm": "norm",
             "mu": "mu"}
    MIXES = ("r", "k", "v", "g", "w")

    def __init__(self, hidden: int, heads: int, dim: int, decay_rank: int, name: str, norm_eps: float = 1e-6, names=None):
        self.hidden, self.heads, self.dim, self.rank = int(hidden), int(heads), int(dim), int(decay_rank)
        self.name, self.norm_eps = name, float(norm_eps)
        self.names = dict(self.NAMES, **(names or {}))
        self.n = self.heads * self.dim
        self.matrix_floats = self.heads * self.dim * self.dim

    def _n(self, key: str) -> str:
        return f"{self.name}.{self.names[key]}"

    def cache_need(self):
        return StateNeed((self.matrix_floats + self.hidden,), torch.float32)

    def tensor_specs(self) -> List[TensorSpec]:
        h, n = self.hidden, self.n
        specs = [TensorSpec(f"{self._n('mu')}.{s}", (h,), "bias") for s in self.MIXES]
        specs += [TensorSpec(self._n(p), (n, h)) for p in "rkvg"]
        specs += [TensorSpec(self._n("w1"), (self.rank, h)), TensorSpec(self._n("w2"), (n, self.rank)),
                  TensorSpec(self._n("w0"), (n,), "bias"), TensorSpec(self._n("u"), (self.heads, self.dim), "bias"),
                  TensorSpec(self._n("norm"), (n,), "norm"), TensorSpec(self._n("o"), (h, n))]
        return specs

    def load(self, tensors: Dict[str, torch.Tensor], rt: Runtime) -> None:
        self.mu = rt.f32(torch.stack([tensors.pop(f"{self._n('mu')}.{s}").to(torch.float32) for s in self.MIXES]))
        self.w_r, self.w_k, self.w_v, self.w_g = (rt.matrix(tensors.pop(self._n(p))) for p in "rkvg")
        self.w_1, self.w_2 = rt.matrix(tensors.pop(self._n("w1"))), rt.matrix(tensors.pop(self._n("w2")))
        self.w0 = rt.f32(tensors.pop(self._n("w0")))
        self.u = rt.f32(tensors.pop(self._n("u"))).reshape(-1)
        self.norm_w = rt.f32(tensors.pop(self._n("norm")))
        self.w_o = rt.matrix(tensors.pop(self._n("o")))
        self.rt = rt

    def flops(self, tokens: int, pairs: int = 0) -> float:
        return super().flops(tokens, pairs) + 6.0 * tokens * self.heads * self.dim * self.dim

    def kernel_jobs(self, dtype) -> Dict[str, tuple]:
        return ops.library_jobs("mb_activations", "mb_recurrent")

    def forward(self, x, ctx, cache, residual: torch.Tensor):
        T = x.shape[0]
        ws = ctx.workspace
        n = self.n
        state = cache.state[:, : self.matrix_floats]
        carry = cache.state[:, self.matrix_floats:]
        ops.stage_name = "token shift"
        mixes = ws.get("wkv_mixes", (len(self.MIXES), T, self.hidden), x.dtype)
        ops.shift_mix(x, carry, ctx, cache.slots, self.mu, mixes)
        ops.stage_name = "r, k, v, g"
        rkvg = ws.get("wkv_rkvg", (4, T, n), x.dtype)
        for i, w in enumerate((self.w_r, self.w_k, self.w_v, self.w_g)):
            ops.gemm(mixes[i], w, rkvg[i])
        ops.stage_name = "decay"
        low = ws.get("wkv_low", (T, self.rank), x.dtype)
        ops.gemm(mixes[4], self.w_1, low)
        ops.tanh_cap(low, 1.0)
        wraw = ws.get("wkv_wraw", (T, n), torch.float32)
        ops.gemm(low, self.w_2, wraw)
        ops.stage_name = "recurrence"
        o = ws.get("wkv_o", (T, n), torch.float32)
        ops.wkv_scan(rkvg[0], rkvg[1], rkvg[2], wraw, self.w0, self.u, state, carry, x, ctx, cache.slots, o, self.heads, self.dim)
        ops.stage_name = "norm, gate"
        out = ws.get("wkv_out", (T, n), x.dtype)
        ops.head_norm_gate(o, self.norm_w, rkvg[3], self.norm_eps, out, self.heads, self.dim)
        ops.stage_name = "o"
        ops.gemm(out, self.w_o, residual, accumulate=True)
        return None


@register_mixer("mamba2")
class Mamba2(Mixer):
    """A selective state space layer with one decay per head and token (Mamba-2: Dao, Gu, "Transformers are SSMs: Generalized
    Models and Efficient Algorithms Through Structured State Space Duality").

    With ``inner = heads * v_head_dim``, N = ``state`` and G = ``groups``, ``W_in h`` is laid out as ``z [inner] | x [inner] |
    B [G N] | C [G N] | dt [heads]``.  x, B and C together pass a causal convolution per channel of ``taps`` taps (weight
    ``[channels, taps]`` whose last column meets the current token, a bias) and silu.  ``dt <- softplus(dt + dt_bias)``; per
    head (head ``a`` uses group ``a // (heads / G)``): ``S_t = exp(-exp(rate_a) dt) S_(t-1) + dt B_t x_t^T`` (``N x v_head_dim``),
    ``y_t = S_t^T C_t + skip_a x_t``.  ``y`` (heads side by side) times ``silu(z)`` is divided by its root mean square in
    ``norm_groups`` equal parts (each by its own), times a weight, then ``W_o`` into the residual.  A request's state is the
    matrices of all heads (float32, zero at first) and the convolution's last ``taps - 1`` inputs: two slots' worth, kept as
    two needs."""

    NAMES = {"in": "in_proj", "conv": "conv", "conv_bias": "conv.bias", "dt_bias": "dt_bias", "rate": "A_log", "skip": "D", "norm": "norm",
             "o": "out_proj"}

    def __init__(self, hidden: int, heads: int, v_head_dim: int, state: int, groups: int, taps: int, name: str, norm_groups: int = 1,
                 norm_eps: float = 1e-6, names=None):
        self.hidden, self.heads, self.v_head_dim, self.state = int(hidden), int(heads), int(v_head_dim), int(state)
        self.groups, self.taps, self.norm_groups = int(groups), int(taps), int(norm_groups)
        self.name, self.norm_eps = name, float(norm_eps)
        if self.heads % self.groups != 0:
            raise ValueError(f"mamba2: {heads} heads cannot share {groups} groups evenly")
        self.inner = self.heads * self.v_head_dim
        if self.inner % self.norm_groups != 0:
            raise ValueError(f"mamba2: the norm's {norm_groups} parts do not divide {self.inner}")
        if self.state > 256 or self.taps > 64:
            raise ValueError("mamba2: a state above 256 rows or more than 64 taps is not supported")
        self.channels = self.inner + 2 * self.groups * self.state
        self.in_dim = 2 * self.inner + 2 * self.groups * self.state + self.heads
        self.names = dict(self.NAMES, **(names or {}))

    def _n(self, key: str) -> str:
        return f"{self.name}.{self.names[key]}"

    def cache_need(self):
        return (StateNeed((self.heads, self.state, self.v_head_dim), torch.float32),
                StateNeed((max(self.taps - 1, 1), self.channels), torch.float32))

    def tensor_specs(self) -> List[TensorSpec]:
        h = self.hidden
        return [TensorSpec(self._n("in"), (self.in_dim, h)), TensorSpec(self._n("conv"), (self.channels, self.taps), "bias", 1.0 / self.taps),
                TensorSpec(self._n("conv_bias"), (self.channels,), "bias"), TensorSpec(self._n("dt_bias"), (self.heads,), "bias"),
                TensorSpec(self._n("rate"), (self.heads,), "bias"), TensorSpec(self._n("skip"), (self.heads,), "bias", 1.0),
                TensorSpec(self._n("norm"), (self.inner,), "norm"), TensorSpec(self._n("o"), (h, self.inner))]

    def load(self, tensors: Dict[str, torch.Tensor], rt: Runtime) -> None:
        self.w_in = rt.matrix(tensors.pop(self._n("in")))
        self.conv_w, self.conv_b = rt.f32(tensors.pop(self._n("conv"))), rt.f32(tensors.pop(self._n("conv_bias")))
        self.dt_bias, self.rate, self.skip = (rt.f32(tensors.pop(self._n(k))) for k in ("dt_bias", "rate", "skip"))
        self.norm_w = rt.f32(tensors.pop(self._n("norm")))
        self.w_o = rt.matrix(tensors.pop(self._n("o")))
        self.rt = rt

    def flops(self, tokens: int, pairs: int = 0) -> float:
        return super().flops(tokens, pairs) + tokens * (6.0 * self.heads * self.state * self.v_head_dim + 2.0 * self.channels * self.taps)

    def kernel_jobs(self, dtype) -> Dict[str, tuple]:
        return ops.library_jobs("mb_ssm")

    def forward(self, x, ctx, cache, residual: torch.Tensor):
        T = x.shape[0]
        ws = ctx.workspace
        matrices, kept = cache
        ops.stage_name = "z|x|B|C|dt"
        rows = ws.get("ssm_rows", (T, self.in_dim), x.dtype)
        ops.gemm(x, self.w_in, rows)
        ops.stage_name = "convolution"
        xbc = ws.get("ssm_xbc", (T, self.channels), x.dtype)
        ops.ssm_conv(rows, self.inner, self.conv_w, self.conv_b, kept.state if self.taps > 1 else kept.state[:, :0], ctx, kept.slots, xbc)
        ops.stage_name = "recurrence"
        y = ws.get("ssm_y", (T, self.inner), torch.float32)
        ops.ssm_scan(xbc, rows, self.inner + self.channels, self.dt_bias, self.rate, self.skip, matrices.state, ctx, matrices.slots, y,
                     self.heads, self.v_head_dim, self.state, self.groups)
        ops.stage_name = "gate, norm"
        out = ws.get("ssm_out", (T, self.inner), x.dtype)
        ops.ssm_gate_norm(y, rows, 0, self.norm_w, self.norm_eps, self.norm_groups, out)
        ops.stage_name = "o"
        ops.gemm(out, self.w_o, residual, accumulate=True)
        return None


@register_mixer("delta_rule")
class DeltaRule(Mixer):
    """A gated delta rule (Yang, Kautz, Hatamizadeh, "Gated Delta Networks: Improving Mamba2 with Delta Rule").

    ``q = W_q x``, ``k = W_k x`` (``kv_heads`` x ``dim``), ``v = W_v x`` (``heads`` x ``vdim``; head ``h`` uses q/k head ``h // (heads /
    kv_heads)``), each through a causal convolution per channel of ``taps`` taps (weight ``[channels, taps]``, the last column on the current
    token) and silu; q and k divided by ``sqrt(sum of squares + 1e-6)`` per head, q also times ``dim^(-1/2)``.  Per head, with ``beta = sigmoid(W_b x)``:
    ``S <- g S``, ``u = beta (v - S^T k)``, ``S <- S + k u^T``, ``o = S^T q`` (``S`` ``dim`` x ``vdim``).

    ``decay`` "head": ``g = exp(-exp(A_log_h) softplus(W_a x + dt_bias))``, one per head; "channel": one per head and key channel (it multiplies
    that channel's row of ``S``), its argument out of two matrices, ``W_a2 (W_a1 x) + dt_bias`` with ``decay_rank`` numbers between.  Each head's ``o`` is
    divided by its root mean square over ``vdim`` (``norm_eps`` under the root), times a weight ``[vdim]``, times ``gate`` ("silu" or "sigmoid") of ``W_g
    x`` or, with ``gate_rank``, of ``W_g2 (W_g1 x)``; then ``out_scale`` and ``W_o`` into the residual.

    A request's state is the matrices of all heads (float32) and the convolution's latest inputs (a ring of ``taps`` rows): two needs."""

    NAMES = {"q": "q", "k": "k", "v": "v", "b": "b", "a": "a", "a1": "a1", "a2": "a2", "dt_bias": "dt_bias", "rate": "A_log", "g": "g", "g1": "g1",
             "g2": "g2", "norm": "norm", "o": "o", "q_conv": "q.conv", "k_conv": "k.conv", "v_conv": "v.conv"}

    def __init__(self, hidden: int, heads: int, kv_heads: int, dim: int, vdim: int, taps: int, name: str, decay: str = "head",
                 decay_rank: Optional[int] = None, gate: str = "silu", gate_rank: Optional[int] = None, norm_eps: float = 1e-6, names=None,
                 out_scale: float = 1.0):
        self.hidden, self.heads, self.kv_heads, self.dim, self.vdim, self.taps = (int(v) for v in (hidden, heads, kv_heads, dim, vdim, taps))
        self.name, self.decay, self.gate = name, decay, gate
        self.decay_rank, self.gate_rank = int(decay_rank) if decay_rank else None, int(gate_rank) if gate_rank else None
        self.norm_eps, self.out_scale = float(norm_eps), float(out_scale)
        if self.heads % self.kv_heads != 0:
            raise ValueError(f"delta_rule: {heads} heads cannot share {kv_heads} q/k heads evenly")
        if decay not in ("head", "channel") or gate not in ops.DELTA_GATES or (decay == "channel") != (self.decay_rank is not None):
            raise ValueError(f"delta_rule: decay {decay!r} (rank {decay_rank}) / gate {gate!r}")
        if self.dim > 256 or self.taps > 64:
            raise ValueError("delta_rule: key heads above 256 or more than 64 taps are not supported")
        self.names = dict(self.NAMES, **(names or {}))
        self.qk, self.hv = self.kv_heads * self.dim, self.heads * self.vdim
        self.channels = 2 * self.qk + self.hv
        self.decays = self.heads * self.dim if decay == "channel" else self.heads
        self.o_dim = self.hv
        self.w_in = self.w_low = self.w_high = self.w_o = None

    def _n(self, key: str) -> str:
        return f"{self.name}.{self.names[key]}"

    def cache_need(self):
        return (StateNeed((self.heads, self.dim, self.vdim), torch.float32), StateNeed((self.taps, self.channels), torch.float32))

    def tensor_specs(self) -> List[TensorSpec]:
        h, hv, n = self.hidden, self.hv, self.decays
        specs = []
        for p, rows in (("q", self.qk), ("k", self.qk), ("v", hv)):
            specs += [TensorSpec(self._n(p), (rows, h)), TensorSpec(self._n(f"{p}_conv"), (rows, self.taps), "bias", 1.0 / self.taps)]
        specs += [TensorSpec(self._n("b"), (self.heads, h)), TensorSpec(self._n("rate"), (self.heads,), "bias"),
                  TensorSpec(self._n("norm"), (self.vdim,), "norm"), TensorSpec(self._n("dt_bias"), (n,), "bias"), TensorSpec(self._n("o"), (h, hv))]
        for low, high, whole, rank, rows in (("a1", "a2", "a", self.decay_rank, n), ("g1", "g2", "g", self.gate_rank, hv)):
            specs += [TensorSpec(self._n(low), (rank, h)), TensorSpec(self._n(high), (rows, rank))] if rank else [TensorSpec(self._n(whole), (rows, h))]
        return specs

    def load(self, tensors: Dict[str, torch.Tensor], rt: Runtime) -> None:
        # One product of the layer's input: q | k | v, then whatever gates and decays come straight from it, then beta (blocks padded to
        # multiples of 8 columns, so that every kernel can take them by 16-byte loads).  Small products of two matrices: their first
        # matrices are one product, their second ones a block-diagonal one over its result.
        blocks: Dict[str, torch.Tensor] = {"qkv": torch.cat([tensors.pop(self._n(p)) for p in "qkv"], dim=0)}
        low: Dict[str, tuple] = {}
        for first, second, whole, rank in (("g1", "g2", "g", self.gate_rank), ("a1", "a2", "a", self.decay_rank)):
            if rank:
                low[whole] = (tensors.pop(self._n(first)), tensors.pop(self._n(second)))
            else:
                blocks[whole] = tensors.pop(self._n(whole))
        blocks["b"] = tensors.pop(self._n("b"))
        self.cols, at, rows = {}, 0, []
        for key, w in blocks.items():
            self.cols[key] = (at, w.shape[0])
            pad = -w.shape[0] % 8
            rows += [w] + ([torch.zeros(pad, w.shape[1], dtype=w.dtype, device=w.device)] if pad else [])
            at += w.shape[0] + pad
        self.w_in = rt.matrix(torch.cat(rows, dim=0))
        self.high_cols = {}
        if low:
            ranks = [-(-first.shape[0] // 8) * 8 for first, _ in low.values()]
            first_all = torch.zeros(sum(ranks), self.hidden, dtype=next(iter(low.values()))[0].dtype)
            second_all = torch.zeros(sum(second.shape[0] for _, second in low.values()), sum(ranks), dtype=first_all.dtype)
            r = c = 0
            for (whole, (first, second)), width in zip(low.items(), ranks):
                first_all[r:r + first.shape[0]] = first.cpu()
                second_all[c:c + second.shape[0], r:r + first.shape[0]] = second.cpu()
                self.high_cols[whole] = (c, second.shape[0])
                r, c = r + width, c + second.shape[0]
            self.w_low, self.w_high = rt.matrix(first_all), rt.matrix(second_all)
        self.conv_w = rt.f32(torch.cat([tensors.pop(self._n(f"{p}_conv")).to(torch.float32) for p in "qkv"], dim=0).t())     # [taps, channels]
        self.rate, self.dt_bias, self.norm_w = (rt.f32(tensors.pop(self._n(k))) for k in ("rate", "dt_bias", "norm"))
        self.w_o = rt.matrix(tensors.pop(self._n("o")))
        self.rt = rt

    def flops(self, tokens: int, pairs: int = 0) -> float:
        return super().flops(tokens, pairs) + tokens * (8.0 * self.heads * self.dim * self.vdim + 2.0 * self.channels * self.taps)

    def kernel_jobs(self, dtype) -> Dict[str, tuple]:
        return ops.delta_rule_jobs(dtype, self.dim, self.vdim)

    def workspace_per_token(self, dtype) -> int:
        """Bytes a step keeps per token beside the products' rows: the convolution's output, the heads' sums and, in chunks of 64 tokens,
        what the two chunked kernels hand over."""
        chunked = self.heads * ops.delta_chunk_bytes(self.dim, self.vdim) // 64 if ops.delta_chunked_supported(dtype, self.dim, self.vdim) else 0
        return self.channels * element_size(dtype) + 4 * self.hv + chunked

    joins_products = True

    def forward(self, x, ctx, cache, residual: torch.Tensor, rows=None, out=None):
        T = x.shape[0]
        ws = ctx.workspace
        H, G, d, dv = self.heads, self.kv_heads, self.dim, self.vdim
        matrices, ring = cache
        if rows is None:
            ops.stage_name = "q|k|v|b"
            rows = ws.get("delta_rows", (T, self.w_in.shape[0]), x.dtype)
            ops.gemm(x, self.w_in, rows)
        high = None
        if self.w_low is not None:
            ops.stage_name = "decay, gate"
            small = ws.get("delta_low", (T, self.w_low.shape[0]), x.dtype)
            ops.gemm(x, self.w_low, small)
            high = ws.get("delta_high", (T, self.w_high.shape[0]), x.dtype)
            ops.gemm(small, self.w_high, high)

        def block(key):
            src, (at, n) = (high, self.high_cols[key]) if key in self.high_cols else (rows, self.cols[key])
            return src[:, at:at + n]

        inputs = ops.DeltaInputs(block("b"), block("a"), block("g"), self.rate, self.dt_bias)
        qkv = block("qkv")
        joined = out is not None
        if not joined:
            out = ws.get("delta_out", (T, self.hv), x.dtype)
        ops.stage_name = "delta rule"
        single = ctx.num_decode if ops.use_delta_single and ops.delta_single_supported(d, dv) else 0
        if single:                                             # requests with one token each come first in the batch
            ops.delta_single(qkv, self.conv_w, ring.state, inputs, matrices.state, ctx, matrices.slots, self.gate, self.norm_w, self.norm_eps,
                             self.out_scale, out, single, H, G, d, dv)
        if ctx.num_requests > single:
            ops.stage_name = "convolution"
            conv = ws.get("delta_conv", (T, self.channels), x.dtype)
            ops.delta_conv(qkv, self.conv_w, ring.state, ctx, ring.slots, conv, single, single)
            ops.stage_name = "delta rule"
            o = ws.get("delta_o", (T, self.hv), torch.float32)
            if (ops.use_chunked_delta_rule and ops.delta_chunked_supported(x.dtype, d, dv) and self.channels % 8 == 0
                    and ctx.max_query_len > ops.DELTA_CHUNKED_FROM):
                ops.delta_chunked(conv, inputs, matrices.state, ctx, matrices.slots, o, H, G, d, dv, single, single)
            else:
                ops.delta_scan(conv, inputs, matrices.state, ctx, matrices.slots, o, H, G, d, dv, single)
            ops.stage_name = "norm, gate"
            ops.delta_norm(o, inputs.gate, self.gate, self.norm_w, self.norm_eps, self.out_scale, out, H, dv, single)
        if joined:
            return None
        ops.stage_name = "o"
        ops.gemm(out, self.w_o, residual, accumulate=True)
        return None


@register_mixer("gated_linear_attention")
class GatedLinearAttention(Mixer):
    """Gated linear attention (Yang, Wang, Shen, Panda, Kim, "Gated Linear Attention Transformers with Hardware-Efficient Training").

    ``q = W_q x dim^(-1/2)``, ``k = W_k x`` (``heads`` x ``dim``), ``v = W_v x`` (``heads`` x ``vdim``); per head
    ``S <- diag(alpha) S + k v^T``, ``o = S^T q`` (``S`` ``dim`` x ``vdim``, float32, zero at first) with a decay per key channel,
    ``alpha = sigmoid(z)^(1 / tau)``, ``z = W_a2 (W_a1 x) + bias`` (``decay_rank`` numbers between).  Each head's ``o`` is divided by its root mean square
    over ``vdim`` (``norm_eps`` under the root), times a weight ``[vdim]``, times ``gate`` ("silu" or "sigmoid") of ``W_g x``; then ``out_scale`` and ``W_o``
    into the residual."""

    NAMES = {"q": "q", "k": "k", "v": "v", "g": "g", "a1": "a1", "a2": "a2", "a_bias": "a2.b", "norm": "norm", "o": "o"}

    def __init__(self, hidden: int, heads: int, dim: int, vdim: int, tau: float, decay_rank: int, name: str, gate: str = "silu", norm_eps: float = 1e-6,
                 names=None, out_scale: float = 1.0):
        self.hidden, self.heads, self.dim, self.vdim, self.rank = (int(v) for v in (hidden, heads, dim, vdim, decay_rank))
        self.name, self.gate, self.tau, self.norm_eps, self.out_scale = name, gate, float(tau), float(norm_eps), float(out_scale)
        if gate not in ops.DELTA_GATES or not self.tau > 0:
            raise ValueError(f"gated_linear_attention: gate {gate!r}, tau {tau}")
        if self.dim > 256 or self.rank > 512:
            raise ValueError("gated_linear_attention: key heads above 256 or a decay rank above 512 are not supported")
        self.names = dict(self.NAMES, **(names or {}))
        self.qk, self.hv = self.heads * self.dim, self.heads * self.vdim
        self.o_dim = self.hv
        self.low_dim = self.rank + -self.rank % 16             # the decays' numbers between the matrices, padded with zeros
        self.w_in = self.w_2 = self.a_bias = self.norm_w = self.w_o = None

    def _n(self, key: str) -> str:
        return f"{self.name}.{self.names[key]}"

    def cache_need(self):
        return StateNeed((self.heads, self.dim, self.vdim), torch.float32)

    def tensor_specs(self) -> List[TensorSpec]:
        h = self.hidden
        return [TensorSpec(self._n("q"), (self.qk, h)), TensorSpec(self._n("k"), (self.qk, h)), TensorSpec(self._n("v"), (self.hv, h)),
                TensorSpec(self._n("g"), (self.hv, h)), TensorSpec(self._n("a1"), (self.rank, h)), TensorSpec(self._n("a2"), (self.qk, self.rank)),
                TensorSpec(self._n("a_bias"), (self.qk,), "bias"), TensorSpec(self._n("norm"), (self.vdim,), "norm"), TensorSpec(self._n("o"), (h, self.hv))]

    def load(self, tensors: Dict[str, torch.Tensor], rt: Runtime) -> None:
        # One product of the layer's input: q | k | v | g | what the decays are made of, in blocks padded to multiples of 8 columns (every kernel
        # can take them by 16-byte loads).  The decays' second matrix is applied inside the recurrence's kernels, in steps of 16 numbers.
        blocks = {p: tensors.pop(self._n(p)) for p in "qkvg"}
        first, second = tensors.pop(self._n("a1")), tensors.pop(self._n("a2"))
        pad = self.low_dim - self.rank
        blocks["low"] = torch.cat([first, first.new_zeros(pad, first.shape[1])], dim=0)
        self.w_2 = rt.matrix(torch.cat([second, second.new_zeros(second.shape[0], pad)], dim=1))
        self.cols, at, rows = {}, 0, []
        for key, w in blocks.items():
            self.cols[key] = (at, w.shape[0])
            rows += [w, w.new_zeros(-w.shape[0] % 8, w.shape[1])]
            at += w.shape[0] + -w.shape[0] % 8
        self.w_in = rt.matrix(torch.cat(rows, dim=0))
        self.a_bias, self.norm_w = rt.f32(tensors.pop(self._n("a_bias"))), rt.f32(tensors.pop(self._n("norm")))
        self.w_o = rt.matrix(tensors.pop(self._n("o")))
        self.rt = rt

    def flops(self, tokens: int, pairs: int = 0) -> float:
        return super().flops(tokens, pairs) + 4.0 * tokens * self.heads * self.dim * self.vdim

    def kernel_jobs(self, dtype) -> Dict[str, tuple]:
        return ops.gla_jobs(dtype, self.dim, self.vdim, self.low_dim)

    def workspace_per_token(self, dtype) -> int:
        """Bytes a step keeps per token beside the products' rows: the heads' sums, and what the chunked kernels hand over."""
        chunked = self.heads * ops.gla_chunk_bytes(self.dim, self.vdim) // 64 if ops.gla_chunked_supported(dtype, self.dim, self.vdim, self.low_dim) else 0
        return 4 * self.hv + chunked

    joins_products = True

    def forward(self, x, ctx, cache, residual: torch.Tensor, rows=None, out=None):
        T = x.shape[0]
        ws = ctx.workspace
        H, d, dv = self.heads, self.dim, self.vdim
        if rows is None:
            ops.stage_name = "q|k|v|g"
            rows = ws.get("gla_rows", (T, self.w_in.shape[0]), x.dtype)
            ops.gemm(x, self.w_in, rows)
        block = lambda key: rows[:, self.cols[key][0]:self.cols[key][0] + self.cols[key][1]]
        inputs = ops.GlaInputs(block("q"), block("k"), block("v"), block("g"), block("low"), self.w_2, self.a_bias, 1.0 / self.tau)
        joined = out is not None
        if not joined:
            out = ws.get("gla_out", (T, self.hv), x.dtype)
        ops.stage_name = "gated linear"
        single = ctx.num_decode if ops.use_gla_single and ops.gla_single_supported(d, dv) else 0
        if single:                                             # requests with one token each come first in the batch
            ops.gla_single(inputs, cache.state, ctx, cache.slots, self.gate, self.norm_w, self.norm_eps, self.out_scale, out, single, H, d, dv)
        if (ctx.num_requests > single and ops.use_chunked_gla and ops.gla_chunked_supported(x.dtype, d, dv, self.low_dim)
                and ctx.max_query_len > ops.GLA_CHUNKED_FROM):
            ops.gla_chunked(inputs, cache.state, ctx, cache.slots, self.gate, self.norm_w, self.norm_eps, self.out_scale, out, H, d, dv, single)
        elif ctx.num_requests > single:
            o = ws.get("gla_o", (T, self.hv), torch.float32)
            ops.gla_scan(inputs, cache.state, ctx, cache.slots, o, H, d, dv, single)
            ops.stage_name = "norm, gate"
            ops.delta_norm(o, inputs.gate, self.gate, self.norm_w, self.norm_eps, self.out_scale, out, H, dv, single)
        if joined:
            return None
        ops.stage_name = "o"
        ops.gemm(out, self.w_o, residual, accumulate=True)
        return None
