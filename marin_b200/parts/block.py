"""How a layer's parts are arranged around the residual stream."""
from __future__ import annotations

from typing import Dict, List

import torch

from ..kernels import ops
from .base import Part, Runtime, spec_bytes
from .registry import lookup, register_block
from .spec import LayerSpec, TensorSpec


@register_block("prenorm")
class PreNormBlock(Part):
    """``h += mixer(norm1(h)); h += feedforward(norm2(h))`` — the residual stream ``h`` stays
    float32 and both parts add into it (crates/model/src/qwen3/layer.rs:56-103).  A layer whose spec has no
    feed-forward has the first sublayer only (and no second norm)."""

    def __init__(self, spec: LayerSpec):
        names = spec.names
        norm_cls = lookup("norm", spec.norm.kind)
        self.norm1 = norm_cls(name=f"{spec.prefix}.{names['norm1']}", **spec.norm.params)
        self.mixer = lookup("mixer", spec.mixer.kind)(name=f"{spec.prefix}.{names['mixer']}", **spec.mixer.params)
        self.norm2 = self.feedforward = None
        if spec.feedforward is not None:
            self.norm2 = norm_cls(name=f"{spec.prefix}.{names['norm2']}", **spec.norm.params)
            self.feedforward = lookup("feedforward", spec.feedforward.kind)(
                name=f"{spec.prefix}.{names['feedforward']}", **spec.feedforward.params)

    def parts(self) -> List[Part]:
        return [p for p in (self.norm1, self.mixer, self.norm2, self.feedforward) if p is not None]

    def tensor_specs(self) -> List[TensorSpec]:
        return [s for p in self.parts() for s in p.tensor_specs()]

    def load(self, tensors: Dict[str, torch.Tensor], rt: Runtime) -> None:
        for p in self.parts():
            p.load(tensors, rt)
        self.rt = rt

    def weight_bytes(self, dtype) -> int:
        return sum(p.weight_bytes(dtype) for p in self.parts())

    def bytes_read(self, tokens: int, dtype) -> int:
        return sum(p.bytes_read(tokens, dtype) for p in self.parts())

    def flops(self, tokens: int, pairs: int = 0) -> float:
        return sum(p.flops(tokens, pairs) for p in self.parts())

    def kernel_jobs(self, dtype) -> Dict[str, tuple]:
        jobs: Dict[str, tuple] = {}
        for p in self.parts():
            jobs.update(p.kernel_jobs(dtype))
        return jobs

    #: ``forward`` takes ``x_in`` / ``next_block`` and returns the next block's input (see there)
    chains_norm = True

    def _rider(self, norm, producer, consumer, out):
        """``norm`` as a rider on ``producer``'s last product, if both parts around it can couple."""
        if getattr(producer, "couples_norm", False) and getattr(consumer, "couples_norm", False) and hasattr(norm, "coupling"):
            return norm.coupling(out)
        return None

    def forward(self, hidden: torch.Tensor, ctx, cache, x_in=None, next_block=None):
        """``x_in``: this block's first norm of ``hidden``, already there or carried by the block before (what that
        block returned).  ``next_block``: the block that runs next; if its first norm can ride on this block's last
        product, its input is returned, else None."""
        ws = ctx.workspace
        normed = ws.get("normed", tuple(hidden.shape), self.rt.dtype)
        if x_in is None:
            ops.stage_name = "norm"
        x = x_in if x_in is not None else self.norm1.forward(hidden, normed)
        if self.feedforward is None:
            rider = None
            if next_block is not None and getattr(next_block, "chains_norm", False):
                rider = self._rider(next_block.norm1, self.mixer, next_block.mixer, normed)
            if rider is not None:
                return self.mixer.forward(x, ctx, cache, hidden, then_norm=rider)
            self.mixer.forward(x, ctx, cache, hidden)
            return None
        rider = self._rider(self.norm2, self.mixer, self.feedforward, normed)
        x = self.mixer.forward(x, ctx, cache, hidden, then_norm=rider) if rider is not None else self.mixer.forward(x, ctx, cache, hidden)
        if x is None:
            ops.stage_name = "norm"
            x = self.norm2.forward(hidden, normed)
        rider = None
        if next_block is not None and getattr(next_block, "chains_norm", False):
            rider = self._rider(next_block.norm1, self.feedforward, next_block.mixer, normed)
        if rider is not None:
            return self.feedforward.forward(x, ctx, hidden, then_norm=rider)
        self.feedforward.forward(x, ctx, hidden)
        return None


@register_block("hyper_prenorm")
class HyperConnectionBlock(Part):
    """A pre-norm layer over ``streams`` copies ``x_1 .. x_S`` of the residual stream (hyper-connections: Zhu et al.,
    "Hyper-Connections").  Sublayer ``q`` (1: the mixer, 2: the feed-forward, where the layer has one) has learned numbers
    ``in[S]``, ``out[S]`` and ``mix[S, S]`` (indexed ``[from, to]``):

        u = sum_s in[s] x_s;   y = sublayer(norm_q(u));   x_t <- sum_s mix[s, t] x_s + out[t] y   (all streams at once).

    ``hidden`` is float32 ``[S, T, h]``.  The sublayers *add* into a float32 buffer ``y`` that the step before left zeroed,
    exactly as they add into the one residual stream of a plain block.  One kernel does a sublayer's write and the next
    sublayer's read and norm, across the border to the next block too when that is a block of this kind (``chains_norm``).
    ``block_params``: ``streams``; ``names``: ``hc1`` / ``hc2`` (the tensors' prefixes), ``in`` / ``out`` / ``mix``."""

    def __init__(self, spec: LayerSpec):
        names = spec.names
        self.streams = int(spec.block_params.get("streams", 1))
        if not 1 <= self.streams <= 8:
            raise ValueError(f"hyper_prenorm: {self.streams} streams (1 to 8)")
        norm_cls = lookup("norm", spec.norm.kind)
        self.norm1 = norm_cls(name=f"{spec.prefix}.{names['norm1']}", **spec.norm.params)
        self.mixer = lookup("mixer", spec.mixer.kind)(name=f"{spec.prefix}.{names['mixer']}", **spec.mixer.params)
        self.norm2 = self.feedforward = None
        if spec.feedforward is not None:
            self.norm2 = norm_cls(name=f"{spec.prefix}.{names['norm2']}", **spec.norm.params)
            self.feedforward = lookup("feedforward", spec.feedforward.kind)(
                name=f"{spec.prefix}.{names['feedforward']}", **spec.feedforward.params)
        for norm in (self.norm1, self.norm2):
            if norm is not None and not (hasattr(norm, "weight") and hasattr(norm, "eps") and hasattr(norm, "unit_offset")):
                raise ValueError("hyper_prenorm: the norm rides on the streams' kernel and has to be an RMS norm")
        self.hc_names = [f"{spec.prefix}.{names.get('hc1', 'hc1')}"] + ([f"{spec.prefix}.{names.get('hc2', 'hc2')}"] if self.feedforward else [])
        self.leaf = {k: names.get(k, k) for k in ("in", "out", "mix")}
        self.hc: List[Dict[str, torch.Tensor]] = []

    def parts(self) -> List[Part]:
        return [p for p in (self.norm1, self.mixer, self.norm2, self.feedforward) if p is not None]

    def _own_specs(self) -> List[TensorSpec]:
        S = self.streams
        out = []
        for n in self.hc_names:
            out += [TensorSpec(f"{n}.{self.leaf['in']}", (S,), "bias", 1.0 / S), TensorSpec(f"{n}.{self.leaf['out']}", (S,), "bias", 1.0),
                    TensorSpec(f"{n}.{self.leaf['mix']}", (S, S), "bias", 1.0 / S)]
        return out

    def tensor_specs(self) -> List[TensorSpec]:
        return [s for p in self.parts() for s in p.tensor_specs()] + self._own_specs()

    def load(self, tensors: Dict[str, torch.Tensor], rt: Runtime) -> None:
        for p in self.parts():
            p.load(tensors, rt)
        self.hc = [{k: rt.f32(tensors.pop(f"{n}.{self.leaf[k]}")) for k in ("in", "out", "mix")} for n in self.hc_names]
        self.rt = rt

    def weight_bytes(self, dtype) -> int:
        return sum(p.weight_bytes(dtype) for p in self.parts()) + sum(spec_bytes(s, dtype) for s in self._own_specs())

    def bytes_read(self, tokens: int, dtype) -> int:
        return sum(p.bytes_read(tokens, dtype) for p in self.parts())

    def flops(self, tokens: int, pairs: int = 0) -> float:
        return sum(p.flops(tokens, pairs) for p in self.parts())

    def kernel_jobs(self, dtype) -> Dict[str, tuple]:
        jobs: Dict[str, tuple] = dict(ops.library_jobs("mb_hyper"))
        for p in self.parts():
            jobs.update(p.kernel_jobs(dtype))
        return jobs

    chains_norm = True

    def _read(self, index: int, rows: torch.Tensor):
        norm = self.norm1 if index == 0 else self.norm2
        return (self.hc[index]["in"], norm.weight, norm.eps, norm.unit_offset, rows)

    def forward(self, hidden: torch.Tensor, ctx, cache, x_in=None, next_block=None):
        S, T, h = hidden.shape
        if S != self.streams:
            raise ValueError(f"hyper_prenorm: the model keeps {S} streams, the block was built for {self.streams}")
        ws = ctx.workspace
        normed = ws.get("normed", (T, h), self.rt.dtype)
        y = ws.get("sublayer_out", (T, h), torch.float32)
        if x_in is None:
            ops.stage_name = "streams, norm"
            ops.hc_step(hidden, y, read=self._read(0, normed))          # also leaves y zeroed
            x_in = normed
        self.mixer.forward(x_in, ctx, cache, y)
        last = 0
        if self.feedforward is not None:
            ops.stage_name = "streams, norm"
            ops.hc_step(hidden, y, write=(self.hc[0]["mix"], self.hc[0]["out"]), read=self._read(1, normed))
            self.feedforward.forward(normed, ctx, y)
            last = 1
        ops.stage_name = "streams, norm"
        write = (self.hc[last]["mix"], self.hc[last]["out"])
        if isinstance(next_block, HyperConnectionBlock) and next_block.streams == S:
            ops.hc_step(hidden, y, write=write, read=next_block._read(0, normed))
            return normed
        ops.hc_step(hidden, y, write=write)
        return None


@register_block("postnorm")
class PostNormBlock(Part):
    """``x <- x + s1 * norm1(mixer(x)); x <- x + s2 * norm2(feedforward(x))``: the norms are on the sublayers' outputs, the sublayers
    read the residual stream itself (in the activation dtype).  ``s1``, ``s2``: a learned vector per sublayer (layer scale: Touvron et al.,
    "Going deeper with Image Transformers"), named by ``block_params["layer_scale"]`` inside the prefix; absent: not scaled.  The norm is an RMS
    or layer norm part.

    The sublayers *add* into a float32 buffer ``y`` that the step before left zeroed, exactly as they add into the stream of a pre-norm
    block; one kernel then norms ``y``, scales it, adds it to the stream, zeroes ``y`` and leaves the stream's new rows in the activation
    dtype for the sublayer behind it, across the border to the next block too when that is a block of this kind (``chains_norm``)."""

    def __init__(self, spec: LayerSpec):
        names = spec.names
        norm_cls = lookup("norm", spec.norm.kind)
        self.norm1 = norm_cls(name=f"{spec.prefix}.{names['norm1']}", **spec.norm.params)
        self.mixer = lookup("mixer", spec.mixer.kind)(name=f"{spec.prefix}.{names['mixer']}", **spec.mixer.params)
        self.norm2 = self.feedforward = None
        if spec.feedforward is not None:
            self.norm2 = norm_cls(name=f"{spec.prefix}.{names['norm2']}", **spec.norm.params)
            self.feedforward = lookup("feedforward", spec.feedforward.kind)(
                name=f"{spec.prefix}.{names['feedforward']}", **spec.feedforward.params)
        for norm in (self.norm1, self.norm2):
            if norm is not None and (not hasattr(norm, "weight") or getattr(norm, "unit_offset", False)):
                raise ValueError("postnorm: the norm rides on the stream's update and has to be an RMS norm or a layer norm")
        scales = spec.block_params.get("layer_scale")
        self.hidden = int(spec.norm.params["dim"])
        self.scale_names = [f"{spec.prefix}.{s}" for s in scales][: 2 if self.feedforward is not None else 1] if scales else []
        self.scales: List[torch.Tensor] = []

    def parts(self) -> List[Part]:
        return [p for p in (self.norm1, self.mixer, self.norm2, self.feedforward) if p is not None]

    def _own_specs(self) -> List[TensorSpec]:
        return [TensorSpec(n, (self.hidden,), "norm") for n in self.scale_names]

    def tensor_specs(self) -> List[TensorSpec]:
        return [s for p in self.parts() for s in p.tensor_specs()] + self._own_specs()

    def load(self, tensors: Dict[str, torch.Tensor], rt: Runtime) -> None:
        for p in self.parts():
            p.load(tensors, rt)
        self.scales = [rt.f32(tensors.pop(n)) for n in self.scale_names]
        self.rt = rt

    def weight_bytes(self, dtype) -> int:
        return sum(p.weight_bytes(dtype) for p in self.parts()) + sum(spec_bytes(s, dtype) for s in self._own_specs())

    def bytes_read(self, tokens: int, dtype) -> int:
        return sum(p.bytes_read(tokens, dtype) for p in self.parts()) + sum(spec_bytes(s, dtype) for s in self._own_specs())

    def flops(self, tokens: int, pairs: int = 0) -> float:
        return sum(p.flops(tokens, pairs) for p in self.parts())

    def kernel_jobs(self, dtype) -> Dict[str, tuple]:
        jobs: Dict[str, tuple] = dict(ops.library_jobs("mb_layer_norm"))
        for p in self.parts():
            jobs.update(p.kernel_jobs(dtype))
        return jobs

    chains_norm = True

    def _join(self, index: int, y: torch.Tensor, hidden: torch.Tensor, rows) -> None:
        norm = self.norm1 if index == 0 else self.norm2
        ops.stage_name = "norm into the stream"
        ops.norm_into(y, getattr(norm, "kind", "rms"), norm.weight, getattr(norm, "bias", None), norm.eps,
                      self.scales[index] if self.scales else None, hidden, rows)

    def forward(self, hidden: torch.Tensor, ctx, cache, x_in=None, next_block=None):
        ws = ctx.workspace
        wide = self.rt.dtype == torch.float32                  # the stream's own rows serve as they are
        rows = hidden if wide else ws.get("stream_rows", tuple(hidden.shape), self.rt.dtype)
        y = ws.get("sublayer_out", tuple(hidden.shape), torch.float32)
        if x_in is None:                                       # (a block of this kind leaves rows and a zeroed y behind)
            ops.stage_name = "stream rows"
            ops.stream_rows(hidden, None if wide else rows, y)
        self.mixer.forward(rows, ctx, cache, y)
        goes_on = isinstance(next_block, PostNormBlock)
        if self.feedforward is not None:
            self._join(0, y, hidden, None if wide else rows)
            self.feedforward.forward(rows, ctx, y)
            self._join(1, y, hidden, rows if goes_on and not wide else None)
        else:
            self._join(0, y, hidden, rows if goes_on and not wide else None)
        return rows if goes_on else None


@register_block("parallel_prenorm")
class ParallelBlock(Part):
    """``x <- x + m (mixer(h) + feedforward(h))`` with one norm, ``h = norm1(x)``, that both sublayers read (a layer without a feed-forward has the mixer
    alone).  ``block_params["residual_mult"]``: ``m`` (1 without it); mixer and feed-forward take it as their ``out_scale``, so that it multiplies
    float32 numbers before they are rounded.  A row the mixer adds to every token (``Mixer.row_bias``) rides on the norm's kernel.

    In bfloat16, where both sublayers allow it (``joins_products``), what they take from ``h`` is one product, the feed-forward's activation applied to
    its columns in the epilogue, and what they add to the stream is one product of their results side by side."""

    #: False: the sublayers' products stay their own (the twin the joined ones are compared with); read when a model is loaded
    join_products = True

    def __init__(self, spec: LayerSpec):
        names = spec.names
        m = float(spec.block_params.get("residual_mult", 1.0))
        scale = {} if m == 1.0 else {"out_scale": m}
        self.norm1 = lookup("norm", spec.norm.kind)(name=f"{spec.prefix}.{names['norm1']}", **spec.norm.params)
        if not (hasattr(self.norm1, "weight") and hasattr(self.norm1, "unit_offset")):
            raise ValueError("parallel_prenorm: the norm has to be an RMS norm")
        self.mixer = lookup("mixer", spec.mixer.kind)(name=f"{spec.prefix}.{names['mixer']}", **{**spec.mixer.params, **scale})
        self.feedforward = None
        if spec.feedforward is not None:
            self.feedforward = lookup("feedforward", spec.feedforward.kind)(name=f"{spec.prefix}.{names['feedforward']}", **{**spec.feedforward.params, **scale})

    def parts(self) -> List[Part]:
        return [p for p in (self.norm1, self.mixer, self.feedforward) if p is not None]

    def tensor_specs(self) -> List[TensorSpec]:
        return [s for p in self.parts() for s in p.tensor_specs()]

    def load(self, tensors: Dict[str, torch.Tensor], rt: Runtime) -> None:
        for p in self.parts():
            p.load(tensors, rt)
        self.mixer.adds_row_bias = False
        self.w_in = self.w_last = None
        mixer, ff = self.mixer, self.feedforward
        if (self.join_products and rt.dtype == torch.bfloat16 and mixer.joins_products and ff is not None and getattr(ff, "joins_products", False)
                and mixer.o_dim % 8 == 0 and mixer.w_in.shape[1] % 8 == 0):
            n = mixer.w_in.shape[0]
            self.plain = n + -n % 32                           # the mixer's rows, in whole steps of the epilogue's warps
            self.w_in = torch.cat([mixer.w_in, mixer.w_in.new_zeros(self.plain - n, mixer.w_in.shape[1]), ff.w_gate_up], dim=0).contiguous()
            self.w_last = torch.cat([mixer.w_o, ff.w_down], dim=1).contiguous()
            mixer.lend_products(self.w_in[:n])
            ff.w_gate_up, ff.w_down = self.w_in[self.plain:], None
        self.rt = rt

    def weight_bytes(self, dtype) -> int:
        return sum(p.weight_bytes(dtype) for p in self.parts())

    def bytes_read(self, tokens: int, dtype) -> int:
        return sum(p.bytes_read(tokens, dtype) for p in self.parts())

    def flops(self, tokens: int, pairs: int = 0) -> float:
        return sum(p.flops(tokens, pairs) for p in self.parts())

    def kernel_jobs(self, dtype) -> Dict[str, tuple]:
        jobs: Dict[str, tuple] = {}
        for p in self.parts():
            jobs.update(p.kernel_jobs(dtype))
        return jobs

    def forward(self, hidden: torch.Tensor, ctx, cache):
        ops.stage_name = "norm"
        x = self.norm1.forward(hidden, ctx.workspace.get("normed", tuple(hidden.shape), self.rt.dtype), self.mixer.row_bias)
        if self.w_in is not None:
            T, n, ff = hidden.shape[0], self.mixer.o_dim, self.feedforward
            ops.stage_name = "inputs, gate|up"
            rows = ctx.workspace.get("layer_rows", (T, self.plain), x.dtype)
            outs = ctx.workspace.get("layer_outs", (T, self.w_last.shape[1]), x.dtype)
            ops.gemm_glu_rows(x, self.w_in, rows, outs[:, n:], ff.activation, ff.out_scale)
            self.mixer.forward(x, ctx, cache, hidden, rows=rows[:, :self.mixer.w_in.shape[0]], out=outs[:, :n])
            ops.stage_name = "o|down"
            ops.gemm(outs, self.w_last, hidden, accumulate=True)
            return
        self.mixer.forward(x, ctx, cache, hidden)
        if self.feedforward is not None:
            self.feedforward.forward(x, ctx, hidden)
