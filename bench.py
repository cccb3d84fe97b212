#!/usr/bin/env python3
"""Decode and prefill throughput of the engine on one B200, with their fractions of roofline.

    python bench.py [--gpus 1] [--steps K] [--warmup W] [--batch 8] [--layers N] [--impl ours|reference]
    python bench.py --arch lakulix|fegarax|nirotar|vogunex|pununex|punolix [--model 4b|8b|14b] [--layers 12] [--batch 8] [--profile]

The default run has the layer sizes of the Qwen3-4B layout with random bfloat16 weights, a batch of 8
sequences and a context of 4096 positions (the last timed step reaches it).  A "step" is one decode
step.  One JSON line is printed:

  value      decoded tokens a second, K steps timed on the device with CUDA events
  e2e        the same through the Python entry point (Engine.step): every step the host packs and sends the next
             step's inputs from pinned memory and reads the sampled ids back (the step after the running one is
             launched before those ids have arrived: its token ids are fed on the device)
  prefill    one 2,048-token prompt in one step: tokens a second and the fraction of the bf16 peak
  roofline   bytes a decode step has to read (every weight once, the cache of the live requests) / its time
  points     decode at batch 1 and 64

``--arch lakulix`` measures another architecture instead, beside the Qwen3 layout of the same width, depth and vocabulary:
Lakulix layers (linear attention, sigmoid attention, time mixing, in turn; a PolyNorm feed-forward in each) at the chosen
layout's sizes, decode at the given batch and the prompt step, each with its fraction of roofline, as one JSON line of
its own form (``--profile``: its stage tables).  ``--arch fegarax`` does the same for Fegarax layers (four residual streams,
attention with the layout's heads, a gate and a sink, eight experts of half the feed-forward width of which two are chosen).
``--arch nirotar`` measures Nirotar layers (windowed attention with a learned sink and attention over a shared latent in turn,
experts without a gate chosen by a table over the token ids, a shared expert) beside the Fegarax layout of the same width,
depth, vocabulary and heads, the closest of the engine's models (attention with a sink, routed experts).
``--arch vogunex`` measures Vogunex layers (attention over a window and pooled blocks with mixed head weights, a state space
layer, attention over a shared latent with a window, in turn; dense and routed feed-forwards; a token shift before every
mixer) beside the Nirotar layers at the same sizes, the closest of the engine's models.
``--arch pununex`` measures Pununex layers (windowed attention with kept first positions beside a gated delta rule, and a delta
rule alone, in turn; dense and routed feed-forwards, norms on the sublayers' outputs) beside the Vogunex layers at the same sizes.
``--arch punolix`` measures Punolix layers (differential attention, and chunked attention behind short convolutions beside gated linear
attention, in turn; a dense feed-forward on the mixer's own norm in each) beside the Pununex layers at the same sizes.
The default workload and its line are not touched by any of them.

Peaks come from MEASURED_PEAKS.json beside this file if present, else 6.65 TB/s and 1.59 PFLOP/s.
Between timed iterations nothing is flushed: a decode step reads gigabytes of weights, far more than the
126 MB L2 holds (config.l2 says so).
"""
import argparse
import json
import os
import statistics
import subprocess
import sys
import threading
import time

ROOT = os.path.dirname(os.path.abspath(__file__))
sys.path.insert(0, ROOT)

QWEN3_4B = {
    "architectures": ["Qwen3ForCausalLM"], "model_type": "qwen3", "num_hidden_layers": 36, "hidden_size": 2560,
    "num_attention_heads": 32, "num_key_value_heads": 8, "head_dim": 128, "intermediate_size": 9728,
    "vocab_size": 151936, "rope_theta": 1000000.0, "rms_norm_eps": 1e-6, "tie_word_embeddings": True,
    "max_position_embeddings": 40960,
}
QWEN3_8B = dict(QWEN3_4B, hidden_size=4096, intermediate_size=12288, tie_word_embeddings=False)
QWEN3_14B = dict(QWEN3_4B, num_hidden_layers=40, hidden_size=5120, num_attention_heads=40, intermediate_size=17408,
                 tie_word_embeddings=False)
LAYOUTS = {"4b": QWEN3_4B, "8b": QWEN3_8B, "14b": QWEN3_14B}
CONTEXT = 4096
PREFILL_TOKENS = 2048
PAGE = 16
PUBLISHED = None     # the reference published no number for this metric on this configuration


def peaks():
    path = os.path.join(ROOT, "MEASURED_PEAKS.json")
    if os.path.exists(path):
        with open(path) as fh:
            p = json.load(fh)
        return {"hbm_gbs": p["hbm_gbs"], "bf16_tflops": p["bf16_tflops"],
                "bf16_tflops_sustained": p.get("bf16_tflops_sustained", p["bf16_tflops"]), "source": "measured"}
    return {"hbm_gbs": 6650.0, "bf16_tflops": 1590.0, "bf16_tflops_sustained": 1400.0, "source": "fallback"}


class ClockSampler:
    """Samples nvidia-smi clocks and throttle reasons while the timed region runs (reads only)."""

    QUERY = ("clocks.sm,clocks.max.sm,power.draw,clocks_event_reasons.hw_slowdown,clocks_event_reasons.hw_thermal_slowdown,"
             "clocks_event_reasons.sw_thermal_slowdown,clocks_event_reasons.sw_power_cap")

    def __init__(self, gpu="0"):
        self.rows, self.proc, self.gpu = [], None, str(gpu)

    @staticmethod
    def gpu_in_use():
        """What nvidia-smi should be asked about: the device this process computes on (its UUID), not index 0 of the
        box, which may be another job's GPU."""
        import torch

        try:
            uuid = str(torch.cuda.get_device_properties(torch.cuda.current_device()).uuid)
            return uuid if uuid.startswith("GPU-") else "GPU-" + uuid
        except Exception:  # noqa: BLE001 - an older torch without the field: the first visible device
            visible = os.environ.get("CUDA_VISIBLE_DEVICES", "").split(",")[0].strip()
            return visible or "0"

    def start(self):
        try:
            self.proc = subprocess.Popen(["nvidia-smi", "-i", self.gpu, f"--query-gpu={self.QUERY}", "--format=csv,noheader,nounits",
                                          "-lms", "50"], stdout=subprocess.PIPE, stderr=subprocess.DEVNULL, text=True)
            threading.Thread(target=self._read, daemon=True).start()
        except OSError:
            self.proc = None

    def _read(self):
        for line in self.proc.stdout:
            self.rows.append([c.strip() for c in line.split(",")])

    def stop(self):
        if self.proc is not None:
            self.proc.terminate()
            try:
                self.proc.wait(timeout=5)
            except subprocess.TimeoutExpired:
                self.proc.kill()
        sm, reasons, smax = [], set(), None
        for r in self.rows:
            try:
                sm.append(float(r[0]))
                smax = float(r[1])
            except (ValueError, IndexError):
                continue
            for name, v in zip(["hw_slowdown", "hw_thermal_slowdown", "sw_thermal_slowdown", "sw_power_cap"], r[3:7]):
                if v == "Active":
                    reasons.add(name)
        busy = [c for c in sm if smax and c > 0.5 * smax] or sm
        return {"sm_mhz": statistics.median(busy) if busy else None, "sm_max_mhz": smax, "reasons": sorted(reasons),
                "samples": len(sm), "samples_under_load": len(busy), "gpu": self.gpu}


def model_bytes_and_flops(engine, batch, tokens):
    """Bytes of weights a decode step of `batch` tokens reads (what the model's parts say they read), and the flops
    of a `tokens`-long prompt with one row of logits (causal: every token looks at itself and what came before)."""
    dtype = engine.rt.dtype
    pairs = tokens * (tokens + 1) // 2
    return engine.model.bytes_read(batch, dtype), engine.model.flops(tokens, pairs, 1)


def kv_bytes_per_token(engine):
    """Bytes one cached position holds over all layers (what a decoded token reads per position of its sequence)."""
    return engine.model.cache_bytes_read(1, engine.rt.dtype)


def fill_cache(engine, seed=1):
    import torch

    g = torch.Generator(device=engine.rt.device).manual_seed(seed)
    for group in engine.cache.groups:
        for t in (group.k, group.v) + ((group.k_pool, group.v_pool) if group.k_pool is not None else ()):
            flat = t.view(-1)
            step = 1 << 28
            for at in range(0, flat.numel(), step):
                n = min(step, flat.numel() - at)
                flat[at:at + n] = (torch.randn(n, device=t.device, generator=g, dtype=torch.float32) * 0.5).to(t.dtype)


def decode_device(engine, batch, steps, warmup, context):
    """K decode steps of `batch` sequences timed on the device; the last step reaches `context`."""
    import torch

    from marin_b200.engine import StepEntry
    from marin_b200.kernels import ops

    runner = engine.runner
    start_len = context - (steps + warmup)
    ids = [f"bench{i}" for i in range(batch)]
    for rid in ids:
        runner.begin(rid)
        engine.cache.reserve(rid, start_len)
        engine.cache.commit(rid, start_len)
    vocab = engine.config.vocab_size
    tokens = torch.randint(0, vocab, (batch,), dtype=torch.int32).tolist()
    out = runner.scratch.ids(batch)

    def one_step(tokens):
        logits = runner.step([StepEntry(rid, [tok], [0]) for rid, tok in zip(ids, tokens)])
        if runner.greedy_ids is None:                       # a replayed graph has found the largest logits already
            with ops.using(runner.scratch):
                ops.argmax(logits, vocab, out)

    for _ in range(warmup):
        one_step(tokens)
    torch.cuda.synchronize()
    begin, end = torch.cuda.Event(enable_timing=True), torch.cuda.Event(enable_timing=True)
    launches = ops.launches
    begin.record()
    for _ in range(steps):
        one_step(tokens)
    end.record()
    torch.cuda.synchronize()
    ms = begin.elapsed_time(end)
    launched = ops.launches - launches
    for rid in ids:
        runner.end(rid)
    mean_context = context - (steps - 1) / 2.0
    return {"tok_s": batch * steps / (ms / 1e3), "ms_per_step": ms / steps, "launches": launched,
            "mean_context": mean_context}


def decode_e2e(engine, batch, steps, warmup, context):
    """The same through Engine.add_request / Engine.step: host token ids in, sampled ids out, every step."""
    import torch

    from marin_b200 import SamplingParams

    vocab = engine.config.vocab_size
    # the prompts are read in portions under the token budget, one request after another, while the requests
    # that are through already decode: leave room for those tokens so that the timed steps end near `context`
    prefill_steps = -(-batch * context // engine.token_budget) + batch
    prompt_len = context - (steps + warmup) - prefill_steps - 2
    g = torch.Generator().manual_seed(3)
    params = SamplingParams(temperature=0.0, max_tokens=context)
    ids = [engine.add_request(torch.randint(0, vocab, (prompt_len,), generator=g).tolist(), params) for _ in range(batch)]
    produced = {i: 0 for i in ids}
    while min(produced.values()) < 1:                       # prompts (untimed)
        for rid, _ in engine.step():
            produced[rid] += 1
    for _ in range(warmup):
        engine.step()
    torch.cuda.synchronize()
    t0 = time.perf_counter()
    got = 0
    for _ in range(steps):
        got += len(engine.step())                           # sampled ids are host ints here
    torch.cuda.synchronize()
    seconds = time.perf_counter() - t0
    for i in ids:
        engine.scheduler.cancel(i)
        engine.forget(i)
    # per step the host sends the packed inputs of the next step without its token ids (those are fed on the device:
    # the step is launched before the host has read the ids of the one before) and reads, from pinned memory that the
    # arg-max kernel writes itself, four ints of status and the sampled ids
    bucket = next(b for b in engine.runner.graph_sizes if b >= batch)
    h2d = 4 * (engine.runner.packed_size(bucket) + 1 - bucket)
    return {"value": got / seconds, "unit": "tokens/s", "h2d_bytes_per_step": h2d, "d2h_bytes_per_step": 4 * (4 + batch),
            "tokens": got}


def prefill_device(engine, tokens, runs, warmup):
    import torch

    from marin_b200.engine import StepEntry

    runner = engine.runner
    vocab = engine.config.vocab_size
    prompt = torch.randint(0, vocab, (tokens,), generator=torch.Generator().manual_seed(5)).tolist()
    times = []
    for i in range(warmup + runs):
        runner.begin("prefill")
        torch.cuda.synchronize()
        begin, end = torch.cuda.Event(enable_timing=True), torch.cuda.Event(enable_timing=True)
        begin.record()
        runner.step([StepEntry("prefill", prompt, [tokens - 1])])
        end.record()
        torch.cuda.synchronize()
        if i >= warmup:
            times.append(begin.elapsed_time(end))
        runner.end("prefill")
    return statistics.median(times)


def profile_mode(engine, args, pk, label=None, batches=None):
    """Where the time of a decode step (batch 1, 8 and 64) and of a 2,048-token prompt goes, stage by stage
    (marin_b200/engine/profile.py).  Text to stdout; no JSON line: nothing measured here is a throughput figure."""
    import torch

    from marin_b200.engine import StepEntry
    from marin_b200.engine.profile import format_table, profile_steps
    from marin_b200.kernels import ops

    runner, vocab = engine.runner, engine.config.vocab_size
    layers = len(engine.model.blocks)
    where = f"Qwen3-{args.model.upper()} layout, {layers} of {LAYOUTS[args.model]['num_hidden_layers']} layers, bfloat16, page {PAGE}"
    if label is not None:
        where = f"{label}, bfloat16, page {PAGE}"
    peaks_line = f"peaks ({pk['source']}): {pk['hbm_gbs']:.0f} GB/s copy, {pk['bf16_tflops']:.0f} TFLOP/s bf16"
    print(f"{where}; {peaks_line}; in-step times under the CUDA profiling interface (medians of 6 steps)\n")
    steps, warmup = 6, 4
    for batch in sorted(set(batches) if batches else {1, 8, 64, args.batch}):
        ids = [f"prof{batch}_{i}" for i in range(batch)]
        for rid in ids:
            runner.begin(rid)
            engine.cache.reserve(rid, CONTEXT - steps - warmup)
            engine.cache.commit(rid, CONTEXT - steps - warmup)
        # (token ids that differ between the requests: a model that chooses experts by the token id should not send them all to the same ones)
        rows = profile_steps(runner, lambda i: [StepEntry(rid, [(5 + i + 7919 * k) % vocab], [0]) for k, rid in enumerate(ids)], steps, warmup)
        print(format_table(rows, pk["hbm_gbs"], pk["bf16_tflops"], f"decode step, batch {batch}, sequences of about {CONTEXT} positions"))
        print()
        for rid in ids:
            runner.end(rid)
    prompt = torch.randint(0, vocab, (PREFILL_TOKENS,), generator=torch.Generator().manual_seed(5)).tolist()
    out = runner.scratch.ids(1)

    def entries(i):
        runner.begin(f"prefill{i}")
        return [StepEntry(f"prefill{i}", prompt, [PREFILL_TOKENS - 1])]

    def after(logits):
        ops.stage_name = "sampling"
        ops.argmax(logits, vocab, out)
        runner.end(next(iter(runner.cache.requests)))

    rows = profile_steps(runner, entries, steps, warmup, after_step=after)
    print(format_table(rows, pk["hbm_gbs"], pk["bf16_tflops"], f"prompt of {PREFILL_TOKENS} tokens in one step"))
    engine.check_device()
    return 0


def lakulix_layout(raw: dict, layers: int) -> dict:
    """A Lakulix configuration at a Qwen3 layout's sizes: the same width, feed-forward width, vocabulary and attention
    heads; linear-attention heads of 128 x 128 and time-mixing heads of 64 filling the width; the three mixers in turn."""
    width, head = raw["hidden_size"], raw["head_dim"]
    lin_heads = width // 128
    mixers = [
        {"type": "lightning", "mixer": {"heads": lin_heads, "dim": 128, "vdim": 128,
                                        "decay": [1.0 - 2.0 ** (-(3 + 5 * i / max(1, lin_heads - 1))) for i in range(lin_heads)]}},
        {"type": "attention", "mixer": {"heads": raw["num_attention_heads"], "kv_heads": raw["num_key_value_heads"], "dim": head,
                                        "vdim": head, "scale": head ** -0.5, "bias_max": 240, "bias_rows": 32,
                                        "q_temp": {"coef": 0.1, "every": 1024}}},
        {"type": "wkv", "mixer": {"heads": width // 64, "dim": 64, "decay_rank": 64}},
    ]
    return {"architecture": "Lakulix", "vocab": raw["vocab_size"], "width": width, "max_positions": 2 * CONTEXT,
            "norm": {"eps": 1e-6}, "logit_softcap": 30.0,
            "layers": [dict(mixers[i % 3], mlp={"kind": "dense", "ff": raw["intermediate_size"]}) for i in range(layers)]}


FEGARAX_LAYERS = ("four residual streams; attention with the layout's heads (values as wide as keys, rotation of half of every head with "
                  "rescaled frequencies, chunks of 8,192 positions: every earlier key is seen at this context, as in the Qwen3 arm), "
                  "a gate, a sink, values mixed with the first layer's; 8 experts of half the layout's feed-forward width, 2 chosen "
                  "(as many active feed-forward weights as the dense layout, four times as many in memory)")


def fegarax_layout(raw: dict, layers: int) -> dict:
    """A Fegarax configuration at a Qwen3 layout's sizes: the same width, vocabulary and attention heads; experts that
    together activate as many feed-forward weights per token as the layout's dense feed-forward."""
    head = raw["head_dim"]
    mixer = {"heads": raw["num_attention_heads"], "kv_heads": raw["num_key_value_heads"], "dim": head, "vdim": head, "scale": head ** -0.5,
             "mask": {"size": 2 * CONTEXT}, "v_mix": True,
             "rot": {"base": 1000000.0, "dims": head // 2, "scaling": {"factor": 4.0, "original": 2048, "fast": 16.0, "slow": 2.0}}}
    mlp = {"kind": "moe", "expert": {"ff": raw["intermediate_size"] // 2}, "router": {"experts": 8, "top": 2}}
    return {"architecture": "Fegarax", "vocab": raw["vocab_size"], "width": raw["hidden_size"], "streams": 4, "embedding": {"scale": 1.0},
            "norm": {"eps": 1e-6}, "max_positions": 2 * CONTEXT, "layers": [{"type": "attention", "mixer": mixer, "mlp": mlp} for _ in range(layers)]}


NIROTAR_LAYERS = ("in turn: attention with the layout's heads (a window of 1,024 positions, neighbouring pairs rotated over half of every "
                  "head with band-scaled frequencies, a learned sink); attention over a shared latent (as many heads, 64 unrotated + 32 "
                  "rotated query numbers, values of 64, page rows of 128 + 32 numbers, a learned sink); attention again; latent attention "
                  "that reads the rows of the latent layer two before it.  8 experts without a gate (squared relu) of 5/8 of the layout's "
                  "feed-forward width, 2 chosen by a table over the token ids, and a shared expert: as many active feed-forward weights "
                  "per token as the Fegarax and the dense layouts")


def nirotar_layout(raw: dict, layers: int) -> dict:
    """A Nirotar configuration at a Qwen3 layout's sizes: the same width, vocabulary and attention heads; experts and a
    shared expert that together activate as many feed-forward weights per token as the layout's dense feed-forward."""
    head, heads = raw["head_dim"], raw["num_attention_heads"]
    attention = {"heads": heads, "kv_heads": raw["num_key_value_heads"], "dim": head, "vdim": head, "scale": head ** -0.5,
                 "mask": {"size": 1024},
                 "rot": {"base": 500000.0, "dims": head // 2, "scaling": {"factor": 8.0, "low": 1.0, "high": 4.0, "original": 2048}}}
    latent = {"heads": heads, "dim": 64, "rot_dim": 32, "vdim": 64, "kv_rank": 128, "scale": 96 ** -0.5, "rot": {"base": 500000.0, "dims": 32}}
    half = raw["intermediate_size"] // 2
    expert = half * 5 // 4 // 64 * 64
    shared = (6 * half - 4 * expert) // 2 // 64 * 64
    mlp = {"kind": "moe", "expert": {"ff": expert}, "router": {"experts": 8, "top": 2}, "shared": {"ff": shared}}
    out = []
    for i in range(layers):
        if i % 2 == 0:
            out.append({"type": "attention", "mixer": attention, "mlp": mlp})
        else:
            out.append({"type": "latent_attention", "mixer": dict(latent, **({"kv_from": i - 2} if i % 4 == 3 else {})), "mlp": mlp})
    return {"architecture": "Nirotar", "vocab": raw["vocab_size"], "width": raw["hidden_size"], "norm": {"eps": 1e-6},
            "max_positions": 2 * CONTEXT, "layers": out}


VOGUNEX_LAYERS = ("in turn: attention with the layout's heads (a window of 1,024 positions and, before it, one pooled key and value per "
                  "block of 64; half of every head rotated, scores capped, the heads' weights mixed) with a dense gelu feed-forward; a "
                  "selective state space layer (heads of 64 filling the width, a state of 128 rows, one group, four taps) with experts; "
                  "attention again; attention over a shared latent (as many heads, 64 unrotated + 32 rotated query numbers through a "
                  "latent of 768, values of 64, page rows of 128 + 32 numbers, a window of 1,024, a gate per head) with experts.  A token "
                  "shift in front of every mixer.  8 gated experts with capped inputs of 3/8 of the layout's feed-forward width, 2 chosen, "
                  "and a shared expert of a quarter of it: as many active feed-forward weights per token as the dense layouts")


def vogunex_layout(raw: dict, layers: int) -> dict:
    """A Vogunex configuration at a Qwen3 layout's sizes: the same width, vocabulary and attention heads; feed-forwards that
    activate as many weights per token as the layout's dense gated one (a dense one without a gate is half as wide again)."""
    head, heads, width, ff = raw["head_dim"], raw["num_attention_heads"], raw["hidden_size"], raw["intermediate_size"]
    attention = {"heads": heads, "kv_heads": raw["num_key_value_heads"], "dim": head, "vdim": head, "scale": head ** -0.5, "softcap": 50.0,
                 "mask": {"size": 1024, "pool": 64}, "rot": {"base": 500000.0, "dims": head // 2}}
    latent = {"heads": heads, "dim": 64, "rot_dim": 32, "vdim": 64, "kv_rank": 128, "q_rank": 768, "scale": 96 ** -0.5, "mask": {"size": 1024},
              "rot": {"base": 500000.0, "dims": 32}}
    ssm = {"heads": width // 64, "vdim": 64, "state": 128, "groups": 1, "conv": 4, "norm_groups": 1}
    expert = ff * 3 // 8 // 64 * 64
    moe = {"kind": "moe", "expert": {"ff": expert, "limit": 7.0}, "router": {"experts": 8, "top": 2},
           "shared": {"ff": (ff - 2 * expert) // 64 * 64, "limit": 7.0}}
    dense = {"kind": "dense", "ff": ff * 3 // 2 // 64 * 64}
    kinds = [("attention", attention, dense), ("mamba2", ssm, moe), ("attention", attention, dense), ("latent_attention", latent, moe)]
    return {"architecture": "Vogunex", "vocab": raw["vocab_size"], "width": width, "embedding": {"scale": 1.0}, "norm": {"eps": 1e-6},
            "max_positions": 2 * CONTEXT,
            "layers": [{"type": kinds[i % 4][0], "mixer": kinds[i % 4][1], "mlp": kinds[i % 4][2]} for i in range(layers)]}


PUNUNEX_LAYERS = ("in turn: attention with the layout's heads (a window of 1,024 positions and the first 4 kept, no rotation, scores capped, a learned "
                  "sink) beside a gated delta rule (heads of 128 x 128 filling the width, four taps, a decay per key channel and a sigmoid gate, each "
                  "out of two matrices of rank 128) with a dense relu-gated feed-forward of the layout's width; a gated delta rule alone (as many "
                  "heads, a decay per head, a silu gate) with experts; the parallel layer with experts; the delta rule with experts.  8 gated experts of "
                  "3/8 of the layout's feed-forward width in 2 groups of which both are kept, no identity outputs (every token activates as many "
                  "weights as in the other designs), 2 chosen, and a shared expert of a quarter of it")


def pununex_layout(raw: dict, layers: int) -> dict:
    """A Pununex configuration at a Qwen3 layout's sizes: the same width, vocabulary and attention heads; feed-forwards that
    activate as many weights per token as the layout's dense gated one."""
    head, heads, width, ff = raw["head_dim"], raw["num_attention_heads"], raw["hidden_size"], raw["intermediate_size"]
    attention = {"heads": heads, "kv_heads": raw["num_key_value_heads"], "dim": head, "vdim": head, "scale": head ** -0.5, "softcap": 50.0,
                 "mask": {"size": 1024, "keep_first": 4}}
    delta = {"heads": width // 128, "kv_heads": width // 128, "dim": 128, "vdim": 128, "conv": 4}
    parallel = {"left": attention, "right": dict(delta, decay_rank=128, gate_rank=128), "left_scale": 0.6, "right_scale": 0.4}
    expert = ff * 3 // 8 // 64 * 64
    moe = {"kind": "moe", "expert": {"ff": expert}, "router": {"experts": 8, "top": 2, "identity": 0, "scale": 1.0, "groups": {"count": 2, "keep": 2}},
           "shared": {"ff": (ff - 2 * expert) // 64 * 64}}
    kinds = [("parallel", parallel, {"kind": "dense", "ff": ff}), ("delta", delta, moe), ("parallel", parallel, moe), ("delta", delta, moe)]
    return {"architecture": "Pununex", "vocab": raw["vocab_size"], "width": width, "norm": {"eps": 1e-6}, "max_positions": 2 * CONTEXT,
            "embedding": {"bigram": {"buckets": 65521, "mul_prev": 31, "mul_cur": 17}},
            "layers": [{"type": kinds[i % 4][0], "mixer": kinds[i % 4][1], "mlp": kinds[i % 4][2]} for i in range(layers)]}


PUNOLIX_LAYERS = ("in turn: differential attention (the layout's heads, two maps of half a head each over values of a whole one, neighbouring pairs rotated, "
                  "scores capped); attention with the layout's heads in chunks of 1,024 positions (four taps over q, k and v, q and k normed, half-split "
                  "pairs with band-scaled frequencies) beside gated linear attention (heads of 128 x 128 filling the width, a decay per key channel out of "
                  "two matrices of rank 16, a silu gate).  The layout's dense feed-forward (a gelu gate) beside every mixer on the same norm; one pass of a "
                  "loop around all of them")


def punolix_layout(raw: dict, layers: int) -> dict:
    """A Punolix configuration at a Qwen3 layout's sizes: the same width, vocabulary, attention heads and feed-forward."""
    head, heads, kv, width = raw["head_dim"], raw["num_attention_heads"], raw["num_key_value_heads"], raw["hidden_size"]
    diff = {"heads": heads, "kv_heads": kv, "dim": head // 2, "vdim": head, "scale": (head // 2) ** -0.5, "softcap": 50.0, "diff": 0.4,
            "rot": {"base": 500000.0, "dims": head // 2}}
    left = {"heads": heads, "kv_heads": kv, "dim": head, "vdim": head, "scale": head ** -0.5, "conv": 4, "mask": {"size": 1024},
            "rot": {"base": 500000.0, "dims": head, "scaling": {"factor": 8.0, "low": 1.0, "high": 4.0, "original": 2048}}}
    right = {"heads": width // 128, "dim": 128, "vdim": 128, "tau": 16.0}
    kinds = [("attention", diff), ("parallel", {"left": left, "right": right, "left_scale": 0.6, "right_scale": 0.8})]
    return {"architecture": "Punolix", "vocab": raw["vocab_size"], "width": width, "norm": {"eps": 1e-6}, "max_positions": 2 * CONTEXT, "residual_mult": 0.5,
            "embedding": {"scale": 1.0}, "loop": {"start": 0, "stop": layers, "times": 1},
            "layers": [{"type": kinds[i % 2][0], "mixer": kinds[i % 2][1], "mlp": {"kind": "dense", "ff": raw["intermediate_size"]}} for i in range(layers)]}


def arch_mode(args, pk, arch: str) -> int:
    """Decode and prompt throughput of another architecture at a Qwen3 layout's sizes, and of that Qwen3 layout at the same
    depth, with their fractions of roofline: one JSON line.  With --profile: the architecture's stage tables."""
    import gc

    import torch

    from marin_b200 import Engine
    from marin_b200.config import FegaraxConfig, LakulixConfig, NirotarConfig, PunolixConfig, PununexConfig, Qwen3Config, VogunexConfig

    layers = args.layers or 12
    raw = dict(LAYOUTS[args.model], num_hidden_layers=layers)
    warmup = max(3, args.warmup)
    title = arch.capitalize()
    # the model it is measured beside: the Qwen3 layout, or for Nirotar the engine's closest model, Fegarax at that layout's sizes
    # (for Vogunex: Nirotar, whose windowed and latent attention and experts with a shared one are the nearest kernels)
    # (for Pununex: Vogunex, which keeps recurrent states beside a window of keys and has experts with a shared one)
    # (for Punolix: Pununex, whose windowed attention has capped scores and stands beside a recurrent mixer too)
    beside = {"nirotar": "fegarax", "vogunex": "nirotar", "pununex": "vogunex", "punolix": "pununex"}.get(arch, "qwen3")
    if arch == "punolix":
        other = PunolixConfig.from_dict(punolix_layout(raw, layers))
    elif arch == "pununex":
        other = PununexConfig.from_dict(pununex_layout(raw, layers))
    elif arch == "vogunex":
        other = VogunexConfig.from_dict(vogunex_layout(raw, layers))
    elif arch == "lakulix":
        other = LakulixConfig.from_dict(lakulix_layout(raw, layers))
    elif arch == "fegarax":
        other = FegaraxConfig.from_dict(fegarax_layout(raw, layers))
    else:
        other = NirotarConfig.from_dict(nirotar_layout(raw, layers))
    arms = {arch: other, beside: FegaraxConfig.from_dict(fegarax_layout(raw, layers)) if beside == "fegarax" else
            NirotarConfig.from_dict(nirotar_layout(raw, layers)) if beside == "nirotar" else
            VogunexConfig.from_dict(vogunex_layout(raw, layers)) if beside == "vogunex" else
            PununexConfig.from_dict(pununex_layout(raw, layers)) if beside == "pununex" else Qwen3Config.from_dict(raw)}
    out = {}
    for name, cfg in arms.items():
        if args.profile and name != arch:
            continue
        engine = Engine(config=cfg, seed=0, dtype="bfloat16", ctx=CONTEXT, page_size=PAGE, max_batch=max(args.batch, 8),
                        token_budget=PREFILL_TOKENS)
        fill_cache(engine)
        if args.profile:
            return profile_mode(engine, args, pk, f"{title} at the Qwen3-{args.model.upper()} layout's sizes, {layers} layers", batches=(1, args.batch))
        weight_bytes, prefill_flops = model_bytes_and_flops(engine, args.batch, PREFILL_TOKENS)
        kv_tok = kv_bytes_per_token(engine)
        clocks = ClockSampler(ClockSampler.gpu_in_use())
        clocks.start()
        run = decode_device(engine, args.batch, args.steps, warmup, CONTEXT)
        prefill_ms = prefill_device(engine, PREFILL_TOKENS, runs=3, warmup=3)
        clock_record = clocks.stop()
        # a layer that keeps a state reads the same bytes whatever the context; a layer that keeps keys reads them all
        state_bytes = sum(n.bytes() for n in engine.cache.state_needs.values())
        # (a layer with a window reads the window's positions, however long the sequence)
        # (one with pooled blocks: the window's positions and one row per block before it)
        # (one with a chunked mask: the positions of the current chunk up to its own, on average over the timed steps)
        def seen(entry, need):
            mixer = engine.model.blocks[engine.model.spec.schedule[entry].layer].mixer
            inner = getattr(mixer, "inner", None)
            chunk = max(getattr(m, "chunk", None) or 0 for m in [mixer] + (inner if isinstance(inner, list) else []))
            if chunk:
                return statistics.mean(p % chunk + 1 for p in range(CONTEXT - args.steps, CONTEXT))
            return min(run["mean_context"], need.window or run["mean_context"])

        paged = sum(g.need.bytes_read(int(run["mean_context"]), engine.rt.dtype) if g.need.pooled else g.need.bytes_per_token(engine.rt.dtype) * seen(e, g.need)
                    for g in engine.cache.groups for e in g.entries)
        step_bytes = weight_bytes + args.batch * (paged + 2 * state_bytes)
        achieved = step_bytes / (run["ms_per_step"] / 1e3) / 1e9
        out[name] = {
            "decode_tok_s": round(run["tok_s"], 1), "decode_ms_per_step": round(run["ms_per_step"], 4), "decode_launches": run["launches"],
            "decode_hbm_gbs": round(achieved, 1), "decode_hbm_frac": round(achieved / pk["hbm_gbs"], 4),
            "prefill_tok_s": round(PREFILL_TOKENS / (prefill_ms / 1e3), 1), "prefill_ms": round(prefill_ms, 3),
            "prefill_flops_frac": round(prefill_flops / (prefill_ms / 1e3) / (pk["bf16_tflops"] * 1e12), 4),
            "weight_bytes": weight_bytes, "clocks": clock_record}
        engine.check_device()
        del engine
        gc.collect()
        torch.cuda.empty_cache()
    print(json.dumps({
        "metric": f"{title} beside the {beside.capitalize() + ' layers at the ' if beside != 'qwen3' else ''}Qwen3-{args.model.upper()} layout at equal width, depth and vocabulary: decode tok/s at batch {args.batch} "
                  f"(context {CONTEXT}), prefill tok/s at {PREFILL_TOKENS} tokens, fractions of roofline",
        "unit": "tokens/s", "n_gpus": 1, "steps": args.steps, "warmup": warmup, "dtype": "bf16", "higher_is_better": True,
        "data": "synthetic (uniform random token ids, seeded random weights)", "peaks": pk,
        "config": {"layers": layers, "width": raw["hidden_size"], "ff": raw["intermediate_size"], "vocab": raw["vocab_size"],
                   "global_batch": args.batch, "seq_len": CONTEXT, "prefill_tokens": PREFILL_TOKENS, "kv_block": PAGE,
                   f"{arch}_layers": FEGARAX_LAYERS if arch == "fegarax" else NIROTAR_LAYERS if arch == "nirotar" else VOGUNEX_LAYERS if arch == "vogunex" else
                   PUNUNEX_LAYERS if arch == "pununex" else PUNOLIX_LAYERS if arch == "punolix" else
                   "lightning (heads of 128 x 128), attention (the layout's heads), wkv (heads of 64) in turn, a dense feed-forward in each",
                   "l2": "inputs larger than L2 (weights read per step exceed 126 MB)"},
        arch: out[arch], beside: out[beside], "impl": "ours"}))
    return 0


def reference_arm():
    """The reference is a Rust workspace (cargo, rustc); neither exists in this image, so it cannot be
    built or installed offline, and a pip install of its source tree has nothing to install (no Python package)."""
    print(json.dumps({"impl": "reference", "unavailable": "Kayleexx/marin is a Rust workspace; no cargo/rustc in this image and no Python package to pip-install"}))
    return 0


def main() -> int:
    global CONTEXT
    ap = argparse.ArgumentParser()
    ap.add_argument("--gpus", type=int, default=1)
    ap.add_argument("--steps", type=int, default=64)
    ap.add_argument("--warmup", type=int, default=8)
    ap.add_argument("--batch", type=int, default=8)
    ap.add_argument("--layers", type=int, default=None, help="fewer layers than the configuration has (recorded in config)")
    ap.add_argument("--impl", default="ours", choices=["ours", "reference"])
    ap.add_argument("--no-points", action="store_true", help="skip decode at batch 1 and 64")
    ap.add_argument("--no-e2e", action="store_true")
    ap.add_argument("--model", default="4b", choices=sorted(LAYOUTS), help="layer sizes: Qwen3-4B (the default), 8B or 14B layout")
    ap.add_argument("--context", type=int, default=CONTEXT, help="context length the last timed decode step reaches (default 4096)")
    ap.add_argument("--profile", action="store_true", help="print where a step's time goes, stage by stage, instead of the JSON line")
    ap.add_argument("--arch", default="qwen3", choices=["qwen3", "lakulix", "fegarax", "nirotar", "vogunex", "pununex", "punolix"],
                    help="qwen3: the default workload; lakulix, fegarax: that architecture at the layout's sizes beside the Qwen3 layout of "
                         "equal size; nirotar: beside the Fegarax layers at that layout's sizes; vogunex: beside the Nirotar layers at those sizes; pununex: beside the Vogunex layers; "
                         "punolix: beside the Pununex layers")
    args = ap.parse_args()
    if args.impl == "reference":
        return reference_arm()
    CONTEXT = args.context
    if args.arch != "qwen3":
        if args.gpus != 1:
            print(f"bench.py: this engine runs on one GPU; --gpus {args.gpus} is not supported")
            return 2
        from marin_b200.kernels import build as _build

        _build.build_all(verbose=False)
        return arch_mode(args, peaks(), args.arch)
    if args.gpus != 1:
        print(f"bench.py: this engine runs on one GPU; --gpus {args.gpus} is not supported")
        return 2
    warmup = max(3, args.warmup)

    import torch

    from marin_b200 import Engine
    from marin_b200.config import Qwen3Config
    from marin_b200.kernels import build

    build.build_all(verbose=False)
    raw = dict(LAYOUTS[args.model])
    full_layers = raw["num_hidden_layers"]
    if args.layers:
        raw["num_hidden_layers"] = args.layers
    cfg = Qwen3Config.from_dict(raw)
    pk = peaks()
    max_batch = args.batch if args.no_points else max(args.batch, 64)
    engine = Engine(config=cfg, seed=0, dtype="bfloat16", ctx=CONTEXT, page_size=PAGE, max_batch=max_batch,
                    token_budget=PREFILL_TOKENS)
    fill_cache(engine)
    if args.profile:
        return profile_mode(engine, args, pk)
    weight_bytes, prefill_flops = model_bytes_and_flops(engine, args.batch, PREFILL_TOKENS)
    kv_tok = kv_bytes_per_token(engine)

    clocks = ClockSampler(ClockSampler.gpu_in_use())
    clocks.start()
    main_run = decode_device(engine, args.batch, args.steps, warmup, CONTEXT)
    # the timed steps last a fraction of a second; the same steps run on (untimed) until the sampler has seen about two
    # seconds of this load, so that the median clock rests on tens of readings
    load_until = time.perf_counter() + 2.0
    while time.perf_counter() < load_until:
        decode_device(engine, args.batch, args.steps, 3, CONTEXT)
    clock_record = clocks.stop()

    step_bytes = weight_bytes + args.batch * main_run["mean_context"] * kv_tok
    achieved = step_bytes / (main_run["ms_per_step"] / 1e3) / 1e9
    roofline = {"bound": "hbm", "achieved": round(achieved, 1), "peak": pk["hbm_gbs"], "unit": "GB/s",
                "frac": round(achieved / pk["hbm_gbs"], 4), "peak_source": pk["source"]}

    prefill_ms = prefill_device(engine, PREFILL_TOKENS, runs=3, warmup=3)
    prefill = {"value": round(PREFILL_TOKENS / (prefill_ms / 1e3), 1), "tokens": PREFILL_TOKENS, "ms": round(prefill_ms, 3),
               "frac": round(prefill_flops / (prefill_ms / 1e3) / (pk["bf16_tflops"] * 1e12), 4),
               "peak_tflops": pk["bf16_tflops"], "peak_source": pk["source"],
               # the step is 17 ms of back-to-back kernels and is timed several times in a row: beside the burst figure,
               # the same against the library's rate in a seconds-long loop under the power cap
               "frac_of_sustained": round(prefill_flops / (prefill_ms / 1e3) / (pk["bf16_tflops_sustained"] * 1e12), 4),
               "peak_tflops_sustained": pk["bf16_tflops_sustained"]}

    points = {}
    if not args.no_points:
        per_seq = -(-CONTEXT // PAGE)
        for b in (1, 64):
            if engine.num_pages < b * per_seq:               # a long context: the pool that fits the device holds fewer sequences
                points[f"decode_b{b}"] = None
                continue
            r = decode_device(engine, b, min(args.steps, 32), 3, CONTEXT)
            points[f"decode_b{b}"] = round(r["tok_s"], 1)
            bytes_b = model_bytes_and_flops(engine, b, PREFILL_TOKENS)[0] + b * r["mean_context"] * kv_tok
            points[f"decode_b{b}_hbm_frac"] = round(bytes_b / (r["ms_per_step"] / 1e3) / 1e9 / pk["hbm_gbs"], 4)

    e2e = None
    if not args.no_e2e:
        e2e = decode_e2e(engine, args.batch, args.steps, warmup, CONTEXT)
        e2e["value"] = round(e2e["value"], 1)

    line = {
        "metric": f"decode tok/s at batch {args.batch} (Qwen3-{args.model.upper()} layout, context {CONTEXT}); prefill tok/s at 2048 tokens; % of roofline",
        "value": round(main_run["tok_s"], 1), "unit": "tokens/s", "n_gpus": 1, "steps": args.steps, "warmup": warmup,
        "ms_per_step": round(main_run["ms_per_step"], 4), "higher_is_better": True, "scaling": "weak",
        "vs_baseline": PUBLISHED, "dtype": "bf16", "data": "synthetic (uniform random token ids, seeded random weights N(0,0.02))",
        "config": {"model": f"Qwen3-{args.model.upper()} layout", "layers": cfg.num_hidden_layers, "layers_full": full_layers, "hidden": cfg.hidden_size,
                   "heads": cfg.num_attention_heads, "kv_heads": cfg.num_key_value_heads, "head_dim": cfg.head_dim,
                   "intermediate": cfg.intermediate_size, "vocab": cfg.vocab_size, "tied": cfg.tie_word_embeddings,
                   "global_batch": args.batch, "seq_len": CONTEXT, "kv_block": PAGE, "prefill_tokens": PREFILL_TOKENS,
                   "parallelism": "1 GPU", "l2": "inputs larger than L2 (weights read per step exceed 126 MB)",
                   "sampling": "greedy on device"},
        "clocks": clock_record, "gpu_launches": main_run["launches"], "prefill": prefill, "roofline": roofline,
        "points": points, "impl": "ours",
    }
    if e2e is not None:
        line["e2e"] = e2e
    engine.check_device()                # a kernel whose bounded wait gave up would make the numbers above worthless: raise
    print(json.dumps(line))
    return 0


if __name__ == "__main__":
    sys.exit(main())
