"""Pununex on the GPU against the plain implementation (``plain_pununex``, float64 on the CPU): every mechanism alone, then
whole models under every way of cutting the work: each request alone and whole; most of it in one step and the rest one
token at a time (eagerly and from captured graphs); portions of changing size down to two tokens; mixed batches of unequal
requests with so few pages that they are used again; greedy generation through the engine's entry point and scheduler; and
the trace replay as a user runs it.  Tolerances: ``part_harness``; whole models in bfloat16 0.1 a row and 0.04 on average, two rows
in a hundred beyond, up to a request's first close choice of experts (a margin under 0.02 in float64)."""
import json
import os
import random
import subprocess
import sys

import numpy as np
import pytest
import torch

import plain_pununex as plain
from helpers import mixed_schedule, portions, random_prompt, run_mixed, run_portions, run_whole
from part_harness import DEV, DTYPES, bf, close, cuts_for, feed, harness, mat, runtime
from pununex_models import CONFIGS, PAGE, _attn, _delta, _moe, _parallel, make_model_dir

pytestmark = pytest.mark.gpu
ROOT = os.path.dirname(os.path.dirname(os.path.abspath(__file__)))
LENGTHS = {"A": {"a": 37, "b": 9, "c": 150, "d": 1, "e": 66, "f": 41, "g": 27},
           "B": {"a": 140, "b": 2, "c": 65, "d": 260, "e": 31, "f": 129, "g": 200},
           "C": {"a": 100, "b": 1, "c": 190, "d": 17, "e": 64}}
MARGIN = 0.02


def doubles(w):
    return {k: v.double() for k, v in w.items()}


def part_of(spec, name, rt, weights):
    from marin_b200.parts import lookup

    part = lookup("mixer", spec.kind)(name=name, **spec.params)
    left = {k: v.clone() for k, v in weights.items()}
    part.load(left, rt)
    assert not left
    return part


# ---- attention: window, kept first positions, capped scores, a learned sink -------------------------------------------------------

def attention_weights(hidden, m, seed, same_qk=False, sink=1.5):
    g = torch.Generator().manual_seed(seed)
    H, G, d, dv = m["heads"], m["kv_heads"], m["dim"], m["vdim"]
    w = {"m.q": mat(g, H * d, hidden), "m.k": mat(g, G * d, hidden), "m.v": mat(g, G * dv, hidden), "m.o": mat(g, hidden, H * dv),
         "m.q.norm": 1.5 + 0.3 * torch.randn(d, generator=g), "m.k.norm": 1.5 + 0.3 * torch.randn(d, generator=g), "m.sink": sink * torch.randn(H, generator=g)}
    if same_qk:
        assert H == G
        w["m.k"], w["m.k.norm"] = w["m.q"].clone(), w["m.q.norm"].clone()
    return {k: bf(v) for k, v in w.items()}


def attention_part(m, hidden, eps, rt, w):
    from marin_b200.config.pununex import _attention as parse
    from marin_b200.models.pununex import _attention as spec_of

    return part_of(spec_of(parse(m, ""), hidden, eps), "m", rt, w)


ATTENTIONS = [_attn(3, 1, 12, 10, 0.3, size=9, keep=4, softcap=4.0), _attn(8, 2, 64, 64, 0.125, size=40, keep=20, softcap=30.0),
              _attn(4, 4, 32, 48, 0.2, size=3, keep=17, softcap=5.0), _attn(16, 1, 16, 16, 0.25, size=33, keep=70), _attn(2, 1, 128, 128, 0.09, size=70, keep=1, softcap=20.0),
              _attn(2, 2, 16, 32, 0.25, size=1, keep=2), _attn(4, 2, 48, 16, 0.15, softcap=6.0), _attn(6, 3, 64, 64, 0.125, size=64, keep=64),
              _attn(5, 1, 96, 80, 0.1, size=16, softcap=50.0)]


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("m", ATTENTIONS, ids=lambda m: f"h{m['heads']}k{m['kv_heads']}d{m['dim']}v{m['vdim']}w{(m.get('mask') or {}).get('size')}f{(m.get('mask') or {}).get('keep_first')}")
def test_attention_alone(dtype, m):
    """Every position has edges of its own (the window's, the kept positions'), so comparing all positions under all cuts covers
    them in prompts and in decoding."""
    rt, hidden, T = runtime(dtype), 48, 150
    w = attention_weights(hidden, m, 5)
    x = bf(torch.randn(T, hidden, generator=torch.Generator().manual_seed(6)))
    want = plain.sink_window_attention(x.double(), doubles(w), "m", m, 1e-5)
    part = attention_part(m, hidden, 1e-5, rt, w)
    for page in (8, 16):
        for cuts in cuts_for(T):
            runner = harness([part.cache_need()], rt, page=page)
            close(feed([part], runner, x.to(rt.dtype), cuts)[0], want, dtype, f"page {page}, cuts {cuts[:4]}")
            runner.cache.check()


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("d", [16, 64])
@pytest.mark.parametrize("at", [0, 1, 4, 5, 6, 7, 60, 63, 64, 128, 179, 180, 181, 182, 199])
def test_one_key_stands_out(dtype, d, at):
    """The last token's query meets its own direction at position ``at`` only.  With a window of 19 over 200 positions and six kept ones
    that key is a kept one, the first that is not, far behind the window, its last position inside or the first outside, or the
    query's own: an output that misses it, or sees what it must not, is wrong by far more than any tolerance.  Few pages: those
    between the kept ones and the window have been given back and used again."""
    rt, hidden, T = runtime(dtype), 32, 200
    m = _attn(2, 2, d, 16, 12.0 / d, size=19, keep=6, softcap=40.0)
    w = attention_weights(hidden, m, 3, same_qk=True, sink=0.5)
    g = torch.Generator().manual_seed(at)
    x = torch.randn(T, hidden, generator=g)
    x[at] = x[T - 1] * 2.0                                     # (the norm takes the length away, the direction is the query's own)
    x = bf(x)
    want = plain.sink_window_attention(x.double(), doubles(w), "m", m, 1e-5)
    part = attention_part(m, hidden, 1e-5, rt, w)
    for cuts in ([T], [T - 1, 1], [T - 30] + [1] * 30, portions(T, [16, 2, 5])):
        runner = harness([part.cache_need()], rt, page=8, pages=30 if max(cuts) > 16 else 8)
        got = feed([part], runner, x.to(rt.dtype), cuts)[0]
        close(got[-40:], want[-40:], dtype, f"at {at}, cuts {cuts[:3]}")
        runner.cache.check()


def test_long_sequences_split_their_keys_over_blocks_of_work():
    """Single tokens of a sequence without a window: the keys are split over several CTAs and merged; kept positions beyond one
    block of 64 before a window count as blocks of their own in that split."""
    for m in (_attn(4, 2, 32, 32, 0.3, softcap=8.0), _attn(4, 1, 32, 32, 0.3, size=300, keep=150, softcap=8.0), _attn(4, 1, 64, 64, 0.2, size=130, keep=700)):
        rt, hidden, T = runtime("bfloat16"), 48, 1100
        w = attention_weights(hidden, m, 9)
        x = bf(torch.randn(T, hidden, generator=torch.Generator().manual_seed(6)))
        want = plain.sink_window_attention(x.double(), doubles(w), "m", m, 1e-5)
        part = attention_part(m, hidden, 1e-5, rt, w)
        runner = harness([part.cache_need()], rt, page=16, pages=200)
        close(feed([part], runner, x.to(rt.dtype), [1060] + [1] * 40)[0], want, "bfloat16", str(m))


# ---- the gated delta rule -----------------------------------------------------------------------------------------------------------

def delta_weights(hidden, m, seed, per_channel, ranks=(12, 20), rate=(-3.5, 1.0), dt=(-1.0, 1.0)):
    g = torch.Generator().manual_seed(seed)
    H, G, d, dv, taps = m["heads"], m["kv_heads"], m["dim"], m["vdim"], m["conv"]
    w = {"m.b": mat(g, H, hidden, 1.5), "m.norm": 1.0 + 0.2 * torch.randn(dv, generator=g), "m.o": mat(g, hidden, H * dv, 1.5),
         "m.A_log": torch.rand(H, generator=g) * (rate[1] - rate[0]) + rate[0]}
    for p, rows in (("q", G * d), ("k", G * d), ("v", H * dv)):
        w[f"m.{p}"], w[f"m.{p}.conv"] = mat(g, rows, hidden, 1.5), 0.7 * torch.randn(rows, taps, generator=g)
    if per_channel:
        w.update({"m.a1": mat(g, ranks[0], hidden), "m.a2": mat(g, H * d, ranks[0]), "m.dt_bias": dt[0] + dt[1] * torch.randn(H * d, generator=g),
                  "m.g1": mat(g, ranks[1], hidden), "m.g2": mat(g, H * dv, ranks[1], 2.0)})
    else:
        w.update({"m.a": mat(g, H, hidden), "m.dt_bias": dt[0] + dt[1] * torch.randn(H, generator=g), "m.g": mat(g, H * dv, hidden)})
    return {k: bf(v) for k, v in w.items()}


def delta_part(m, hidden, eps, rt, w, per_channel):
    from marin_b200.config.pununex import _delta as parse
    from marin_b200.models.pununex import _delta as spec_of

    raw = dict(m, decay_rank=w["m.a1"].shape[0], gate_rank=w["m.g1"].shape[0]) if per_channel else m
    return part_of(spec_of(parse(raw, "", per_channel), hidden, eps), "m", rt, w)


DELTAS = [_delta(4, 2, 10, 14, 3), _delta(2, 2, 64, 64, 4), _delta(6, 2, 32, 48, 2), _delta(1, 1, 128, 128, 4), _delta(3, 1, 16, 80, 7),
          _delta(2, 1, 160, 32, 1), _delta(2, 2, 48, 12, 5), _delta(2, 1, 64, 256, 4), _delta(5, 5, 7, 6, 2)]


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("per_channel", [False, True], ids=["head", "channel"])
@pytest.mark.parametrize("m", DELTAS, ids=lambda m: f"h{m['heads']}k{m['kv_heads']}d{m['dim']}v{m['vdim']}c{m['conv']}")
def test_delta_rule_alone(dtype, per_channel, m):
    rt, hidden, T = runtime(dtype), 48, 150
    w = delta_weights(hidden, m, 11, per_channel)
    x = bf(torch.randn(T, hidden, generator=torch.Generator().manual_seed(12)))
    want = plain.delta_mixer(x.double(), doubles(w), "m", m, 1e-5, per_channel)
    part = delta_part(m, hidden, 1e-5, rt, w, per_channel)
    for cuts in cuts_for(T) + [[1] * T, portions(T, [17, 3, 1, 1, 2]), portions(T, [64, 1, 2]), portions(T, [63, 65, 9])]:
        runner = harness([part.cache_need()], rt)
        close(feed([part], runner, x.to(rt.dtype), cuts)[0], want, dtype, f"cuts {cuts[:4]}")
    runner = harness([part.cache_need()], rt)                         # a slot that is used again starts from nothing
    for req in ("a", "b", "c"):
        close(feed([part], runner, x.to(rt.dtype), [50, 1, 1, T - 52], req=req)[0], want, dtype, req)


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("per_channel", [False, True], ids=["head", "channel"])
@pytest.mark.parametrize("d,dv", [(16, 12), (32, 32)])
def test_a_slow_state_remembers_the_first_tokens(dtype, per_channel, d, dv):
    """Decay rates so small that after 400 tokens the first ones still show: a state that is dropped or zeroed between steps is
    seen at once.  Later tokens bring nearly nothing (their betas are near zero)."""
    rt, hidden, T = runtime(dtype), 32, 400
    m = _delta(2, 1, d, dv, 2)
    w = delta_weights(hidden, m, 13, per_channel, rate=(-9.0, -8.0))
    direction = torch.randn(hidden, generator=torch.Generator().manual_seed(15))
    w["m.b"] = bf((direction / hidden ** 0.5)[None].repeat(2, 1))
    x = 0.5 * torch.randn(T, hidden, generator=torch.Generator().manual_seed(14)) - direction
    x[:3] = 2.0 * torch.randn(3, hidden, generator=torch.Generator().manual_seed(16)) + 2.0 * direction
    x = bf(x)
    want = plain.delta_mixer(x.double(), doubles(w), "m", m, 1e-5, per_channel)
    without = plain.delta_mixer(x.double()[3:], doubles(w), "m", m, 1e-5, per_channel)
    assert (want[-1] - without[-1]).abs().max() > 0.2 * want[-1].abs().max()          # the first tokens do matter at the end
    part = delta_part(m, hidden, 1e-5, rt, w, per_channel)
    for cuts in ([T], [T - 100] + [1] * 100, portions(T, [64, 1, 2]), portions(T, [130, 7])):
        runner = harness([part.cache_need()], rt)
        close(feed([part], runner, x.to(rt.dtype), cuts)[0], want, dtype, f"cuts {cuts[:3]}")


def recurrence(q, k, v, beta_raw, a_raw, rate, dt_bias, state, cuts, H, G, d, dv, chunked):
    """``ops.delta_scan`` or ``ops.delta_chunked`` over portions: q, k, v as a convolution would leave them."""
    from marin_b200.engine import StepEntry
    from marin_b200.kernels import ops

    rt = runtime("bfloat16")
    runner = harness([], rt)
    runner.begin("r")
    T = q.shape[0]
    outs, at = [], 0
    for n in cuts:
        ctx = runner.build_context([StepEntry("r", [0] * n, [])])
        rows = torch.cat([q[at:at + n].reshape(n, -1), k[at:at + n].reshape(n, -1), v[at:at + n].reshape(n, -1)], dim=1).to(DEV).contiguous()
        inp = ops.DeltaInputs(beta_raw[at:at + n].to(DEV).contiguous(), a_raw[at:at + n].to(DEV).contiguous(), None, rate.to(DEV), dt_bias.to(DEV))
        o = torch.full((n, H * dv), float("nan"), device=DEV)
        (ops.delta_chunked if chunked else ops.delta_scan)(rows, inp, state, ctx, ctx.state_slots, o, H, G, d, dv)
        outs.append(o.cpu())
        runner.cache.commit("r", at + n)
        at += n
    runner.end("r")
    assert at == T
    return torch.cat(outs)


@pytest.mark.parametrize("chunked", [False, True], ids=["scan", "chunked"])
@pytest.mark.parametrize("per_channel", [False, True], ids=["head", "channel"])
@pytest.mark.parametrize("strength", [0.002, 0.3, 4.0, 60.0])
@pytest.mark.parametrize("d,dv", [(32, 48), (64, 32), (128, 32)])
def test_the_recurrence_is_exact_for_weak_and_strong_decays(chunked, per_channel, strength, d, dv):
    """The recurrence's own arithmetic is 32-bit: on bf16 inputs taken as they are the result and the final state agree with float64
    to about 1e-4, whatever the decays: from nothing forgotten to everything forgotten within a token (where the exponent of a
    chunk's sums reaches thousands), weak and strong channels side by side."""
    H, G, T = 4, 2, 200
    g = torch.Generator().manual_seed(int(strength * 10) + d)
    q, k = (bf(torch.randn(T, G, d, generator=g)) for _ in range(2))
    k[5:60] = k[4]                                                    # one direction again and again: u must correct, not add up
    v = bf(torch.randn(T, H, dv, generator=g))
    beta_raw = bf(2.0 * torch.randn(T, H, generator=g) + 1.0)
    n = H * d if per_channel else H
    a_raw, dt_bias = bf(2.0 * torch.randn(T, n, generator=g)), torch.randn(n, generator=g)
    if per_channel:
        a_raw[:, ::3] -= 30.0                                         # every third channel never forgets
    rate = torch.log(torch.full((H,), strength) * torch.tensor([1.0, 0.5, 2.0, 0.1]))
    start = torch.randn(H, d, dv, generator=g)
    of = torch.arange(H) // (H // G)
    Q = (plain.unit(q.double()) * d ** -0.5)[:, of]
    K = plain.unit(k.double())[:, of]
    decay = plain.softplus(a_raw.double() + dt_bias.double())
    decay = torch.exp(-torch.exp(rate.double())[None, :, None] * (decay.reshape(T, H, d) if per_channel else decay[:, :, None].expand(T, H, d)))
    ends = []
    want = plain.delta_rule(Q, K, v.double(), torch.sigmoid(beta_raw.double()), decay, start.double(), ends)
    for cuts in ([T], portions(T, [64]), portions(T, [65, 100, 2]), portions(T, [9, 3])):
        state = torch.zeros(5, H, d, dv, device=DEV)
        state[:] = start.to(DEV)
        got = recurrence(q, k, v, beta_raw, a_raw, rate, dt_bias, state, cuts, H, G, d, dv, chunked)
        slot = next(i for i in range(5) if not torch.equal(state[i].cpu(), start))
        for name, a, b in (("o", got.double().reshape(T, H, dv), want), ("state", state[slot].double().cpu(), ends[0])):
            err, size = (a - b).abs().max(), b.pow(2).mean().sqrt()
            assert torch.isfinite(a).all() and err <= 3e-4 * size + 1e-6, (name, cuts[:3], float(err), float(size))


def test_several_requests_in_one_step_share_the_chunks_memory():
    """Portions of unequal length and single tokens in one step: every request's result is what it gets alone."""
    from marin_b200.engine import StepEntry

    m, hidden = _delta(4, 2, 32, 32, 4), 48
    rt = runtime("bfloat16")
    w = delta_weights(hidden, m, 17, True)
    part = delta_part(m, hidden, 1e-5, rt, w, True)
    lengths = {"a": [130, 1, 1, 40], "b": [1, 1, 70, 1], "c": [2, 65, 63, 2], "d": [64, 128, 1, 9]}
    xs = {r: bf(torch.randn(sum(n), hidden, generator=torch.Generator().manual_seed(i))) for i, (r, n) in enumerate(lengths.items())}
    runner = harness([part.cache_need()], rt)
    for r in lengths:
        runner.begin(r)
    at, got = {r: 0 for r in lengths}, {r: [] for r in lengths}
    for step in range(4):
        entries = [StepEntry(r, [0] * lengths[r][step], []) for r in lengths]
        ctx = runner.build_context(entries)
        rows = torch.cat([xs[s.req_id][at[s.req_id]:at[s.req_id] + s.count] for s in sorted(ctx.spans, key=lambda s: s.start)]).to(DEV).contiguous()
        residual = torch.zeros(rows.shape[0], hidden, device=DEV)
        part.forward(rows, ctx, runner.views.view(0, ctx), residual)
        for s in ctx.spans:
            got[s.req_id].append(residual[s.start:s.start + s.count].cpu())
            at[s.req_id] += s.count
            runner.cache.commit(s.req_id, at[s.req_id])
    for r in lengths:
        want = plain.delta_mixer(xs[r].double(), doubles(w), "m", m, 1e-5, True)
        close(torch.cat(got[r]), want, "bfloat16", r)


@pytest.mark.parametrize("dtype", DTYPES)
def test_mixers_side_by_side_are_weighted_and_added(dtype):
    from marin_b200.config.pununex import _mixer as parse
    from marin_b200.models.pununex import _mixer as spec_of

    rt, hidden, T = runtime(dtype), 64, 120
    raw = _parallel(_attn(4, 2, 32, 32, 0.2, size=20, keep=3, softcap=9.0), _delta(3, 1, 32, 48, 3), 0.4, -1.3)
    w = {k.replace("m.", "m.left.", 1): v for k, v in attention_weights(hidden, raw["left"], 1).items()}
    w.update({k.replace("m.", "m.right.", 1): v for k, v in delta_weights(hidden, raw["right"], 2, True).items()})
    x = bf(torch.randn(T, hidden, generator=torch.Generator().manual_seed(3)))
    want = plain.mixer({"type": "parallel", "mixer": raw}, x.double(), doubles(w), "m", 1e-5)
    m = parse("parallel", dict(raw, right=dict(raw["right"], decay_rank=12, gate_rank=20)), "")
    part = part_of(spec_of("parallel", m, hidden, 1e-5), "m", rt, w)
    for cuts in cuts_for(T):
        runner = harness([part.cache_need()], rt, page=8)
        close(feed([part], runner, x.to(rt.dtype), cuts)[0], want, dtype, f"cuts {cuts[:4]}")


# ---- embedding ------------------------------------------------------------------------------------------------------------------------

@pytest.mark.parametrize("dtype", DTYPES)
def test_bigram_embedding_carries_the_token_before_across_steps(dtype):
    from marin_b200.engine import StepEntry
    from marin_b200.parts import lookup

    rt, hidden, vocab = runtime(dtype), 20, 50
    # products beyond 2^31 before the remainder is taken
    bigram = {"buckets": 23, "mul_prev": 100000007, "mul_cur": 99999989}
    g = torch.Generator().manual_seed(1)
    w = {"embed": bf(torch.randn(vocab, hidden, generator=g)), "bigram": bf(torch.randn(24, hidden, generator=g))}
    part = lookup("embedding", "token_table")(vocab=vocab, hidden=hidden, name="embed", tensor="embed", bigram=bigram, bigram_tensor="bigram")
    part.load({k: v.clone() for k, v in w.items()}, rt)
    rng = random.Random(2)
    runner = harness([part.cache_need()], rt)
    for cuts in ([40], [1] * 40, portions(40, [2]), portions(40, [5, 1, 1, 9])):
        tokens = [rng.randrange(vocab) for _ in range(40)]
        want = plain.embedding(tokens, doubles(w), bigram)
        runner.begin("r")                                             # (the slot of the request before, used again)
        got, at = [], 0
        for n in cuts:
            ctx = runner.build_context([StepEntry("r", tokens[at:at + n], [])])
            out = torch.zeros(n, hidden, device=DEV)
            part.forward(ctx.token_ids, out, ctx.positions, ctx=ctx, cache=runner.views.view(0, ctx))
            got.append(out.cpu())
            at += n
            runner.cache.commit("r", at)
        runner.end("r")
        close(torch.cat(got), want, "float32", f"cuts {cuts[:4]}", exact=1e-6)


# ---- norms and feed-forwards ------------------------------------------------------------------------------------------------------------

@pytest.mark.parametrize("rows,n", [(1, 44), (3, 128), (300, 320), (7, 2560), (200, 5120), (2, 1001), (150, 36)])
@pytest.mark.parametrize("kind", ["layer", "rms"])
def test_the_norm_that_joins_the_stream(rows, n, kind):
    from marin_b200.kernels import ops

    g = torch.Generator().manual_seed(rows + n)
    y, hidden = 3.0 + 2.0 * torch.randn(rows, n, generator=g), torch.randn(rows, n, generator=g)
    y[0] *= 1e-3                                                      # a row whose variance is near eps
    w, b, s = (torch.randn(n, generator=g) for _ in range(3))
    for bias, scale, wide in ((b, s, False), (None, s, True), (b, None, False)):
        v = y.double()
        if kind == "layer":
            want = plain.layer_norm(v, w.double(), bias.double() if bias is not None else torch.zeros(n).double(), 1e-5)
        else:
            want = plain.rms_norm(v, w.double(), 1e-5) + (bias.double() if bias is not None else 0.0)
        want = hidden.double() + want * (scale.double() if scale is not None else 1.0)
        dy, dh = y.to(DEV), hidden.to(DEV)
        out = torch.zeros(rows, n, device=DEV, dtype=torch.float32 if wide else torch.bfloat16)
        dev = lambda t: t.to(DEV) if t is not None else None
        ops.norm_into(dy, kind, dev(w), dev(bias), 1e-5, dev(scale), dh, out)
        close(dh, want, "float32", "stream", exact=2e-5)
        assert torch.equal(out, dh.to(out.dtype)) and not bool(dy.any())
    if kind == "layer":
        out = torch.zeros(rows, n, device=DEV)
        dy = y.to(DEV)
        ops.layer_norm(dy, w.to(DEV), b.to(DEV), 1e-5, out)
        close(out, plain.layer_norm(y.double(), w.double(), b.double(), 1e-5), "float32", "plain", exact=2e-5)
        assert torch.equal(dy.cpu(), y)


def feedforward_part(mlp, hidden, rt, w):
    from marin_b200.config.pununex import _mlp
    from marin_b200.models.pununex import _feedforward
    from marin_b200.parts import lookup

    spec = _feedforward(_mlp(mlp, ""), hidden)
    part = lookup("feedforward", spec.kind)(name="f", **spec.params)
    left = {k: v.clone() for k, v in w.items()}
    part.load(left, rt)
    assert not left
    return part


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("hidden,ff,T", [(40, 56, 9), (128, 256, 150), (64, 33, 1), (256, 2048, 700)])
def test_dense_relu_feed_forward_alone(dtype, hidden, ff, T):
    rt = runtime(dtype)
    g = torch.Generator().manual_seed(hidden)
    w = {"f.gate": bf(mat(g, ff, hidden)), "f.up": bf(mat(g, ff, hidden)), "f.down": bf(mat(g, hidden, ff, 1.5))}
    x = bf(torch.randn(T, hidden, generator=g))
    want = plain.feed_forward(x.double(), doubles(w), "f", {"kind": "dense", "ff": ff})
    part = feedforward_part({"kind": "dense", "ff": ff}, hidden, rt, w)
    close(feed([part], harness([], rt), x.to(rt.dtype), [T], mixer=False)[0], want, dtype)


EXPERTS = [(40, 24, 5, 2, dict(identity=1, groups=(3, 2), scale=1.5, shared=40), 23), (128, 64, 8, 3, dict(identity=4, groups=(3, 1), scale=2.5, shared=128), 300),
           (128, 128, 4, 1, dict(identity=2, groups=(2, 1), shared=64), 7), (64, 64, 2, 2, {}, 50), (64, 32, 3, 3, dict(scale=0.3, shared=32), 1),
           (128, 64, 12, 4, dict(identity=4, groups=(8, 5), shared=64), 1200), (64, 64, 2, 2, dict(identity=6, scale=3.0), 90), (64, 64, 5, 5, dict(identity=1, groups=(6, 5)), 33)]


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("hidden,ff,E,top,more,T", EXPERTS, ids=lambda v: str(v) if isinstance(v, int) else "")
def test_routed_experts_alone(dtype, hidden, ff, E, top, more, T):
    """Rows whose choice is a close call in float64 are left out.  All choice scores are below zero (a group that is not kept must
    count as less than any of them), and the correction overrules the scores in most rows (the weights must stay without it)."""
    rt = runtime(dtype)
    g = torch.Generator().manual_seed(hidden + E)
    mlp = _moe(ff, E, top, **more)
    n = E + mlp["router"].get("identity", 0)
    w = {"f.router": bf(mat(g, n, hidden)), "f.correction": bf(0.3 * torch.randn(n, generator=g) - 2.0)}
    for e in range(E):
        w[f"f.e{e}.gate"], w[f"f.e{e}.up"], w[f"f.e{e}.down"] = bf(mat(g, ff, hidden)), bf(mat(g, ff, hidden)), bf(mat(g, hidden, ff, 1.5))
    if more.get("shared"):
        s = more["shared"]
        w["f.shared.gate"], w["f.shared.up"], w["f.shared.down"] = bf(mat(g, s, hidden)), bf(mat(g, s, hidden)), bf(mat(g, hidden, s, 1.5))
    x = bf(torch.randn(3 * T + 8, hidden, generator=g))
    margins = plain.route(x.double(), doubles(w), "f", mlp["router"])[2]
    x = x[margins > 1e-3][:T].contiguous()
    assert x.shape[0] >= T // 2
    want = plain.routed_mlp(x.double(), doubles(w), "f", mlp)
    part = feedforward_part(mlp, hidden, rt, w)
    close(feed([part], harness([], rt), x.to(rt.dtype), [x.shape[0]], mixer=False)[0], want, dtype)
    if x.shape[0] > 12:                                               # few rows at a time: other tiles, the same rows
        close(feed([part], harness([], rt), x[:12].to(rt.dtype), [1, 2, 9], mixer=False)[0], want[:12], dtype)


# ---- whole models -----------------------------------------------------------------------------------------------------------------

class Case:
    def __init__(self, tmp, name, dtype):
        from marin_b200.engine import load_model

        self.name, self.dtype = name, dtype
        self.raw = CONFIGS[name]
        self.dir = make_model_dir(str(tmp / f"{name}-{dtype}"), name, seed=11)
        self.w = plain.read_weights(self.dir)
        rng = random.Random(5)
        self.tokens = {rid: random_prompt(rng, self.raw["vocab"], n) for rid, n in LENGTHS[name].items()}
        self.want, self.safe = {}, {}
        for rid, t in self.tokens.items():
            margins = []
            self.want[rid] = plain.forward(self.raw, self.w, t, None, margins)
            tight = torch.stack(margins).min(dim=0).values < MARGIN if margins else torch.zeros(len(t), dtype=torch.bool)
            self.safe[rid] = int(torch.nonzero(tight)[0]) if bool(tight.any()) else len(t)
        self.rt = runtime(dtype)
        self.config, self.model = load_model(self.dir, self.rt)
        self.page = PAGE[name]
        self.loose = 0.0 if dtype == "float32" else 0.02

    def runner(self, num_pages, max_requests=4, graphs=False):
        from marin_b200.cache import CacheManager
        from marin_b200.engine import Runner

        cache = CacheManager(self.model.cache_needs(), [e.cache_of for e in self.model.spec.schedule], self.page, num_pages, max_requests)
        cache.allocate(self.rt.device, self.rt.dtype)
        runner = Runner(self.model, cache, self.rt, 512)
        if graphs:
            runner.enable_graphs((1, 2, 4))
        return runner

    def close(self, got, rid, what):
        close(got, self.want[rid], self.dtype, what, self.loose, self.safe[rid], 0.1, 0.04)


@pytest.fixture(scope="module", params=[(n, d) for n in CONFIGS for d in DTYPES], ids=lambda p: f"{p[0]}-{p[1]}")
def case(request, tmp_path_factory):
    return Case(tmp_path_factory.mktemp("pununex"), *request.param)


def test_the_residual_stream_after_every_layer(case):
    from marin_b200.engine import StepEntry

    rid = "a"
    want = []
    plain.forward(case.raw, case.w, case.tokens[rid], want)
    got = {}
    runner = case.runner(64)
    runner.begin(rid)
    runner.step([StepEntry(rid, case.tokens[rid], [0])], observe=lambda i, h: got.__setitem__(i, h.clone()))
    assert len(got) == len(want) + 1
    for i in range(len(want)):
        close(got[i + 1], want[i], case.dtype, f"after layer {i}", case.loose, case.safe[rid], 0.1, 0.04)


def test_whole_prompts_and_the_first_tokens(case):
    runner = case.runner(64)
    for rid, tokens in case.tokens.items():
        case.close(run_whole(runner, rid, tokens), rid, f"{rid} whole")
    runner.cache.check()


@pytest.mark.parametrize("graphs", [False, True])
def test_prefill_then_token_by_token(case, graphs):
    """Most of a prompt in one step and the rest one token at a time, eagerly and from captured graphs: a tail long enough for
    every window to pass wholly over decoded tokens; and a request decoded from its very first token."""
    runner = case.runner(64, graphs=graphs)
    for rid, tail in (("c", 100), ("a", 30), ("e", 5)):
        tokens = case.tokens[rid]
        n = max(len(tokens) - tail, 0)
        sizes = ([n] if n > 0 else []) + [1] * (len(tokens) - n)
        case.close(run_portions(runner, rid + "t", tokens, sizes), rid, f"{rid}, last {tail} one by one")
    rid = "e"
    case.close(run_portions(runner, rid + "1", case.tokens[rid], [1] * len(case.tokens[rid])), rid, f"{rid} token by token")
    runner.cache.check()


def test_portions_of_changing_size_down_to_two_tokens(case):
    runner = case.runner(64)
    for rid in ("c", "a"):
        tokens = case.tokens[rid]
        for sizes in ([7, 2, 13, 3, 2, 5], [2], [case.page, case.page + 1, case.page - 1], [64, 1, 2]):
            case.close(run_portions(runner, rid + "p", tokens, portions(len(tokens), sizes)), rid, f"{rid} in {sizes}")


@pytest.mark.parametrize("graphs", [False, True])
def test_mixed_batches_reuse_pages_and_slots(case, graphs):
    """Up to four live requests, portions of some beside single tokens of others, in a pool that holds the four largest only:
    pages and slots of finished requests are handed to the next ones."""
    rng = random.Random(9)
    lengths = {rid: len(t) for rid, t in case.tokens.items()}
    sched = mixed_schedule(rng, lengths, max_live=4, decode_tail=6)
    pool = sum(sorted((-(-n // case.page) for n in lengths.values()), reverse=True)[:4])
    runner = case.runner(pool, max_requests=4, graphs=graphs)
    for again in ("", ", second time"):
        got = run_mixed(runner, case.tokens, sched)
        for rid in case.tokens:
            case.close(got[rid], rid, f"{rid} mixed{again}")
        runner.cache.check()
        assert all(g.pool.num_held == 0 for g in runner.cache.groups)


def test_a_batch_gives_each_request_what_it_gets_alone(case):
    """float32: the logits of a request are the same bits whatever else the step holds and however its prompt was cut into
    portions of several tokens."""
    if case.dtype != "float32":
        pytest.skip("bit equality is the 32-bit path's claim")
    from marin_b200.engine import StepEntry

    runner = case.runner(96)
    alone = {rid: run_whole(runner, rid, case.tokens[rid]) for rid in ("a", "c", "e")}
    for rid in alone:
        runner.begin(rid)
    logits = runner.step([StepEntry(rid, case.tokens[rid], list(range(len(case.tokens[rid])))) for rid in ("a", "c", "e")])
    k = 0
    for rid in ("a", "c", "e"):
        n = len(case.tokens[rid])
        assert torch.equal(logits[k:k + n], alone[rid]), rid
        k += n
        runner.end(rid)
    cuts = portions(len(case.tokens["a"]), [5, 2, 9])
    cuts = cuts if cuts[-1] > 1 else cuts[:-2] + [cuts[-2] + 1]
    cut = run_portions(runner, "ap", case.tokens["a"], cuts)
    close(cut, alone["a"].double().cpu(), "float32", "cut", exact=2e-5)


def test_greedy_generation_through_the_engine(case):
    """The entry point, the scheduler and device sampling: the tokens are those the plain implementation's logits rank first (a
    token whose plain logit lies within 1e-3 (32-bit) or 0.15 (16-bit) of the largest counts as first; in 16 bits a sequence
    is followed only as far as no choice of experts is a close call)."""
    from marin_b200.engine import Engine
    from marin_b200.sampling.sampler import SamplingParams

    engine = Engine(case.dir, dtype=case.dtype, ctx=256, page_size=case.page, num_pages=64, max_batch=4, token_budget=32)
    prompts = [case.tokens["a"][:21], case.tokens["e"][:3], case.tokens["c"][:40]]
    outs = engine.generate(prompts, SamplingParams(temperature=0.0, max_tokens=10))
    slack = 1e-3 if case.dtype == "float32" else 0.15
    for prompt, out in zip(prompts, outs):
        assert len(out.tokens) == 10
        seq = list(prompt)
        for token in out.tokens:
            margins = []
            logits = plain.forward(case.raw, case.w, seq, None, margins)[-1]
            if case.dtype != "float32" and margins and min(float(mm.min()) for mm in margins) < MARGIN:
                break
            assert logits[token] >= logits.max() - slack, (len(seq), token, int(logits.argmax()))
            seq.append(token)


def test_preempted_requests_start_again_from_their_first_token(tmp_path):
    """So few pages that a running request is preempted: it comes back with prompt and generated tokens recomputed, its state and the
    token before its first one as at a sequence's start, and produces what it produces alone."""
    from marin_b200.engine import Engine
    from marin_b200.sampling.sampler import SamplingParams

    d = make_model_dir(str(tmp_path / "m"), "A", seed=21)
    rng = random.Random(4)
    prompts = [random_prompt(rng, 83, n) for n in (30, 26, 33)]
    params = SamplingParams(temperature=0.0, max_tokens=40)
    many = Engine(d, dtype="float32", ctx=128, page_size=4, num_pages=200, max_batch=3, token_budget=32)
    few = Engine(d, dtype="float32", ctx=128, page_size=4, num_pages=22, max_batch=3, token_budget=32)
    alone = [many.generate([p], params)[0].tokens for p in prompts]
    assert [o.tokens for o in few.generate(prompts, params)] == alone


def test_trace_replay_as_a_user_runs_it(tmp_path):
    """bin/trace_run in a process of its own: steps on standard input, logits read back from files."""
    name, dtype = "B", "float32"
    raw = CONFIGS[name]
    d = make_model_dir(str(tmp_path / "model"), name, seed=12)
    w = plain.read_weights(d)
    rng = random.Random(3)
    lengths = {"a": 70, "b": 130, "c": 41, "d": 64, "e": 100, "f": 2}
    tokens = {rid: random_prompt(rng, raw["vocab"], n) for rid, n in lengths.items()}
    want = {rid: plain.forward(raw, w, t) for rid, t in tokens.items()}
    sched = mixed_schedule(rng, lengths, max_live=4, decode_tail=5)
    pool = sum(sorted((-(-n // 64) * 64 for n in lengths.values()), reverse=True)[:4])
    out = str(tmp_path / "out")
    proc = subprocess.Popen([sys.executable, os.path.join(ROOT, "bin", "trace_run"), "--model", d, "--dtype", dtype, "--out", out,
                             "--max-tokens", str(pool)], stdin=subprocess.PIPE, stdout=subprocess.PIPE, text=True)
    fed = {rid: 0 for rid in tokens}
    for i, (entries, ends) in enumerate(sched):
        line, rows = [], []
        for rid, n in entries:
            wanted = [n - 1] if n > 2 else list(range(n))
            line.append({"id": rid, "tokens": tokens[rid][fed[rid]:fed[rid] + n], "want": wanted})
            rows.append(want[rid][[fed[rid] + k for k in wanted]])
            fed[rid] += n
        proc.stdin.write(json.dumps({"step": i, "entries": line, "end": ends}) + "\n")
        proc.stdin.flush()
        assert proc.stdout.readline().strip() == f"done {i}"
        got = torch.from_numpy(np.fromfile(os.path.join(out, f"{i}.f32"), dtype="<f4").reshape(-1, raw["vocab"]).copy())
        close(got, torch.cat(rows), dtype, f"step {i}")
    proc.stdin.close()
    assert proc.wait(timeout=120) == 0


def test_the_command_line_takes_a_pununex_folder(tmp_path):
    """Random-weights mode from a config.json of this design, greedy generation, and the bench command with its stage table."""
    run = [sys.executable, os.path.join(ROOT, "bin", "marin-run")]
    cfg = tmp_path / "cfg.json"
    cfg.write_text(json.dumps(CONFIGS["B"]))
    model = str(tmp_path / "model")
    out = subprocess.run(run + ["random", "--config", str(cfg), "--seed", "3", "--out", model], capture_output=True, text=True)
    assert out.returncode == 0, out.stderr
    assert sorted(os.listdir(model)) == ["config.json", "model.safetensors"]
    a = subprocess.run(run + [model, "--prompt-ids", "5,6,7,8,9", "--temp", "0", "--max-tokens", "6"], capture_output=True, text=True)
    b = subprocess.run(run + [model, "--prompt-ids", "5 6 7 8 9", "--temp", "0", "--max-tokens", "6"], capture_output=True, text=True)
    assert a.returncode == 0 and b.returncode == 0, a.stderr + b.stderr
    assert a.stdout == b.stdout and len(a.stdout.split()) == 6
    e = subprocess.run(run + ["bench", model, "--prompt-tokens", "16", "--tokens", "8", "--runs", "2", "--warmup", "1", "--profile"],
                       capture_output=True, text=True)
    assert e.returncode == 0, e.stderr
    for stage in ("embedding", "norm into the stream", "inputs of both", "q|k|v|b", "attention", "delta rule", "convolution", "decay, gate", "router", "experts", "gate|up, relu",
                  "head", "sampling"):
        assert stage in e.stdout, stage
