"""Punolix on the GPU against the plain implementation (``plain_punolix``, float64 on the CPU): every mechanism alone, then whole models under
every way of cutting the work: each request alone and whole; most of it in one step and the rest one token at a time (eagerly and from
captured graphs); portions of changing size down to two tokens; mixed batches of unequal requests with so few pages that they are used
again; greedy generation through the engine's entry point and scheduler; and the trace replay as a user runs it.  Tolerances:
``part_harness``; whole models in bfloat16 0.1 a row and 0.04 on average, two rows in a hundred beyond."""
import json
import math
import os
import random
import subprocess
import sys

import numpy as np
import pytest
import torch

import plain_punolix as plain
from helpers import mixed_schedule, portions, random_prompt, run_mixed, run_portions, run_whole
from part_harness import DEV, DTYPES, bf, close, cuts_for, feed, harness, mat, runtime
from punolix_models import (CONFIGS, PAGE, Draw, _diff, _layer, _left, _parallel, _right, _rot, attention_tensors, left_tensors, make_model_dir,
                            right_tensors)

pytestmark = pytest.mark.gpu
ROOT = os.path.dirname(os.path.dirname(os.path.abspath(__file__)))
LENGTHS = {"A": {"a": 37, "b": 9, "c": 150, "d": 1, "e": 66, "f": 41, "g": 27},
           "B": {"a": 140, "b": 2, "c": 65, "d": 260, "e": 31, "f": 129, "g": 200},
           "C": {"a": 100, "b": 1, "c": 190, "d": 17, "e": 64}}


def doubles(w):
    return {k: v.double() for k, v in w.items()}


def drawn(kind, hidden, m, seed, rank=None):
    """A mixer's random tensors under the name "m"."""
    w, matrix = {}, Draw(seed, hidden)
    if kind == "right":
        right_tensors(matrix.normal, matrix, w, "m", m, rank)
    else:
        (attention_tensors if kind == "attention" else left_tensors)(matrix.normal, matrix, w, "m", m)
    return {k: bf(v) for k, v in w.items()}


def part_of(kind, m, hidden, rt, w, **more):
    """The mixer a configuration of this kind stands for, with these weights."""
    from marin_b200.config import punolix as config
    from marin_b200.models import punolix as model
    from marin_b200.parts import lookup

    if kind == "right":
        m = dict(m, decay_rank=w["m.a1"].shape[0])
    parse, spec_of = {"attention": (config._differential, model._differential), "left": (config._chunked, model._chunked), "right": (config._linear, model._linear)}[kind]
    spec = spec_of(parse(m, ""), hidden, 1e-5)
    part = lookup("mixer", spec.kind)(name="m", **spec.params, **more)
    left = {k: v.clone() for k, v in w.items()}
    part.load(left, rt)
    assert not left
    return part


def inputs(T, hidden, seed):
    return bf(torch.randn(T, hidden, generator=torch.Generator().manual_seed(seed)))


def label(m):
    return "h{heads}k{kv}d{dim}v{vdim}".format(heads=m["heads"], kv=m.get("kv_heads", ""), dim=m["dim"], vdim=m["vdim"])


# ---- differential attention ---------------------------------------------------------------------------------------------------------

DIFFS = [_diff(3, 1, 6, 10, 0.5, _rot(4, 500.0), 0.25, softcap=6.0), _diff(4, 1, 64, 128, 0.125, _rot(64, 9000.0), 0.3, softcap=20.0),
         _diff(6, 3, 32, 64, 0.2, _rot(32, 700.0), 0.5), _diff(2, 2, 32, 128, 0.18, _rot(2, 100.0), 0.8, softcap=4.0), _diff(8, 1, 64, 64, 0.125, _rot(16, 10000.0), 0.1),
         _diff(4, 2, 8, 16, 0.4, _rot(8, 50.0), 0.3, softcap=5.0), _diff(2, 1, 128, 96, 0.09, _rot(128, 10000.0), 0.4, softcap=30.0), _diff(5, 5, 40, 48, 0.16, _rot(40, 300.0), -0.3),
         _diff(12, 1, 16, 32, 0.25, _rot(16, 900.0), 0.2)]


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("m", DIFFS, ids=label)
def test_differential_attention_alone(dtype, m):
    rt, hidden, T = runtime(dtype), 48, 150
    w = drawn("attention", hidden, m, 5)
    x = inputs(T, hidden, 6)
    want = plain.differential_attention(x.double(), doubles(w), "m", m, 1e-5)
    part = part_of("attention", m, hidden, rt, w)
    for page in (8, 16):
        for cuts in cuts_for(T):
            runner = harness([part.cache_need()], rt, page=page)
            close(feed([part], runner, x.to(rt.dtype), cuts)[0], want, dtype, f"page {page}, cuts {cuts[:4]}")
            runner.cache.check()


def test_both_maps_and_the_biases_matter():
    """What the comparisons above would not notice if it did not show: the second map, its weight, every bias, the cap."""
    m, hidden = DIFFS[1], 48
    w = doubles(drawn("attention", hidden, m, 5))
    x = inputs(60, hidden, 6).double()
    want = plain.differential_attention(x, w, "m", m, 1e-5)
    off = lambda other: float((other - want).pow(2).mean().sqrt() / want.pow(2).mean().sqrt())
    assert 0.2 < plain.lam_of(w, "m", m["diff"]) < 0.9
    for name in ("m.q.b", "m.k.b", "m.v.b"):
        assert off(plain.differential_attention(x, dict(w, **{name: torch.zeros_like(w[name])}), "m", m, 1e-5)) > 0.1, name
    assert off(plain.differential_attention(x, w, "m", dict(m, diff=-0.6), 1e-5)) > 0.2
    swapped = dict(w, **{"m.q": w["m.q"].reshape(-1, 2, m["dim"], hidden).flip(1).reshape_as(w["m.q"])})
    assert off(plain.differential_attention(x, swapped, "m", m, 1e-5)) > 0.2
    assert off(plain.differential_attention(x, w, "m", dict(m, softcap=None), 1e-5)) > 0.002


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("which", [0, 1])
@pytest.mark.parametrize("dim,vdim", [(6, 12), (32, 64), (64, 128), (24, 48)])
@pytest.mark.parametrize("at", [0, 1, 7, 8, 63, 64, 127, 128, 198, 199])
def test_one_key_stands_out_in_one_map(dtype, which, dim, vdim, at):
    """The last token's query meets its own direction at position ``at`` (and at itself) only, in one of the two maps: the other map sees nothing but
    small scores.  A map that is read with the other's keys, or a far key that is missed, is wrong by far more than any tolerance.  (Queries and
    keys read the first half of the rows, values the second: what is found is not what the last token has itself.)"""
    rt, hidden, T = runtime(dtype), 40, 200
    m = _diff(2, 2, dim, vdim, 20.0 / dim, _rot(2, 1e9), 0.4, softcap=60.0)
    w = drawn("attention", hidden, m, 3)
    q = w["m.q"].reshape(2, 2, dim, hidden).clone()
    q[:, 1 - which] *= 0.05
    q[..., hidden // 2:] = 0
    q[:, :, :2] = 0                                                            # (the pair that turns holds no more than its bias)
    w["m.q"], w["m.k"] = q.reshape(-1, hidden), q.reshape(-1, hidden).clone()
    w["m.v"][:, :hidden // 2] = 0
    for b in ("q", "k"):
        w[f"m.{b}.b"] = bf(0.02 * w[f"m.{b}.b"].float())
    x = torch.randn(T, hidden, generator=torch.Generator().manual_seed(at)) * 0.4
    x[T - 1, :hidden // 2] *= 4.0
    x[at, :hidden // 2] = x[T - 1, :hidden // 2]
    x[:, hidden // 2:] *= 2.5
    x = bf(x)
    want = plain.differential_attention(x.double(), doubles(w), "m", m, 1e-5)
    without = x.clone()
    without[at, :hidden // 2] = 0.0
    if at < T - 1:
        change = plain.differential_attention(without.double(), doubles(w), "m", m, 1e-5)[-1] - want[-1]
        assert change.pow(2).mean().sqrt() > 0.25 * want[-1].pow(2).mean().sqrt()
    part = part_of("attention", m, hidden, rt, w)
    for cuts in ([T], [T - 1, 1], [T - 30] + [1] * 30, portions(T, [16, 2, 5])):
        runner = harness([part.cache_need()], rt, page=16, pages=30)
        got = feed([part], runner, x.to(rt.dtype), cuts)[0]
        close(got[-40:], want[-40:], dtype, f"at {at}, cuts {cuts[:3]}")


@pytest.mark.parametrize("m", [_diff(6, 3, 32, 64, 0.3, _rot(32, 5000.0), 0.3, softcap=12.0), _diff(2, 1, 64, 128, 0.2, _rot(64, 5000.0), 0.5),
                               _diff(3, 1, 24, 48, 0.3, _rot(24, 5000.0), 0.2, softcap=9.0)], ids=label)
def test_long_sequences_split_their_keys_over_blocks_of_work(m):
    """Single tokens of a long sequence: the keys are split over several CTAs, both maps' parts merged and combined; and a prompt of many tiles."""
    rt, hidden, T = runtime("bfloat16"), 48, 1100
    w = drawn("attention", hidden, m, 9)
    x = inputs(T, hidden, 6)
    want = plain.differential_attention(x.double(), doubles(w), "m", m, 1e-5)
    part = part_of("attention", m, hidden, rt, w)
    runner = harness([part.cache_need()], rt, page=16, pages=200)
    close(feed([part], runner, x.to(rt.dtype), [1060] + [1] * 40)[0], want, "bfloat16", str(m))


# ---- attention inside chunks, behind a short convolution ---------------------------------------------------------------------------

LEFTS = [_left(4, 2, 12, 10, 0.3, _rot(8, 900.0, (3.0, 1.0, 4.0, 60)), conv=3, chunk=11), _left(8, 2, 128, 64, 0.09, _rot(64, 50000.0, (8.0, 1.0, 4.0, 128)), conv=4, chunk=70),
         _left(4, 4, 64, 64, 0.125, _rot(64, 10000.0), conv=2, chunk=33), _left(4, 1, 32, 48, 0.2, _rot(32, 1000.0, (2.0, 0.5, 3.0, 32)), chunk=1),
         _left(6, 3, 48, 32, 0.15, _rot(24, 1000.0), conv=7, chunk=64), _left(2, 2, 16, 16, 0.25, _rot(2, 100.0), conv=1), _left(5, 1, 64, 128, 0.125, _rot(32, 1e5), conv=4, chunk=16),
         _left(3, 1, 20, 20, 0.25, _rot(20, 1000.0), conv=5, chunk=50)]


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("m", LEFTS, ids=lambda m: label(m) + f"c{m.get('conv')}m{(m.get('mask') or {}).get('size')}")
def test_chunked_attention_alone(dtype, m):
    """Every position has edges of its own (its chunk's, the convolution's reach), so comparing all positions under all cuts covers them in
    prompts and in decoding; then a slot that is used again, whose convolution must see nothing of the request before."""
    rt, hidden, T = runtime(dtype), 48, 150
    w = drawn("left", hidden, m, 5)
    x = inputs(T, hidden, 6)
    want = plain.chunked_attention(x.double(), doubles(w), "m", m, 1e-5)
    part = part_of("left", m, hidden, rt, w)
    for page in (8, 16):
        for cuts in cuts_for(T) + [[1] * T]:
            runner = harness([part.cache_need()], rt, page=page)
            close(feed([part], runner, x.to(rt.dtype), cuts)[0], want, dtype, f"page {page}, cuts {cuts[:4]}")
            runner.cache.check()
    for req in ("a", "b"):
        close(feed([part], runner, x.to(rt.dtype), [1, 2, 1, 50, 1, 1, T - 56], req=req)[0], want, dtype, req)


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("d", [16, 64])
@pytest.mark.parametrize("last", [159, 160, 161, 199])
@pytest.mark.parametrize("at", [0, 79, 80, 119, 120, 121, 158, 159, 160])
def test_one_key_stands_out_at_the_chunks_edges(dtype, d, last, at):
    """Chunks of 40: the query at ``last`` (the last of a chunk, the first, the second, the last again) meets its own direction at ``at``: its chunk's first
    position, the last of the chunk before, far behind, or (beyond ``last``) not yet there."""
    rt, hidden, T = runtime(dtype), 32, 200
    m = _left(2, 2, d, 16, 14.0 / d, _rot(2, 1e9), chunk=40)
    w = drawn("left", hidden, m, 3)
    w["m.k"], w["m.k.b"], w["m.k.norm"] = w["m.q"].clone(), w["m.q.b"].clone(), w["m.q.norm"].clone()
    x = torch.randn(T, hidden, generator=torch.Generator().manual_seed(at + last))
    x[at] = x[last] * 1.5
    x = bf(x)
    want = plain.chunked_attention(x.double(), doubles(w), "m", m, 1e-5)
    part = part_of("left", m, hidden, rt, w)
    for cuts in ([T], [last, T - last], [100] + [1] * 100, portions(T, [16, 2, 5])):
        runner = harness([part.cache_need()], rt, page=8)
        got = feed([part], runner, x.to(rt.dtype), cuts)[0]
        close(got[last - 5:last + 1], want[last - 5:last + 1], dtype, f"last {last}, at {at}, cuts {cuts[:3]}")


# ---- gated linear attention -----------------------------------------------------------------------------------------------------------

RIGHTS = [(_right(3, 6, 9, 8.0), 5), (_right(4, 64, 64, 16.0), 16), (_right(2, 32, 48, 4.0), 40), (_right(1, 128, 128, 16.0), 32), (_right(2, 16, 256, 1.0), 16),
          (_right(1, 128, 12, 32.0), 8), (_right(3, 48, 80, 5.0), 24), (_right(2, 160, 32, 16.0), 16), (_right(2, 64, 144, 10.0), 17), (_right(1, 80, 16, 2.0), 130)]


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("m,rank", RIGHTS, ids=lambda v: label(v) if isinstance(v, dict) else f"r{v}")
def test_gated_linear_attention_alone(dtype, m, rank):
    rt, hidden, T = runtime(dtype), 48, 150
    w = drawn("right", hidden, m, 11, rank)
    x = inputs(T, hidden, 12)
    want = plain.gated_linear_attention(x.double(), doubles(w), "m", m, 1e-5)
    part = part_of("right", m, hidden, rt, w)
    for cuts in cuts_for(T) + [[1] * T, portions(T, [17, 3, 1, 1, 2]), portions(T, [64, 1, 2]), portions(T, [63, 65, 9])]:
        runner = harness([part.cache_need()], rt)
        close(feed([part], runner, x.to(rt.dtype), cuts)[0], want, dtype, f"cuts {cuts[:4]}")
    runner = harness([part.cache_need()], rt)                         # a slot that is used again starts from nothing
    for req in ("a", "b", "c"):
        close(feed([part], runner, x.to(rt.dtype), [50, 1, 1, T - 52], req=req)[0], want, dtype, req)


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("d,dv", [(16, 12), (32, 32), (64, 144)])
def test_a_slow_state_remembers_the_first_tokens(dtype, d, dv):
    """Decays so near 1 that after 400 tokens the first ones still show: a state that is dropped or zeroed between steps is seen at once.  Later tokens
    bring small keys."""
    rt, hidden, T = runtime(dtype), 32, 400
    m = _right(2, d, dv, 16.0)
    w = drawn("right", hidden, m, 13, 16)
    w["m.a2.b"] = bf(torch.full((2 * d,), 9.0))
    direction = torch.randn(hidden, generator=torch.Generator().manual_seed(15))
    # (keys see only the direction, which the later tokens have little of)
    w["m.k"] = bf(torch.randn(2 * d, 1, generator=torch.Generator().manual_seed(17)) * direction[None] / hidden ** 0.5)
    x = torch.randn(T, hidden, generator=torch.Generator().manual_seed(14))
    x -= (x @ direction)[:, None] * direction[None] / direction.pow(2).sum() * 0.995
    x[:3] += 3.0 * direction
    x = bf(x)
    want = plain.gated_linear_attention(x.double(), doubles(w), "m", m, 1e-5)
    without = plain.gated_linear_attention(x.double()[3:], doubles(w), "m", m, 1e-5)
    assert (want[-1] - without[-1]).abs().max() > 0.3 * want[-1].abs().max()          # the first tokens do matter at the end
    part = part_of("right", m, hidden, rt, w)
    for cuts in ([T], [T - 100] + [1] * 100, portions(T, [64, 1, 2]), portions(T, [130, 7])):
        runner = harness([part.cache_need()], rt)
        # (where a query is nearly at right angles to the one direction the keys have, the head's norm magnifies rounding: a few rows)
        close(feed([part], runner, x.to(rt.dtype), cuts)[0], want, dtype, f"cuts {cuts[:3]}", 0.03, exact=1e-2)


@pytest.mark.parametrize("chunked", [False, True], ids=["scan", "chunked"])
@pytest.mark.parametrize("bias,tau", [(9.0, 16.0), (1.0, 16.0), (-4.0, 1.0), (-90.0, 1.0)])
@pytest.mark.parametrize("d,dv", [(32, 144), (64, 160), (128, 256), (64, 64), (128, 128)])
def test_the_recurrence_is_exact_for_weak_and_strong_decays(chunked, bias, tau, d, dv):
    """The recurrence's own arithmetic is 32-bit: on bf16 inputs taken as they are the result and the final state agree with float64 to about
    1e-4, whatever the decays: from nothing forgotten to everything forgotten within a token (where the exponent of a chunk's sums reaches
    thousands), weak and strong channels side by side.  (Where one kernel norms and gates a head too, the state is looked at alone.)"""
    from marin_b200.engine import StepEntry
    from marin_b200.kernels import ops

    H, T, rank = 3, 200, 32
    g = torch.Generator().manual_seed(int(abs(bias) * 10) + d)
    q, k = (bf(torch.randn(T, H * d, generator=g)) for _ in range(2))
    v, low = bf(torch.randn(T, H * dv, generator=g)), bf(torch.randn(T, rank, generator=g))
    w2, b = bf(torch.randn(H * d, rank, generator=g) * 0.3), bias + 2.0 * torch.randn(H * d, generator=g)
    b[::3] = 40.0                                                     # every third channel never forgets
    start = torch.randn(H, d, dv, generator=g)
    alpha = torch.exp(-torch.nn.functional.softplus(-(low.double() @ w2.double().T + b.double()), threshold=1e9) / tau).reshape(T, H, d)
    ends = []
    want = plain.linear_recurrence(q.double().reshape(T, H, d) * d ** -0.5, k.double().reshape(T, H, d), v.double().reshape(T, H, dv), alpha, start.double(), ends)
    rt = runtime("bfloat16")
    norm_w = torch.ones(dv, device=DEV)
    rows = torch.cat([q, k, v, torch.zeros_like(v), low], dim=1).to(DEV).contiguous()
    cols = [0, H * d, 2 * H * d, 2 * H * d + H * dv, 2 * H * d + 2 * H * dv, rows.shape[1]]
    whole = ops._gla_slice(dv) == dv
    for cuts in ([T], portions(T, [64]), portions(T, [65, 100, 2]), portions(T, [9, 3])):
        state = torch.zeros(5, H, d, dv, device=DEV)
        state[:] = start.to(DEV)
        runner = harness([], rt)
        runner.begin("r")
        outs, at = [], 0
        for n in cuts:
            ctx = runner.build_context([StepEntry("r", [0] * n, [])])
            part = [rows[at:at + n, a:e] for a, e in zip(cols[:-1], cols[1:])]
            inp = ops.GlaInputs(part[0], part[1], part[2], part[3], part[4], w2.to(DEV), b.to(DEV), 1.0 / tau)
            if chunked:
                out = torch.empty(n, H * dv, device=DEV, dtype=torch.bfloat16)
                ops.gla_chunked(inp, state, ctx, ctx.state_slots, "silu", norm_w, 1e-5, 1.0, out, H, d, dv)
                outs.append(None if whole else ctx.workspace.get("gla_o", (n, H * dv), torch.float32).cpu())
            else:
                o = torch.full((n, H * dv), float("nan"), device=DEV)
                ops.gla_scan(inp, state, ctx, ctx.state_slots, o, H, d, dv)
                outs.append(o.cpu())
            runner.cache.commit("r", at + n)
            at += n
        runner.end("r")
        slot = next(i for i in range(5) if not torch.equal(state[i].cpu(), start))
        checks = [("state", state[slot].double().cpu(), ends[0])]
        if outs[0] is not None:
            checks.append(("o", torch.cat(outs).double().reshape(T, H, dv), want))
        for name, a, e in checks:
            err, size = (a - e).abs().max(), e.pow(2).mean().sqrt()
            assert torch.isfinite(a).all() and err <= 4e-4 * size + 1e-6, (name, cuts[:3], float(err), float(size))


def test_several_requests_in_one_step_share_the_chunks_memory():
    """Portions of unequal length and single tokens in one step, through a whole parallel mixer: every request's result is what it gets alone."""
    from marin_b200.config.punolix import _mixer as parse
    from marin_b200.engine import StepEntry
    from marin_b200.models.punolix import _mixer as spec_of
    from marin_b200.parts import lookup

    hidden, rt = 48, runtime("bfloat16")
    raw = _parallel(_left(4, 2, 32, 32, 0.2, _rot(32, 1000.0), conv=4, chunk=30), _right(4, 32, 32, 8.0), 0.7, 0.8)
    w = {k.replace("m.", "m.left.", 1): v for k, v in drawn("left", hidden, raw["left"], 1).items()}
    w.update({k.replace("m.", "m.right.", 1): v for k, v in drawn("right", hidden, raw["right"], 2, 12).items()})
    spec = spec_of("parallel", parse("parallel", dict(raw, right=dict(raw["right"], decay_rank=12)), ""), hidden, 1e-5)
    part = lookup("mixer", spec.kind)(name="m", **spec.params)
    part.load({k: v.clone() for k, v in w.items()}, rt)
    lengths = {"a": [130, 1, 1, 40], "b": [1, 1, 70, 1], "c": [2, 65, 63, 2], "d": [64, 128, 1, 9]}
    xs = {r: inputs(sum(n), hidden, i) for i, (r, n) in enumerate(lengths.items())}
    runner = harness([part.cache_need()], rt)
    for r in lengths:
        runner.begin(r)
    at, got = {r: 0 for r in lengths}, {r: [] for r in lengths}
    for step in range(4):
        for r in lengths:
            runner.cache.reserve(r, at[r] + lengths[r][step])
        ctx = runner.build_context([StepEntry(r, [0] * lengths[r][step], []) for r in lengths])
        rows = torch.cat([xs[s.req_id][at[s.req_id]:at[s.req_id] + s.count] for s in sorted(ctx.spans, key=lambda s: s.start)]).to(DEV).contiguous()
        residual = torch.zeros(rows.shape[0], hidden, device=DEV)
        part.forward(rows, ctx, runner.views.view(0, ctx), residual)
        for s in ctx.spans:
            got[s.req_id].append(residual[s.start:s.start + s.count].cpu())
            at[s.req_id] += s.count
            runner.cache.commit(s.req_id, at[s.req_id])
    for r in lengths:
        want = plain.mixer({"type": "parallel", "mixer": raw}, xs[r].double(), doubles(w), "m", 1e-5)
        close(torch.cat(got[r]), want, "bfloat16", r)


# ---- the layer: one norm, two sublayers, a multiplier, rows that ride on the norm -----------------------------------------------------------------

@pytest.mark.parametrize("join", [False, True], ids=["own", "joined"])
@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("kind", ["attention", "parallel", "odd", "alone"])
def test_a_layer_alone(dtype, kind, join, monkeypatch):
    """Mixer and feed-forward on one norm, with and without shared products; "odd": widths that no shared product takes; "alone": no feed-forward."""
    from marin_b200.config.punolix import PunolixLayer
    from marin_b200.engine import StepEntry
    from marin_b200.models.punolix import _feedforward, _mixer
    from marin_b200.parts.block import ParallelBlock
    from marin_b200.parts.spec import LayerSpec, PartSpec
    from punolix_models import random_weights

    monkeypatch.setattr(ParallelBlock, "join_products", join)
    hidden, T, mult = 64, 130, 0.3
    raw = {"attention": _layer("attention", _diff(6, 3, 32, 64, 0.2, _rot(32, 700.0), 0.5, softcap=9.0), 96),
           "parallel": _layer("parallel", _parallel(_left(4, 2, 32, 48, 0.2, _rot(32, 700.0), conv=4, chunk=40), _right(3, 32, 48, 8.0), 0.4, -1.3), 80),
           "odd": _layer("parallel", _parallel(_left(3, 1, 12, 10, 0.3, _rot(8, 700.0), conv=3, chunk=40), _right(3, 6, 9, 8.0), 0.4, -1.3), 52),
           "alone": _layer("parallel", _parallel(_left(4, 2, 32, 48, 0.2, _rot(32, 700.0), conv=2), _right(3, 32, 48, 8.0), 0.9, 0.6), None)}[kind]
    w = {k: v for k, v in random_weights({"width": hidden, "vocab": 8, "layers": [raw]}, 4).items() if k.startswith("l0.")}
    if raw["type"] == "parallel":
        raw["mixer"]["right"]["decay_rank"] = w["l0.mix.right.a1"].shape[0]
    layer = PunolixLayer.parse(raw, 0)
    rt = runtime(dtype)
    spec = LayerSpec(block="parallel_prenorm", norm=PartSpec("rmsnorm", {"dim": hidden, "eps": 1e-5, "tensor": ""}), mixer=_mixer(layer.type, layer.mixer, hidden, 1e-5),
                     feedforward=_feedforward(layer.mlp, hidden), prefix="l0", names={"norm1": "norm1", "mixer": "mix", "feedforward": "mlp"}, block_params={"residual_mult": mult})
    block = ParallelBlock(spec)
    left = {k: v.clone() for k, v in w.items()}
    block.load(left, rt)
    assert not left and (block.w_in is not None) == (join and dtype == "bfloat16" and kind in ("attention", "parallel"))
    x = torch.randn(T, hidden, generator=torch.Generator().manual_seed(3))
    want = plain.parallel_layer(raw, x.double(), doubles(w), "l0", 1e-5, mult)
    for cuts in cuts_for(T):
        runner = harness([block.mixer.cache_need()], rt)
        runner.begin("r")
        got, at = [], 0
        for n in cuts:
            runner.cache.reserve("r", at + n)
            ctx = runner.build_context([StepEntry("r", [0] * n, [])])
            rows = x[at:at + n].to(DEV).contiguous()
            block.forward(rows, ctx, runner.views.view(0, ctx))
            got.append(rows.cpu())
            runner.cache.commit("r", at + n)
            at += n
        runner.end("r")
        close(torch.cat(got) - x, want - x.double(), dtype, f"cuts {cuts[:4]}")


@pytest.mark.parametrize("T", [1, 7, 16, 33, 64, 100, 129, 300, 1030])
@pytest.mark.parametrize("K,P,I,act", [(64, 0, 48, "gelu_tanh"), (128, 96, 64, "gelu_tanh"), (520, 416, 336, "silu"), (256, 32, 16, "relu"), (512, 1056, 3200, "gelu_tanh")])
def test_gated_products_with_a_plain_part(T, K, P, I, act):
    """The activation in the epilogue, times a factor, into a column block of a wider buffer, beside the plain rows of the same product."""
    from marin_b200.kernels import ops

    g = torch.Generator().manual_seed(T + K)
    x, wp, wg, wu = (bf(torch.randn(n, K, generator=g) / (1 if i == 0 else K ** 0.5)) for i, n in enumerate((T, P, I, I)))
    w = torch.cat([wp, ops.interleave_gate_up(wg * 2, wu)], dim=0).to(DEV).contiguous()
    wide = torch.full((T, I + 24), 7.0, device=DEV, dtype=torch.bfloat16)
    rows = torch.empty(T, P, device=DEV, dtype=torch.bfloat16) if P else None
    ops.gemm_glu_rows(x.to(DEV), w, rows, wide[:, 16:16 + I], act, 0.3)
    z, u = x.double() @ (wg * 2).double().T, x.double() @ wu.double().T
    want = {"gelu_tanh": plain.gelu_tanh, "silu": plain.silu, "relu": lambda v: v.clamp(min=0)}[act](z) * u * 0.3
    assert bool((wide[:, :16] == 7).all()) and bool((wide[:, 16 + I:] == 7).all())
    for got, ref in ((wide[:, 16:16 + I], want),) + (((rows, x.double() @ wp.double().T),) if P else ()):
        err = (got.double().cpu() - ref).abs()
        assert bool((err <= 2 ** -8 * ref.abs() + 2e-5).all()), float(err.max())


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("n,I", [(44, 60), (64, 96)])
def test_a_gelu_feed_forward(dtype, n, I):
    from marin_b200.parts import lookup

    rt, T = runtime(dtype), 50
    g = torch.Generator().manual_seed(2)
    w = {"f.gate": bf(2 * mat(g, I, n)), "f.up": bf(mat(g, I, n)), "f.down": bf(mat(g, n, I))}
    part = lookup("feedforward", "swiglu")(hidden=n, intermediate=I, name="f", activation="gelu_tanh", names=("gate", "up", "down"), out_scale=-0.7)
    part.load({k: v.clone() for k, v in w.items()}, rt)
    x = inputs(T, n, 3)
    close(feed([part], harness([], rt), x.to(rt.dtype), [T], mixer=False)[0], -0.7 * plain.feed_forward(x.double(), doubles(w), "f"), dtype)


@pytest.mark.parametrize("n", [44, 512, 2560, 8192, 9000])
def test_rows_that_ride_on_a_norm_and_rows_that_enter_the_stream(n):
    from marin_b200.kernels import ops

    g = torch.Generator().manual_seed(n)
    x, y, w, b = torch.randn(13, n, generator=g), torch.randn(13, n, generator=g), torch.randn(n, generator=g), torch.randn(n, generator=g)
    rows, out = x.to(DEV), torch.empty(13, n, device=DEV)
    ops.rmsnorm(rows, w.to(DEV), 1e-5, out, then_add=b.to(DEV))
    close(out, x.double() / plain.rms(x.double(), 1e-5) * w.double(), "float32", "norm", exact=1e-5)
    assert torch.equal(rows.cpu(), x + b)
    again = torch.empty(13, n, device=DEV)
    ops.rmsnorm(x.to(DEV), w.to(DEV), 1e-5, again)
    assert torch.equal(again, out)
    ops.stream_enter(rows, y.to(DEV), w.to(DEV), rows)
    assert torch.equal(rows.cpu(), ((x + b) + y) + w)
    ops.stream_enter(rows, None, None, again)
    assert torch.equal(again, rows)


# ---- whole models -----------------------------------------------------------------------------------------------------------------------

class Case:
    """A model folder loaded in one dtype, the plain logits of its requests, and runners over it."""

    def __init__(self, tmp, name, dtype):
        from marin_b200.engine import load_model

        self.name, self.dtype, self.raw = name, dtype, CONFIGS[name]
        self.dir = make_model_dir(str(tmp / f"{name}{dtype}"), name, seed=31)
        self.w = plain.read_weights(self.dir)
        rng = random.Random(5)
        self.tokens = {rid: random_prompt(rng, self.raw["vocab"], n) for rid, n in LENGTHS[name].items()}
        self.want = {rid: plain.forward(self.raw, self.w, t) for rid, t in self.tokens.items()}
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
        # (32-bit: a head's norm magnifies rounding where the first tokens' q . k nearly cancel)
        close(got, self.want[rid], self.dtype, what, self.loose, None, 0.1, 0.04, 1e-3)


@pytest.fixture(scope="module", params=[(n, d) for n in CONFIGS for d in DTYPES], ids=lambda p: f"{p[0]}-{p[1]}")
def case(request, tmp_path_factory):
    return Case(tmp_path_factory.mktemp("punolix"), *request.param)


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
        close(got[i + 1], want[i], case.dtype, f"after layer run {i}", case.loose, None, 0.1, 0.04)


def test_whole_prompts_and_the_first_tokens(case):
    runner = case.runner(64)
    for rid, tokens in case.tokens.items():
        case.close(run_whole(runner, rid, tokens), rid, f"{rid} whole")
    runner.cache.check()


@pytest.mark.parametrize("graphs", [False, True])
def test_prefill_then_token_by_token(case, graphs):
    """Most of a prompt in one step and the rest one token at a time, eagerly and from captured graphs: a tail long enough for
    every chunk to pass wholly over decoded tokens; and a request decoded from its very first token."""
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
    token whose plain logit lies within 1e-3 (32-bit) or 0.15 (16-bit) of the largest counts as first)."""
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
            logits = plain.forward(case.raw, case.w, seq)[-1]
            assert logits[token] >= logits.max() - slack, (len(seq), token, int(logits.argmax()))
            seq.append(token)


def test_preempted_requests_start_again_from_their_first_token(tmp_path):
    """So few pages that a running request is preempted: it comes back with prompt and generated tokens recomputed, its states as
    at a sequence's start, and produces what it produces alone."""
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


def test_the_command_line_takes_a_punolix_folder(tmp_path):
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
    for stage in ("embedding", "pass entered", "norm", "inputs, gate|up", "heads", "attention", "gated linear", "o|down", "head", "sampling"):
        assert stage in e.stdout, stage
