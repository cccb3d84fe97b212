"""Pununex configurations drawn at random (any order of the two layer kinds; attention and delta head counts and sizes inside and
outside what the tensor-core kernels take; windows from one position to longer than the sequence, no, few and more kept positions than
the window is long, with and without a cap; one to seven taps; dense, routed and no feed-forwards, groups, identity outputs, with and
without a bigram embedding) through the step function in float32 and in bfloat16, with pages of 16: whole, with a decoded tail, in
changing portions and in a mixed batch with few pages, against the plain implementation.  Every size a configuration allows must
run, through a fused path or a plain one, and give the same result.  ``MARIN_B200_RANDOM_SEEDS`` widens the sweep."""
import math
import os
import random

import pytest
import torch

import plain_pununex as plain
from helpers import mixed_schedule, random_prompt, run_mixed, run_portions, run_whole
from part_harness import DTYPES, close, runtime
from pununex_models import _attn, _delta, _dense, _moe, _parallel, random_weights, write_model

pytestmark = pytest.mark.gpu
SEEDS = int(os.environ.get("MARIN_B200_RANDOM_SEEDS", "6"))
PAGE = 16


def draw_attention(rng: random.Random) -> dict:
    kv = rng.choice([1, 2, 3, 4])
    heads = kv * rng.choice([1, 2, 4, 8])
    dim = rng.choice([16, 24, 48, 64, 64, 128])
    vdim = rng.choice([dim, dim, 16, 40, 80])
    return _attn(heads, kv, dim, vdim, rng.choice([0.7, 1.0]) / math.sqrt(dim), size=rng.choice([None, 1, 5, 16, 33, 64, 100, 300]),
                 keep=rng.choice([None, 0, 1, 4, 16, 17, 70]), softcap=rng.choice([None, 2.0, 10.0, 50.0]))


def draw_delta(rng: random.Random) -> dict:
    kv = rng.choice([1, 2, 3])
    dim, vdim = rng.choice([(6, 32), (16, 16), (16, 9), (32, 32), (32, 48), (32, 40), (64, 32), (64, 96), (128, 64), (128, 32)])
    return _delta(kv * rng.choice([1, 1, 2, 3]), kv, dim, vdim, rng.choice([1, 2, 3, 4, 4, 7]))


def draw_layer(rng: random.Random) -> dict:
    experts, identity = rng.choice([2, 3, 4, 6, 8, 16]), rng.choice([0, 0, 2, 4])
    n = experts + identity
    count = rng.choice([c for c in (1, 2, 4) if n % c == 0])
    keep = rng.randint(1, count)
    top = min(n // count * keep, rng.choice([1, 2, 4]))
    moe = _moe(rng.choice([32, 64, 96, 128]), experts, top, identity=rng.choice([identity, identity or None]), groups=(count, keep) if count > 1 else None,
               scale=rng.choice([1.0, 0.4, 2.5]), shared=rng.choice([None, 64, 96]))
    mlp = rng.choice([None, _dense(rng.choice([48, 64, 200])), moe, moe])
    if rng.random() < 0.4:
        return {"type": "delta", "mixer": draw_delta(rng), "mlp": mlp}
    return {"type": "parallel", "mixer": _parallel(draw_attention(rng), draw_delta(rng), rng.choice([1.0, 0.5, -0.8]), rng.choice([1.0, 0.7, 1.3])), "mlp": mlp}


def draw(rng: random.Random) -> dict:
    raw = {"architecture": "Pununex", "vocab": rng.choice([97, 300, 512]), "width": rng.choice([64, 96, 128, 200, 256]), "norm": {"eps": rng.choice([1e-6, 1e-5])},
           "layers": [draw_layer(rng) for _ in range(rng.randint(2, 5))]}
    if rng.random() < 0.8:
        raw["embedding"] = {"bigram": {"buckets": rng.choice([1, 53, 601]), "mul_prev": rng.choice([1, 29, 40503]), "mul_cur": rng.choice([1, 17, 65599])}}
    return raw


# Sizes nearer a real model's: wide heads, many experts in groups, delta heads of 128 x 128 and of 64 x 256.
LARGER = {
    "architecture": "Pununex", "vocab": 1000, "width": 512, "norm": {"eps": 1e-5}, "embedding": {"bigram": {"buckets": 4001, "mul_prev": 7919, "mul_cur": 31}},
    "layers": [
        {"type": "parallel", "mixer": _parallel(_attn(16, 4, 128, 128, 1.0 / math.sqrt(128), size=90, keep=5, softcap=30.0), _delta(4, 4, 128, 128, 4), 0.6, 0.4),
         "mlp": _dense(1024)},
        {"type": "delta", "mixer": _delta(8, 2, 64, 256, 4), "mlp": _moe(256, 24, 6, identity=8, groups=(8, 3), scale=2.5, shared=512)},
        {"type": "parallel", "mixer": _parallel(_attn(8, 8, 64, 64, 0.125, size=64, keep=80, softcap=12.0), _delta(6, 2, 64, 64, 3), 1.0, 1.0), "mlp": _moe(128, 8, 2)},
    ],
}


def compare(tmp_path, raw, dtype, weight_seed, rng, lengths, what):
    from marin_b200.cache import CacheManager
    from marin_b200.engine import Runner, load_model
    from marin_b200.kernels import build

    d = write_model(str(tmp_path / "m"), raw, random_weights(raw, weight_seed))
    w = plain.read_weights(d)
    tokens = {rid: random_prompt(rng, raw["vocab"], n) for rid, n in lengths.items()}
    want, safe = {}, {}
    for rid, t in tokens.items():
        margins = []
        want[rid] = plain.forward(raw, w, t, None, margins)
        tight = torch.stack(margins).min(dim=0).values < 0.03 if margins else torch.zeros(len(t), dtype=torch.bool)
        safe[rid] = int(torch.nonzero(tight)[0]) if bool(tight.any()) else len(t)
    rt = runtime(dtype)
    _, model = load_model(d, rt)
    build.build_for(model, rt.dtype, verbose=False)            # (its kernels side by side, not one after the other at first use)

    def runner(num_pages, graphs=False):
        cache = CacheManager(model.cache_needs(), [e.cache_of for e in model.spec.schedule], PAGE, num_pages, 4)
        cache.allocate(rt.device, rt.dtype)
        r = Runner(model, cache, rt, 512)
        if graphs:
            r.enable_graphs((1, 2, 4))
        return r

    def same(got, rid, how):
        close(got, want[rid], dtype, f"{what}: {rid} {how}", 0.03 if dtype == "bfloat16" else 0.0, safe[rid], 0.12, 0.05, 5e-4)

    r = runner(64, graphs=True)
    for rid in ("a", "c"):
        same(run_whole(r, rid, tokens[rid]), rid, "whole")
    n = lengths["a"]
    same(run_portions(r, "at", tokens["a"], [n - 40] + [1] * 40), "a", "with a decoded tail")
    same(run_portions(r, "ap", tokens["a"], [63, 2, 1, 30, n - 96]), "a", "in portions")
    pool = sum(sorted((-(-k // PAGE) for k in lengths.values()), reverse=True)[:4])
    r = runner(pool)
    got = run_mixed(r, tokens, mixed_schedule(random.Random(weight_seed), lengths, max_live=4, decode_tail=8))
    for rid in tokens:
        same(got[rid], rid, "in a mixed batch")
    r.cache.check()


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("seed", range(SEEDS))
def test_a_random_pununex_configuration(tmp_path, seed, dtype):
    rng = random.Random(3000 + seed)
    raw = draw(rng)
    lengths = {"a": rng.choice([150, 190, 230]), "b": rng.choice([1, 2, 17]), "c": rng.choice([64, 65, 129]), "d": 40, "e": 90}
    compare(tmp_path, raw, dtype, 70 + seed, rng, lengths, f"seed {seed}, {[layer['type'] for layer in raw['layers']]}")


@pytest.mark.parametrize("dtype", DTYPES)
def test_a_larger_pununex_configuration(tmp_path, dtype):
    compare(tmp_path, LARGER, dtype, 5, random.Random(77), {"a": 170, "b": 3, "c": 65}, "larger")
