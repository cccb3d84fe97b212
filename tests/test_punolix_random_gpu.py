"""Punolix configurations drawn at random (any order of the two layer kinds; head counts and sizes inside and outside what the tensor-core
kernels take; chunks from one position to longer than the sequence; with and without caps, convolutions, scaled frequencies; loops anywhere, of
any number of passes, and none) through the step function in float32 and in bfloat16, with pages of 16: whole, with a decoded tail, in
changing portions and in a mixed batch with few pages, against the plain implementation.  Every size a configuration allows must run,
through a fused path or a plain one, and give the same result.  ``MARIN_B200_RANDOM_SEEDS`` widens the sweep."""
import math
import os
import random

import pytest

import plain_punolix as plain
from helpers import mixed_schedule, random_prompt, run_mixed, run_portions, run_whole
from part_harness import DTYPES, close, runtime
from punolix_models import _diff, _layer, _left, _parallel, _right, _rot, random_weights, write_model

pytestmark = pytest.mark.gpu
SEEDS = int(os.environ.get("MARIN_B200_RANDOM_SEEDS", "6"))
PAGE = 16


def draw_rot(rng: random.Random, dim: int, scaled: bool) -> dict:
    scaling = rng.choice([None, (4.0, 1.0, 4.0, 64), (16.0, 0.5, 2.0, 200)]) if scaled else None
    return _rot(rng.choice([dim, dim, dim // 2 // 2 * 2]), rng.choice([300.0, 10000.0, 1e6]), scaling)


def draw_layer(rng: random.Random) -> dict:
    ff = rng.choice([None, 48, 64, 200, 256])
    if rng.random() < 0.55:
        kv = rng.choice([1, 2, 3])
        dim = rng.choice([8, 12, 16, 32, 32, 64, 64, 128])
        return _layer("attention", _diff(kv * rng.choice([1, 2, 4]), kv, dim, rng.choice([2 * dim, 2 * dim, dim, 64, 40]) if dim <= 64 else rng.choice([64, 128]),
                                         rng.choice([0.7, 1.0, 1.3]) / math.sqrt(dim), draw_rot(rng, dim, False), rng.choice([0.2, 0.4, 0.8]), rng.choice([None, 5.0, 30.0])), ff)
    kv = rng.choice([1, 2, 4])
    dim = rng.choice([16, 24, 48, 64, 64, 128])
    left = _left(kv * rng.choice([1, 2, 4]), kv, dim, rng.choice([dim, 64, 40]), 1.0 / math.sqrt(dim), draw_rot(rng, dim, True), rng.choice([None, 1, 2, 4, 4, 6]),
                 rng.choice([None, 1, 16, 33, 64, 100, 300]))
    d, dv = rng.choice([(6, 32), (16, 16), (16, 9), (32, 32), (32, 48), (64, 32), (64, 96), (128, 64), (128, 128), (48, 160)])
    return _layer("parallel", _parallel(left, _right(rng.choice([1, 2, 3]), d, dv, rng.choice([1.0, 8.0, 16.0])), rng.choice([1.0, 0.5, -0.8]), rng.choice([1.0, 0.7, 1.3])), ff)


def draw(rng: random.Random) -> dict:
    n = rng.randint(2, 4)
    raw = {"architecture": "Punolix", "vocab": rng.choice([97, 300, 512]), "width": rng.choice([64, 96, 128, 200]), "norm": {"eps": rng.choice([1e-6, 1e-5])},
           "layers": [draw_layer(rng) for _ in range(n)], "embedding": {"scale": rng.choice([1.0, 11.3])}, "residual_mult": rng.choice([1.0, 0.6, 0.25])}
    if rng.random() < 0.8:
        start = rng.randrange(n)
        raw["loop"] = {"start": start, "stop": rng.randint(start + 1, n), "times": rng.choice([1, 2, 2, 3])}
    return raw


# Sizes nearer a real model's: wide heads, two maps of 64 over values of 128 in groups of four heads, a decay rank of 16 over heads of 128 x 128.
LARGER = {
    "architecture": "Punolix", "vocab": 1000, "width": 512, "norm": {"eps": 1e-5}, "embedding": {"scale": 22.0}, "residual_mult": 0.4, "loop": {"start": 1, "stop": 2, "times": 3},
    "layers": [
        _layer("attention", _diff(8, 2, 64, 128, 0.125, _rot(64, 10000.0), 0.2, 50.0), 1024),
        _layer("parallel", _parallel(_left(8, 2, 128, 128, 128 ** -0.5, _rot(128, 500000.0, (8.0, 1.0, 4.0, 64)), 4, 96), _right(4, 128, 128, 16.0), 0.6, 0.7), 768),
        _layer("attention", _diff(4, 4, 64, 128, 0.125, _rot(64, 10000.0), 0.5), None),
    ],
}


def compare(tmp_path, raw, dtype, weight_seed, rng, lengths, what):
    from marin_b200.cache import CacheManager
    from marin_b200.engine import Runner, load_model
    from marin_b200.kernels import build

    d = write_model(str(tmp_path / "m"), raw, random_weights(raw, weight_seed))
    w = plain.read_weights(d)
    tokens = {rid: random_prompt(rng, raw["vocab"], n) for rid, n in lengths.items()}
    want = {rid: plain.forward(raw, w, t) for rid, t in tokens.items()}
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
        close(got, want[rid], dtype, f"{what}: {rid} {how}", 0.03 if dtype == "bfloat16" else 0.0, None, 0.12, 0.05, 5e-4)

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
def test_a_random_punolix_configuration(tmp_path, seed, dtype):
    rng = random.Random(4000 + seed)
    raw = draw(rng)
    lengths = {"a": rng.choice([150, 190, 230]), "b": rng.choice([1, 2, 17]), "c": rng.choice([64, 65, 129]), "d": 40, "e": 90}
    compare(tmp_path, raw, dtype, 70 + seed, rng, lengths, f"seed {seed}, {[layer['type'] for layer in raw['layers']]}")


@pytest.mark.parametrize("dtype", DTYPES)
def test_a_larger_punolix_configuration(tmp_path, dtype):
    compare(tmp_path, LARGER, dtype, 5, random.Random(77), {"a": 170, "b": 3, "c": 65}, "larger")
