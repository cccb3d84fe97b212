"""What the tests of single parts and of whole models share: running a part over rows of a request in portions with its own
cache, comparing with float64 rows at stated tolerances, and loading a model folder once for many schedules.

Tolerances.  float32: |diff| <= exact (1 + |ref|), the reference being float64.  bfloat16: the root mean square of the difference
over a row at most ``row_bound`` of the reference's own root mean square and ``mean_bound`` on average, ``loose_rows`` of the rows
beyond.  ``safe``: the first row behind which a choice of experts is a close call in float64 (in 16 bits it may fall the other way,
and the states and keys behind it carry that on): from there on rows must only stay numbers of the reference's size.
"""
from __future__ import annotations

import math
import os
from types import SimpleNamespace

import torch

from helpers import portions

DEV = torch.device(os.environ.get("MARIN_B200_TEST_DEVICE", "cuda:0"))
DTYPES = ["float32", "bfloat16"]


def torch_dtype(name):
    return torch.float32 if name == "float32" else torch.bfloat16


def runtime(dtype):
    from marin_b200.parts import Runtime

    return Runtime(DEV, torch_dtype(dtype))


def bf(t):
    return t.to(torch.bfloat16)


def mat(g, r, c, gain=1.0):
    return torch.randn(r, c, generator=g) * gain / math.sqrt(c)


def close(got, want, dtype, what="", loose_rows=0.0, safe=None, row_bound=0.06, mean_bound=0.03, exact=2e-4):
    got, want = got.detach().double().cpu(), want.double()
    assert got.shape == want.shape, (what, got.shape, want.shape)
    assert bool(torch.isfinite(got).all()), f"{what}: a result that is not a number"
    wide = str(dtype).endswith("float32")
    if safe is not None and safe < got.shape[0] and not wide:
        scale = want.pow(2).mean().sqrt()
        rest = (got[safe:] - want[safe:]).reshape(got.shape[0] - safe, -1).pow(2).mean(dim=1).sqrt() / scale
        assert rest.median() <= 0.75, f"{what}: behind the first close call the median row is {rest.median():.3e} off"
        got, want = got[:safe], want[:safe]
        if safe == 0:
            return
        if safe < 8:                                   # too few rows for an average: every one within twice the bound
            row_bound, mean_bound = 2 * row_bound, 2 * row_bound
    if wide:
        bad = (got - want).abs() > exact * (1 + want.abs())
        if bad.any():
            first = int(torch.nonzero(bad.reshape(bad.shape[0], -1).any(dim=1))[0])
            raise AssertionError(f"{what}: first wrong row {first} of {got.shape[0]}, max err {(got - want).abs().max():.3e}")
        return
    scale = want.pow(2).mean().sqrt()
    rows = (got - want).reshape(got.shape[0], -1).pow(2).mean(dim=1).sqrt() / scale
    over = rows > row_bound
    allowed = int(math.ceil(loose_rows * rows.numel()))
    if int(over.sum()) > allowed or (bool((~over).any()) and rows[~over].mean() > mean_bound):
        raise AssertionError(f"{what}: {int(over.sum())} of {rows.numel()} rows beyond {row_bound} (first {int(torch.nonzero(over)[0]) if over.any() else -1}, "
                             f"max {rows.max():.3e}), mean of the others {rows[~over].mean():.3e}")


def harness(needs, rt, page=8, pages=80, ctx_len=2048):
    from marin_b200.cache import CacheManager
    from marin_b200.engine import Runner

    cache = CacheManager(list(needs), [None] * len(needs), page, pages, 4)
    cache.allocate(rt.device, rt.dtype)
    return Runner(SimpleNamespace(spec=SimpleNamespace(vocab_size=1 << 30)), cache, rt, ctx_len)


def feed(parts, runner, x, cuts, req="r", mixer=True):
    """Runs ``x`` [T, hidden] through the parts (each on the same input, mixers with their view of the cache) in portions
    ``cuts``; returns what each added to a zero residual."""
    from marin_b200.engine import StepEntry

    runner.begin(req)
    got, at = [[] for _ in parts], 0
    for n in cuts:
        runner.cache.reserve(req, at + n)
        ctx = runner.build_context([StepEntry(req, [0] * n, [])])
        for i, part in enumerate(parts):
            residual = torch.zeros(n, x.shape[1], device=DEV)
            rows = x[at:at + n].to(DEV).contiguous()
            if mixer:
                part.forward(rows, ctx, runner.views.view(i, ctx), residual)
            else:
                part.forward(rows, ctx, residual)
            got[i].append(residual.cpu())
        runner.cache.commit(req, at + n)
        at += n
    runner.end(req)
    assert at == x.shape[0]
    return [torch.cat(g) for g in got]


def cuts_for(T):
    return [[T], [max(T - 40, 1)] + [1] * (T - max(T - 40, 1)), portions(T, [7, 2, 13, 3, 2, 5]), portions(T, [2])]
