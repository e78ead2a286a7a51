"""Fofisun configurations drawn at random (seeded): every size, constant, the order of layers, the loop and what a
configuration may leave out move at once, small odd sizes as well as sizes at which the tensor-core kernels take over, and
each draw goes through the four ways of cutting against the plain model, in 32-bit and in bfloat16."""
import random

import pytest

import harness as h
from fofisun_configs import attention, config, dense, moe, write_model
from test_fofisun_engine import TOL, compare, replay, tokens

pytestmark = pytest.mark.gpu


def draw(rng: random.Random, large: bool) -> dict:
    layers = []
    for _ in range(rng.randrange(1, 5)):
        mlp, kind = None, rng.random()
        ff = rng.choice([64, 96, 128]) if large else rng.choice([1, 2, 8, 16]) * rng.randrange(1, 9)
        if kind < 0.35:
            mlp = dense(ff)
        elif kind < 0.85:
            experts = rng.choice([1, 2, 4, 8, 16]) if large else rng.choice([1, 2, 3, 5, 8, 12, 33])
            top = rng.choice([t for t in (1, 2, 3, 4, 6, 10) if t <= experts])
            mlp = moe(experts, top, ff, rng.choice([0.5, 1.0, 3.0, 7.0]), shared=rng.choice([None, ff, 2 * ff, 24]), shared_limit=rng.choice([None, 0.8, 5.0]))
        kv = rng.choice([1, 1, 2, 3])
        heads = kv * rng.choice([1, 2, 4, 6, 9])
        dim = rng.choice([32, 64, 96]) if large else rng.choice([2, 5, 8, 12, 16, 24, 40, 48])
        vdim = rng.choice([64, 128, 192]) if large else rng.choice([2, 7, 8, 16, 20, 32, 64, 72])
        layers.append(attention(heads, kv, dim, vdim, rng.choice([0.5, 1.0, 2.0]) * dim ** -0.5, rng.choice([0.0, 0.2, 0.5, 0.8]),
                                conv=rng.choice([None, 1, 2, 3, 4, 4, 4, 6]), window=rng.choice([None, 1, 2, 7, 16, 33, 64, 96, 150, 1000]),
                                keep=rng.choice([None, 0, 1, 4, 16, 17, 64, 100]), mlp=mlp))
    n = len(layers)
    loop = None
    if rng.random() < 0.6:
        lo = rng.randrange(n)
        loop = (lo, rng.randrange(lo + 1, n + 1), rng.choice([1, 2, 3]))
    width = rng.choice([256, 320, 384]) if large else rng.choice([2, 3, 8, 16]) * rng.randrange(3, 20)
    return config(rng.randrange(60, 900), width, rng.choice([1e-5, 1e-6, 3e-4]), layers, loop=loop)


@pytest.mark.parametrize("seed,large", [(s, False) for s in range(1, 9)] + [(s, True) for s in range(101, 105)])
def test_a_random_configuration_in_the_four_ways_of_cutting(seed, large, tmp_path):
    from hi_b200.engine.core import Engine

    rng = random.Random(seed)
    cfg = draw(rng, large)
    page = rng.choice([16, 64, 64, 128]) if large else rng.choice([8, 16, 64])
    lengths = [rng.randrange(1, 40), rng.randrange(20, 120), rng.randrange(60, 200)] + ([rng.randrange(200, 420)] if large else [rng.randrange(40, 260)])
    mdir = str(tmp_path / "m")
    weights = write_model(mdir, cfg, seed=seed)
    reqs = {f"r{i}": tokens(cfg, n, seed * 10 + i) for i, n in enumerate(lengths)}
    rounded = lambda n: -(-n // page) * page
    cap = max(rounded(n) for n in lengths) + 2 * page
    mixed_cap = max(cap, sum(sorted(rounded(n) for n in lengths)[-2:]) + page)
    prompt = {r: min(len(t), max(2, len(t) - 24)) for r, t in reqs.items()}       # the rest is decoded token by token
    for dtype in ("float32", "bfloat16"):
        for regime, steps, pool in (("whole", h.trace_whole(reqs), cap), ("tail", h.trace_tail_decode(reqs), cap),
                                    ("portions", h.trace_portions(reqs), cap),
                                    ("mixed", h.trace_mixed(reqs, max_tokens=mixed_cap, page=page, seed=seed, prefill_len=prompt), mixed_cap)):
            eng = Engine.from_dir(mdir, dtype=dtype, kv_page_size=page, kv_cache_tokens=pool, max_active_requests=4, debug_poison=True)
            got, forced = replay(eng, steps, dtype)
            compare(cfg, weights, reqs, got, TOL[dtype], f"seed {seed} {cfg} page {page}: {dtype} {regime}", forced)
            assert not eng.manager.requests
            for p in eng.manager.pools:
                assert p.free == p.total, "pages were lost"
