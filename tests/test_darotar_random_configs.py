"""Darotar configurations drawn at random (seeded): every size, constant, the order of layers, whose latents a layer reads
and what a configuration may leave out move at once, small odd sizes as well as sizes at which the tensor-core kernels take
over, and each draw goes through the four ways of cutting against the plain model, in 32-bit and in bfloat16."""
import random

import pytest

import harness as h
from darotar_configs import attention, config, latent, moe, write_model
from test_darotar_engine import TOL, compare, replay, tokens

pytestmark = pytest.mark.gpu


def draw(rng: random.Random, large: bool) -> dict:
    layers, sources = [], []
    for i in range(rng.randrange(2, 6)):
        mlp, ff = None, rng.choice([64, 96, 128]) if large else rng.choice([1, 2, 8, 16]) * rng.randrange(1, 9)
        if rng.random() < 0.8:
            experts = rng.choice([1, 2, 4, 8, 16]) if large else rng.choice([1, 2, 3, 5, 8, 12, 33])
            mlp = moe(experts, rng.choice([t for t in (1, 1, 2, 3, 4, 6, 10) if t <= experts]), ff)
        base = rng.choice([10.0, 500.0, 10000.0, 1e6])
        if rng.random() < 0.4:
            kv = rng.choice([1, 1, 2, 3])
            dim = rng.choice([64, 128, 192]) if large else rng.choice([2, 5, 8, 12, 16, 24, 40, 48])
            layers.append(attention(kv * rng.choice([1, 2, 4, 6, 9]), kv, dim, rng.choice([0.3, 1.0, 2.0]) * dim ** -0.5, base,
                                    dims=rng.choice([dim // 2 * 2, 2, dim // 4 * 2 or 2]), factor=rng.choice([None, 1.0, 0.5, 3.0, 40.0]),
                                    window=rng.choice([None, 1, 2, 7, 16, 33, 64, 96, 150, 1000]), mlp=mlp))
            continue
        heads, dim = rng.choice([1, 2, 3, 8, 17]), rng.choice([32, 64]) if large else rng.choice([1, 4, 7, 16, 24])
        q_rank = rng.choice([64, 96]) if large else rng.randrange(1, 40)
        vdim = rng.choice([32, 64, 128]) if large else rng.choice([1, 3, 8, 20, 32])
        if sources and rng.random() < 0.6:
            j = rng.choice(sources)
            m = layers[j]["mixer"]
            layers.append(latent(heads, dim, m["rot_dim"], vdim, m["kv_rank"], q_rank, rng.choice([0.3, 1.0]) * (dim + m["rot_dim"]) ** -0.5,
                                 m["rot"]["base"], kv_from=j, mlp=mlp))
            continue
        rank, rot = rng.choice([(32, 32), (96, 32), (128, 48)]) if large else (rng.choice([1, 5, 16, 40, 70]), rng.choice([2, 4, 6, 16, 26]))
        sources.append(i)
        layers.append(latent(heads, dim, rot, vdim, rank, q_rank, rng.choice([0.3, 1.0]) * (dim + rot) ** -0.5, base, mlp=mlp))
    width = rng.choice([192, 320, 384]) if large else rng.choice([2, 3, 8, 16]) * rng.randrange(3, 20)
    return config(rng.randrange(60, 900), width, rng.choice([1e-5, 1e-6, 3e-4]), layers, mult=rng.choice([1.0, 0.2, 0.5, 1.3]))


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
