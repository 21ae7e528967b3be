"""Pubunex configurations drawn from seeds: random sizes (odd ones and those the tensor-core
kernels take), random order of the three mixers, layers without a feed-forward, experts and
shared experts with bounds of their own or no shared expert, loops over any stretch of layers
from one pass to four or none, rotations of part of the head, of all of it or none, with and
without scaled frequencies, one to eight taps.  Each model runs a cut
request, an unequal batch that is decoded together, and greedy generation, in both precisions,
against the plain model."""
import random
import shutil

import pytest

from pubunex_util import (attention, config, delta, latent, moe, rotation, tokens, write_folder)
from test_pubunex_gpu import TD, recorded_alone, recorded_batch, rows_agree

pytestmark = pytest.mark.gpu


def draw(seed):
    rng = random.Random(9000 + seed)
    wide = seed % 2 == 1                       # every second model has tensor-core sizes
    mult = 8 if wide else 1

    def one_mixer():
        r = rng.random()
        if r < 0.4:
            kv = rng.choice([1, 2, 3])
            dim = rng.choice([16, 32, 64, 128]) if wide else rng.choice([6, 9, 16, 20, 33, 70])
            # (a unit vector or a norm of a head of a few values turns their signs into the
            # output: it jumps where they cross zero, and no comparison in 16 bits holds there)
            vdim = rng.choice([16, 32, 64]) if wide else rng.randint(8, 40)
            return delta(kv * rng.choice([1, 2, 4]), kv, dim, vdim, rng.randint(1, 8))
        if r < 0.7:
            kv = rng.choice([1, 2, 3])
            dim = rng.choice([16, 32, 48, 64, 128]) if wide else 2 * rng.randint(2, 14)
            vdim = dim if rng.random() < 0.4 and dim > 8 else (rng.choice([16, 32, 64, 128]) if wide
                                                   else rng.randint(9, 30))
            rot = None
            if rng.random() < 0.85:
                dims = dim if rng.random() < 0.4 else 2 * rng.randint(1, dim // 2)
                sc = None
                if rng.random() < 0.7:
                    slow = rng.choice([0.5, 1.0, 2.0])
                    sc = (rng.choice([1.0, 2.0, 8.0, 32.0]), rng.choice([16, 100, 4096]),
                          slow * rng.choice([2.0, 16.0, 32.0]), slow)
                rot = rotation(dims, rng.choice([50.0, 1e4, 5e5]), sc)
            return attention(kv * rng.choice([1, 2, 4]), kv, dim, vdim, 1.3 / dim ** 0.5, rot)
        if wide:
            d, r_, dv, R = (rng.choice([16, 32, 64]), rng.choice([8, 16, 32]),
                            rng.choice([16, 32, 64]), rng.choice([32, 64, 96, 160]))
        else:
            d, r_, dv, R = (rng.randint(3, 20), 2 * rng.randint(1, 8), rng.randint(8, 24),
                            rng.randint(5, 60))
        return latent(rng.choice([1, 2, 3, 4, 8]), d, r_, dv, R, 1.3 / (d + r_) ** 0.5,
                      rng.choice([50.0, 1e4, 5e5]))

    def one_ff():
        if rng.random() < 0.2:
            return None
        experts = rng.randint(1, 9)
        shared = None if rng.random() < 0.3 else mult * rng.randint(4 if not wide else 1, 12)
        return moe(experts, rng.randint(1, experts), mult * rng.randint(8 if not wide else 2, 16),
                   rng.choice([0.5, 1.0, 3.0, 7.0]), shared, rng.choice([None, 0.7, 2.0]))

    n = rng.randint(2, 5)
    layers = [(one_mixer(), one_ff()) for _ in range(n)]
    loop = None
    if rng.random() < 0.8:
        start = rng.randrange(n)
        loop = (start, rng.randint(start + 1, n), rng.randint(1, 4 if n < 4 else 3))
    width = rng.choice([64, 128, 192]) if wide else rng.randint(33, 120)
    return config(width, rng.randint(60, 400), layers, loop, eps=rng.choice([1e-6, 1e-5, 1e-3]))


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("seed", range(14))
def test_a_drawn_configuration(seed, dtype):
    from agave_b200.engine.api import Engine
    cfg = draw(seed)
    folder = write_folder(cfg, seed, TD[dtype], prefix=f"pubunex_draw{seed}_")
    try:
        eng = Engine(folder, dtype=dtype, max_tokens=4096)
        V = cfg["vocab"]
        toks = tokens(120 + 7 * seed, V, seed)
        rows_agree(*recorded_alone(eng, folder, toks, len(toks) - 20, dtype), dtype,
                   f"seed {seed} alone")
        seqs = [tokens(n, V, 100 + seed + n) for n in (70 + seed, 9, 1 + seed)]
        lens = [max(1, len(s) - 4 - 2 * i) for i, s in enumerate(seqs)]
        for i, (got, ref) in enumerate(recorded_batch(eng, folder, seqs, lens, dtype)):
            rows_agree(got, ref, dtype, f"seed {seed} request {i}")
        prompts = [tokens(n, V, 500 + seed + n) for n in (3, 40)]
        outs = eng.generate(prompts, max_new_tokens=6, stop_token_ids=[])
        slack = 2e-3 if dtype == "float32" else 8e-2
        misses = 0
        for p, g in zip(prompts, outs):
            ref = recorded_alone(eng, folder, p + g, len(p), dtype)[1]
            for k, t in enumerate(g):
                row = ref[len(p) - 1 + k]
                misses += float(row.max() - row[t]) > slack * float(row.abs().max())
        assert misses <= (0 if dtype == "float32" else 2), misses
    finally:
        shutil.rmtree(folder, ignore_errors=True)
