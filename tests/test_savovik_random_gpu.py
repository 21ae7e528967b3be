"""Savovik configurations drawn from seeds: random sizes (odd ones and those the tensor-core
kernels take), random order of the three mixers, layers without a feed-forward, layers that run
an earlier layer's weights, masks from one token to longer than the prompt or none, caps,
rotations of part of the head, of all of it or none, with and without scaled frequencies, one to
eight taps, states, ranks and groups from one up.  Each model runs a cut request, an unequal
batch that is decoded together, and greedy generation, in both precisions, against the plain
model."""
import random
import shutil

import pytest
import torch

from savovik_util import (attention, config, heads, mamba2, parallel, plain_logits, rotation, scan,
                          tokens, write_folder)
from test_savovik_gpu import TD, alone, rows_agree

pytestmark = pytest.mark.gpu


def draw(seed):
    rng = random.Random(7000 + seed)
    wide = seed % 2 == 1                       # every second model has tensor-core sizes
    mult = 8 if wide else 1

    def head_args(softcap):
        kv = rng.choice([1, 2, 3])
        dim = rng.choice([16, 32, 48, 64, 128]) if wide else 2 * rng.randint(2, 14)
        vdim = dim if rng.random() < 0.4 and dim > 8 else (rng.choice([16, 32, 64, 128]) if wide
                                               else rng.randint(9, 30))
        rot = None
        if rng.random() < 0.85:
            dims = dim if rng.random() < 0.4 else 2 * rng.randint(1, dim // 2)
            sc = rng.choice([None, 2.0, 8.0, "bands"])
            if sc == "bands":
                low = rng.choice([0.5, 1.0, 2.0])
                sc = (rng.choice([2.0, 8.0]), low, low * rng.choice([2.0, 4.0]),
                      rng.choice([8, 32, 256]))
            rot = rotation(dims, rng.choice([50.0, 1e4, 5e5]), sc)
        return heads(kv * rng.choice([1, 2, 4]), kv, dim, vdim, 1.3 / dim ** 0.5,
                     size=rng.choice([None, 1, 2, 5, 33, 64, 65, 100, 128, 500]), rot=rot,
                     softcap=rng.choice([None, 1.0, 5.0, 30.0]) if softcap else None)

    def one_mixer():
        r = rng.random()
        if r < 0.35:
            return parallel(head_args(False),
                            scan(mult * rng.randint(1, 24 if wide else 90), rng.choice([1, 4, 7, 16, 24, 40]),
                                 rng.randint(1, 20), rng.randint(1, 8)),
                            rng.choice([1.0, 0.5, 1.6]), rng.choice([1.0, 0.7, -1.2]))
        if r < 0.7:
            groups = rng.choice([1, 2, 3])
            n = groups * rng.choice([1, 2, 4])
            vdim = rng.choice([16, 32, 64]) if wide else rng.randint(1, 40)
            # (a norm over a part of a few channels turns their signs into the output: it jumps
            # where they cross zero together, and no comparison in 16 bits holds there)
            parts = [k for k in (1, n) if n * vdim // k >= 12] or [1]
            return mamba2(n, max(vdim, 12 // n + 1),
                          rng.choice([16, 64, 128]) if wide else rng.randint(1, 60), groups,
                          rng.choice(parts), rng.randint(1, 8))
        return "attention", head_args(True)

    layers = []
    for i in range(rng.randint(2, 6)):
        if i and rng.random() < 0.3:
            layers.append(rng.randrange(i))
            while isinstance(layers[layers[-1]], int):         # (a layer with tensors of its own)
                layers[-1] = layers[layers[-1]]
        else:
            layers.append((one_mixer(), None if rng.random() < 0.25 else mult * rng.randint(3, 30)))
    width = rng.choice([64, 128, 192]) if wide else rng.randint(33, 120)
    return config(width, rng.randint(60, 400), layers, eps=rng.choice([1e-6, 1e-5, 1e-3]))


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("seed", range(14))
def test_a_drawn_configuration(seed, dtype):
    from agave_b200.engine.api import Engine
    cfg = draw(seed)
    folder = write_folder(cfg, seed, TD[dtype], prefix=f"savovik_draw{seed}_")
    try:
        eng = Engine(folder, dtype=dtype, max_tokens=4096)
        V = cfg["vocab"]
        toks = tokens(150 + 7 * seed, V, seed)
        rows_agree(alone(eng, toks, len(toks) - 20), plain_logits(folder, toks), dtype,
                   f"seed {seed} alone")
        seqs = [tokens(n, V, 100 + seed + n) for n in (70 + seed, 9, 1 + seed)]
        lens = [max(1, len(s) - 4 - 2 * i) for i, s in enumerate(seqs)]
        slots = [eng.acquire() for _ in seqs]
        got = [[] for _ in seqs]
        out = eng.step([(sl, s[:n]) for sl, s, n in zip(slots, seqs, lens)],
                       [list(range(n)) for n in lens])
        o = 0
        for i, n in enumerate(lens):
            got[i].append(out[o:o + n])
            o += n
        at = list(lens)
        while any(a < len(s) for a, s in zip(at, seqs)):
            live = [i for i in range(len(seqs)) if at[i] < len(seqs[i])]
            out = eng.step([(slots[i], [seqs[i][at[i]]]) for i in live], [[0]] * len(live))
            for r, i in enumerate(live):
                got[i].append(out[r:r + 1])
                at[i] += 1
        for sl in slots:
            eng.release(sl)
        for i, s in enumerate(seqs):
            rows_agree(torch.cat(got[i]), plain_logits(folder, s), dtype, f"seed {seed} request {i}")
        prompts = [tokens(n, V, 500 + seed + n) for n in (3, 40)]
        outs = eng.generate(prompts, max_new_tokens=6, stop_token_ids=[])
        slack = 2e-3 if dtype == "float32" else 8e-2
        misses = 0
        for p, g in zip(prompts, outs):
            ref = plain_logits(folder, p + g)
            for k, t in enumerate(g):
                row = ref[len(p) - 1 + k]
                misses += float(row.max() - row[t]) > slack * float(row.abs().max())
        assert misses <= (0 if dtype == "float32" else 2), misses
    finally:
        shutil.rmtree(folder, ignore_errors=True)
