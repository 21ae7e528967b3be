"""Pubunex on the GPU against the plain implementation (tests/plain/pubunex_plain.py): each
mechanism alone, then whole models of five small configurations through the engine: the stream
after every layer run, whole prompts, the last tokens one by one, unequal batches against each
request alone, slots, pages and states used again, lengths round page borders and round the
rounds of the delta rule's scan, long decoding, greedy generation through the scheduler, and
trace replay as a process.

Where random weights would hide a fault, the inputs are made so that it shows: one key far back
among hundreds gets a score that stands out; sinks take a good share of the weight; decays are
set next to one and one far token writes much more than the others, so that what was written
hundreds of tokens ago still decides the read-out; expert gates lie on both sides of the bound.
"""
import dataclasses
import json
import math
import os
import shutil
import subprocess
import sys
import tempfile

import numpy as np
import pytest
import torch

from plain import pubunex_plain as P
from pubunex_util import (CONFIGS, attention, config, delta, folder_for, latent, plain_logits,
                          rotation, tokens, write_folder)
from test_kadavik_gpu import _Cache, alone, rel_err, rnd, summed
from util import ROOT

pytestmark = pytest.mark.gpu
DEV = "cuda"
DTYPES = ["float32", "bfloat16"]
TD = {"float32": torch.float32, "bfloat16": torch.bfloat16}


def rows_agree(got, ref, dtype, what=""):
    """Logit rows against reference rows: max error over the row's greatest logit.  32-bit:
    every row within 3e-4.  bfloat16: every row within 0.3 and all but one in twenty-five (at
    least one) within 0.12 (up to eleven layer runs of strong weights between 8-bit
    mantissas)."""
    got, ref = got.detach().double().cpu(), ref.detach().double().cpu()
    assert got.shape == ref.shape, (got.shape, ref.shape)
    assert torch.isfinite(got).all()
    err = (got - ref).abs().amax(dim=1) / ref.abs().amax(dim=1)
    worst = f"{what}: row {err.argmax().item()} of {len(err)} off by {err.max().item():.2e}"
    if dtype == "float32":
        assert err.max().item() <= 3e-4, worst
    else:
        assert err.max().item() <= 0.3, worst
        over = int((err > 0.12).sum().item())
        assert over <= max(1, len(err) // 25), f"{what}: {over} of {len(err)} rows off; " + worst


def run_alone(part, h, new, td):
    """One sequence through a mixer in steps of ``new`` tokens."""
    oc = _Cache(part.cache_request(), 1, td)
    got, at = [], 0
    for n in new:
        got.append(summed(part.forward(h[at:at + n].to(DEV), oc.step([n]), 0, True)))
        at += n
    return torch.cat(got)


def run_batches(part, plain, H, td, tol, rounds):
    """Three sequences start together with unequal lengths and go on one token at a time, the
    shorter ones ending first; then others take the freed slots, pages and states."""
    oc = _Cache(part.cache_request(), 3, td)
    for round_, (starts, totals) in enumerate(rounds):
        hs = [rnd(n, H, seed=100 + 10 * round_ + i).to(td) for i, n in enumerate(totals)]
        got = [[] for _ in hs]
        y = summed(part.forward(torch.cat([x[:n] for x, n in zip(hs, starts)]).to(DEV),
                                oc.step(list(starts)), 0, True))
        o = 0
        for i, n in enumerate(starts):
            got[i].append(y[o:o + n])
            o += n
        at = list(starts)
        while any(a < n for a, n in zip(at, totals)):
            live = [i for i in range(3) if at[i] < totals[i]]
            y = summed(part.forward(torch.cat([hs[i][at[i]:at[i] + 1] for i in live]).to(DEV),
                                    oc.step([1] * len(live), live), 0, True))
            for r, i in enumerate(live):
                got[i].append(y[r:r + 1])
                at[i] += 1
        for i in range(3):
            assert rel_err(torch.cat(got[i]), plain(hs[i].double())) < tol, (round_, i)
            oc.again(i)


ROUNDS = [((70, 1, 7), (82, 5, 60)), ((2, 65, 3), (9, 70, 50)), ((300, 20, 1), (303, 22, 30))]


# ------------------------------------------------------------ bounded gates
def _clamped(x, wg, wu, alpha, limit, scale=None):
    g, u = x @ wg.T, x @ wu.T
    if scale is not None:
        g, u = g * scale[:, None], u * scale[:, None]
    g, u = g.clamp(max=limit), u.clamp(min=-limit, max=limit)
    return g * torch.sigmoid(alpha * g) * (u + 1.0)


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("T, K, N", [(1, 72, 33), (8, 128, 256), (8, 1024, 512), (40, 256, 192), (64, 512, 64),
                                     (100, 128, 384), (130, 192, 128), (300, 256, 520), (33, 50, 21),
                                     (600, 128, 128)])
def test_bounded_gate_in_every_form_of_the_gated_product(dtype, T, K, N):
    """Few tokens (split over a cluster and not), middle and long prompts, sizes no tensor core
    takes: bounds that bite on both sides, an alpha that is not one."""
    from agave_b200 import kernels
    from agave_b200.config.base import ClampedGateSpec
    from agave_b200.parts.linear import GatedLinear
    td = TD[dtype]
    x = rnd(T, K, seed=1).to(td)
    wg, wu = (rnd(N, K, seed=s, std=1.5 / K ** 0.5).to(td) for s in (2, 3))
    for alpha, limit in ((1.702, 0.9), (0.7, 2.5)):
        part = GatedLinear(wg.to(DEV), wu.to(DEV), ClampedGateSpec(limit=limit, alpha=alpha))
        ref = _clamped(x.double(), wg.double(), wu.double(), alpha, limit)
        assert rel_err(part(x.to(DEV)), ref) < (5e-6 if dtype == "float32" else 8e-3)
        assert kernels.linear_tc_status() == 0
    # the bounds matter, each of them
    g, u = x.double() @ wg.double().T, x.double() @ wu.double().T
    assert (g > 0.9).any() and (u > 0.9).any() and (u < -0.9).any() and (g < -0.9).any()


def test_a_bounded_gate_needs_a_pair_and_a_limit():
    from agave_b200 import kernels
    x = torch.ones(2, 8, device=DEV)
    w = torch.ones(4, 8, device=DEV)
    out = torch.empty(2, 4, device=DEV)
    with pytest.raises(kernels.KernelError):
        kernels.linear(x, w, out, None, ("clamped", 1.0, 1.0))
    with pytest.raises(kernels.KernelError):
        kernels.linear(x, w, out, w, ("clamped", 1.0, 0.0))
    with pytest.raises(kernels.KernelError):
        kernels.linear(x, w, out, w, "relu2")


# ------------------------------------------------------------ experts
def _moe_weights(H, E, ff, shared, seed, td):
    lin = 1.0 / H ** 0.5
    W = {"router": rnd(E, H, seed=seed, std=2.0 * lin)}
    for i, (n, f) in enumerate([(f"e{e}", ff) for e in range(E)] +
                               ([("shared", shared)] if shared else [])):
        W[n + ".gate"] = rnd(f, H, seed=seed + 10 + 3 * i, std=1.6 * lin)
        W[n + ".up"] = rnd(f, H, seed=seed + 11 + 3 * i, std=1.6 * lin)
        W[n + ".down"] = rnd(H, f, seed=seed + 12 + 3 * i, std=1.0 / f ** 0.5)
    return {k: v.to(td) for k, v in W.items()}


def _moe_part(W, H, E, top, ff, limit, shared, shared_limit, td):
    from agave_b200.config.pubunex import PubunexConfig, PubunexExpert, PubunexExperts
    from agave_b200.parts.moe import RoutedFeedForward
    spec = PubunexConfig._ffn_spec(PubunexExperts(
        experts=E, top=top, expert=PubunexExpert(ff, limit),
        shared=PubunexExpert(shared, shared_limit) if shared else None))
    part = RoutedFeedForward(spec, H, td, torch.device(DEV))
    t = {"router.weight": W["router"]}
    for n, p in [(f"e{e}", f"experts.{e}") for e in range(E)] + ([("shared",) * 2] if shared else []):
        for x in ("gate", "up", "down"):
            t[f"{p}.{x}_proj.weight"] = W[f"{n}.{x}"]
    assert set(t) == set(RoutedFeedForward.param_specs(spec, H))
    part.load(t, td, torch.device(DEV))
    return part


MOE = [(1, 72, 5, 2, 24, 0.8, 20, 2.0), (40, 96, 1, 1, 32, 1.0, 0, 1.0), (33, 128, 4, 4, 64, 1.5, 8, 0.5),
       (200, 128, 7, 3, 64, 0.7, 96, 0.7), (600, 64, 3, 2, 128, 1.2, 64, 3.0), (130, 76, 6, 1, 18, 2.0, 22, 1.0),
       (9, 64, 16, 5, 24, 0.6, 0, 1.0)]


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("T, H, E, top, ff, limit, shared, shared_limit", MOE)
def test_experts_whose_weight_multiplies_their_input(dtype, T, H, E, top, ff, limit, shared,
                                                     shared_limit):
    """Router, grouped products on the tensor cores and without them, the shared expert with a
    bound of its own; weighing the outputs instead would be another function."""
    td = TD[dtype]
    W = _moe_weights(H, E, ff, shared, 300 + T, td)
    x = rnd(T, H, seed=301).to(td)
    part = _moe_part(W, H, E, top, ff, limit, shared, shared_limit, td)
    Wd = {k: v.double() for k, v in W.items()}
    f = {"expert": {"ff": ff, "limit": limit}, "router": {"experts": E, "top": top}}
    if shared:
        f["shared"] = {"ff": shared, "limit": shared_limit}
    ids, wts = (t.cpu() for t in part.route(x.to(DEV)))
    s = torch.sigmoid(x.double() @ Wd["router"].T)
    assert (wts.double() - s.gather(1, ids.long())).abs().max() < 3e-6
    # no expert that was left out scores above one that was chosen
    left = s.clone().scatter_(1, ids.long(), -1.0)
    assert (left.max(-1).values - wts.double().min(-1).values).max() < 1e-5
    ref = P.experts(x.double(), f, Wd, "", ids.long())
    y = summed(part.forward(x.to(DEV), None))
    assert rel_err(y, ref) < (2e-5 if dtype == "float32" else 2e-2)
    part.weigh_input = False
    assert rel_err(summed(part.forward(x.to(DEV), None)), ref) > 5e-2


# ------------------------------------------------------------ joins
@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("R, H, n_terms", [(1, 72, 2), (5, 128, 5), (300, 76, 3), (40, 1024, 4), (7, 33, 5)])
def test_a_bias_is_a_term_of_the_join(dtype, R, H, n_terms):
    """One row for all rows among branches in partial sums and in the compute dtype; up to five
    terms; with and without a stream."""
    from agave_b200 import kernels
    td = TD[dtype]
    h, w = rnd(R, H, seed=1).float(), rnd(H, seed=2, std=0.3).float() + 1.0
    terms, want = [], torch.zeros(R, H, dtype=torch.float64)
    for i in range(n_terms):
        y = (rnd(3, R, H, seed=10 + i).float(), rnd(H, seed=10 + i).float(),
             rnd(R, H, seed=10 + i).to(td))[i % 3]
        mult = (1.0, 1.0, -0.5, 2.0, 0.7)[i]
        want = want + mult * (y.double().sum(0) if y.dim() == 3 else y.double())
        terms.append((y.to(DEV), mult, -1))
    hd = h.to(DEV)
    x = torch.empty(R, H, dtype=td, device=DEV)
    kernels.gated_join(hd, terms, None, None, None, w.to(DEV), 1e-5, x)
    assert rel_err(hd, h.double() + want) < 2e-6
    assert rel_err(x, P.rms(h.double() + want, 1e-5) * w.double()) < (5e-6 if dtype == "float32" else 6e-3)
    x = torch.empty(R, H, device=DEV)
    kernels.gated_join(None, terms, None, None, None, None, 0.0, x)
    assert rel_err(x, want) < 2e-6


# ------------------------------------------------------------ the delta rule
def _mixer_spec(kind, m, eps=1e-5):
    """The library's lowering of one mixer, through a configuration of one layer."""
    from agave_b200.config.pubunex import PubunexConfig
    raw = {"layers": [{"type": kind, "mixer": m, "mlp": None}], "norm": {"eps": eps}, "vocab": 8,
           "width": 8}
    return PubunexConfig.from_dict(raw).to_model_spec().blocks[0].mixer


def _part(kind, W, m, H, td):
    from agave_b200.models.pubunex import _MIXERS
    from agave_b200.parts.base import mixer_class
    spec = _mixer_spec(kind, m)
    cls = mixer_class(spec.kind)
    part = cls(spec, H, td, torch.device(DEV))
    back = {v: k for k, v in _MIXERS[kind].items()}
    t = {back[k]: v for k, v in W.items()}
    assert set(t) == set(cls.param_specs(spec, H))
    part.load(t, td, torch.device(DEV))
    return part


def _mixer_weights(kind, m, H, seed, td):
    """A mixer's tensors as the folder writer makes them."""
    from pubunex_util import make_tensors
    cfg = config(H, 8, [((kind, m), None)])
    p = "l0.mix."
    return {k[len(p):]: v.to(td) for k, v in make_tensors(cfg, seed, torch.float64).items()
            if k.startswith(p)}


def _plain_of(kind, m, W):
    Wd = {k: v.double() for k, v in W.items()}
    return lambda h: P.mixer(kind, h.double(), m, Wd, "", 1e-5)


def _delta(*a):
    return delta(*a)[1]


DELTA = [(72, _delta(4, 2, 10, 14, 3)), (128, _delta(4, 2, 64, 64, 4)), (96, _delta(1, 1, 16, 16, 1)),
         (76, _delta(2, 1, 130, 33, 6)), (64, _delta(6, 1, 18, 7, 2)), (64, _delta(2, 2, 128, 64, 4)),
         (48, _delta(3, 3, 1, 1, 4)), (64, _delta(2, 1, 300, 20, 2)),
         # (more taps than the convolution holds in registers)
         (64, _delta(2, 1, 24, 20, 9)), (48, _delta(4, 2, 64, 32, 17)), (64, _delta(4, 4, 33, 40, 8)),
         (40, _delta(1, 1, 200, 3, 2)), (64, _delta(12, 3, 128, 128, 2)), (64, _delta(16, 4, 48, 136, 3)),
         # (enough columns for the forms that hold more of them a lane, the last ones partly empty)
         (48, _delta(26, 13, 100, 122, 2)), (48, _delta(40, 5, 40, 61, 2)), (32, _delta(3, 1, 256, 250, 2))]


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("H, m", DELTA)
def test_the_delta_rule_as_prompt_and_token_by_token(dtype, H, m):
    """Alone: the whole sequence in one step; a prompt and then tokens one by one, from cuts at
    the first token, before the convolution is full, inside a round of the scan and at its and
    its buffers' borders."""
    td = TD[dtype]
    T = 70
    W = _mixer_weights("delta", m, H, 70, td)
    part, plain = _part("delta", W, m, H, td), _plain_of("delta", m, W)
    h = rnd(T, H, seed=71).to(td)
    ref = plain(h)
    tol = 5e-5 if dtype == "float32" else 4e-2
    for new in ([T], [1] * T, [2] + [1] * 68, [16] + [1] * 54, [43] + [1] * 27, [65] + [1] * 5):
        assert rel_err(run_alone(part, h, new, td), ref) < tol, new[:2]


@pytest.mark.parametrize("n", [1, 2, 3, 4, 5, 7, 8, 9, 12, 15, 16, 17, 23, 24, 31, 32, 33])
def test_every_length_round_a_round_of_the_scan(n):
    """32-bit: prompts that end at every place of a round, of four tokens and of eight; the state
    they leave decides the tokens after them."""
    for m in (_delta(2, 1, 20, 12, 3), _delta(2, 2, 64, 24, 3), _delta(2, 1, 128, 16, 3)):
        W = _mixer_weights("delta", m, 48, 40 + n, torch.float32)
        part, plain = _part("delta", W, m, 48, torch.float32), _plain_of("delta", m, W)
        h = rnd(n + 5, 48, seed=n).float()
        assert rel_err(run_alone(part, h, [n] + [1] * 5, torch.float32), plain(h)) < 5e-5


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("m", [_delta(4, 2, 24, 40, 4), _delta(4, 1, 64, 32, 3), _delta(2, 2, 128, 48, 2),
                               _delta(2, 2, 16, 24, 12)])
def test_delta_unequal_batches_and_slots_used_again(dtype, m):
    """A freed slot's state and stored convolution inputs must start at zero again; sequences
    whose rounds begin at any place of the step's tokens."""
    td = TD[dtype]
    W = _mixer_weights("delta", m, 96, 90, td)
    run_batches(_part("delta", W, m, 96, td), _plain_of("delta", m, W), 96, td,
                5e-5 if dtype == "float32" else 4e-2, ROUNDS)


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("m", [_delta(4, 2, 24, 12, 3), _delta(2, 1, 64, 64, 4), _delta(2, 2, 128, 32, 2)])
def test_what_was_written_hundreds_of_tokens_ago_decides(dtype, m):
    """Decays next to one, and writes that only one early token makes at all: the read-out 600
    tokens later is what that token wrote, and decoding must still have it.  The convolution
    passes the current token."""
    td = TD[dtype]
    H, T, far = 64, 640, 9
    W = {k: v.double() for k, v in _mixer_weights("delta", m, H, 500, td).items()}
    for n in "qkv":
        W[n + ".conv"][:] = 0.0
        W[n + ".conv"][:, -1] = 1.0
    # beta is next to nothing but where axis 5 is set
    W["b"][:] = 0.0
    W["b"][:, 4] = -12.0
    W["b"][:, 5] = 14.0
    W["A_log"][:] = -7.0
    W = {k: v.to(td) for k, v in W.items()}
    h = rnd(T, H, seed=501)
    h[:, 4] = 1.0
    h[:, 5] = 0.0
    h[far, 5] = 1.0
    h = h.to(td)
    plain = _plain_of("delta", m, W)
    ref = plain(h)
    h2 = h.clone()
    h2[far, 7:] = -h2[far, 7:]
    assert (plain(h2)[-20:] - ref[-20:]).abs().max() > 0.3 * ref[-20:].abs().max()
    got = run_alone(_part("delta", W, m, H, td), h, [600] + [1] * 40, td)
    tol = 5e-4 if dtype == "float32" else 6e-2
    assert rel_err(got[-40:], ref[-40:]) < tol
    assert rel_err(got[20:], ref[20:]) < 2 * tol


def test_delta_states_of_strong_decays_and_full_writes():
    """32-bit: decays down to nothing (their products underflow inside a round) and beta next to
    one with keys that hardly differ: the substitution inside a round is exact there too."""
    m, H, T = _delta(2, 1, 64, 32, 2), 48, 50
    W = {k: v.float() for k, v in _mixer_weights("delta", m, H, 520, torch.float32).items()}
    W["k"] = W["k"] * 0.02
    W["k"][:, 3] = rnd(64, seed=3).float() * 3.0
    W["b"][:] = 0.0
    W["b"][:, 3] = 9.0
    for log in (-9.0, 0.0, 3.0, 6.0):
        W["A_log"][:] = log
        h = rnd(T, H, seed=521).float()
        h[:, 3] = 1.0 + 0.1 * h[:, 3]
        ref = _plain_of("delta", m, W)(h)
        part = _part("delta", W, m, H, torch.float32)
        assert rel_err(run_alone(part, h, [T], torch.float32), ref) < 2e-4, log
        assert rel_err(run_alone(part, h, [30] + [1] * 20, torch.float32), ref) < 2e-4, log


def test_the_delta_read_out_with_a_sigmoid_gate():
    """The gate's other activation, and heads wider than a lane keeps."""
    from agave_b200 import kernels
    from agave_b200.engine.batch import PREFILL, StepContext
    i32 = dict(dtype=torch.int32, device=DEV)
    for T, H, dv, silu in ((5, 3, 300, True), (5, 2, 37, False), (400, 4, 64, False), (3, 2, 700, False)):
        o, row = rnd(T, H * dv, seed=1).float(), rnd(T, H * dv + 8, seed=2).float()
        w = rnd(dv, seed=3).float()
        slots = torch.tensor([0, -1], **i32)
        seq = torch.tensor([0] * (T - 1) + [1], **i32)
        ctx = StepContext(mode=PREFILL, n_tokens=T, batch=2, tokens=None, positions=None,
                          seq_index=seq, cu_seqlens=None, slots=slots, lens=None, max_len=0,
                          max_new=0, cache=None, dtype=torch.float32, device=torch.device(DEV))
        y = torch.empty(T, H * dv, device=DEV)
        kernels.head_delta_out(o.to(DEV), row.to(DEV), None, H * dv + 8, 8, w.to(DEV), 1e-5, H, dv,
                               silu, ctx, y)
        g = row.double()[:, 8:].view(T, H, dv)
        ref = P.rms(o.double().view(T, H, dv), 1e-5) * w.double() * \
            (P.silu(g) if silu else torch.sigmoid(g))
        ref[-1] = 0.0                                  # (the padding entry's token)
        assert rel_err(y, ref.reshape(T, -1)) < 5e-6


# ------------------------------------------------------------ attention
def test_scaled_frequencies_on_the_device_tables():
    """cos and sin, multiplied, at positions far beyond the original context."""
    from agave_b200.config.base import RotarySpec, WavelengthScalingSpec
    from agave_b200.engine.batch import PREFILL, StepContext
    from agave_b200.parts.rope import RotaryEmbedding
    sc = (8.0, 500, 10.0, 1.0)
    rope = RotaryEmbedding(RotarySpec(theta=1000.0, rotary_dim=16, scaling=WavelengthScalingSpec(
        factor=sc[0], original=sc[1], fast=sc[2], slow=sc[3])), 20)
    pos = torch.tensor([0, 1, 2, 77, 1000, 4099], dtype=torch.int32, device=DEV)
    ctx = StepContext(mode=PREFILL, n_tokens=6, batch=1, tokens=None, positions=pos,
                      seq_index=None, cu_seqlens=None, slots=None, lens=None, max_len=0,
                      max_new=0, cache=None, dtype=torch.float32, device=torch.device(DEV))
    cos, sin = rope.tables(ctx)
    f, mult = P.frequencies(rotation(16, 1000.0, sc))
    a = pos.cpu().double()[:, None] * torch.tensor(f, dtype=torch.float64)[None, :]
    assert (cos.cpu().double() - torch.cos(a) * mult).abs().max() < 2e-6
    assert (sin.cpu().double() - torch.sin(a) * mult).abs().max() < 2e-6
    assert mult > 1.1


YARN = (8.0, 64, 4.0, 0.5)
ATTENTION = [
    # T, H, (kind, mixer)
    (90, 72, attention(4, 2, 10, 14, 0.4, rotation(6, 1000.0, YARN))),
    (200, 128, attention(8, 2, 64, 128, 0.13, rotation(32, 20000.0, YARN))),
    (150, 64, attention(2, 2, 24, 8, 0.3, rotation(24, 50.0))),
    (70, 96, attention(1, 1, 16, 16, 0.3)),
    (300, 80, attention(6, 3, 128, 48, 0.09, rotation(2, 1e5, (3.0, 32, 8.0, 2.0)))),
    (220, 64, attention(8, 1, 64, 64, 0.15, rotation(64, 1e4, YARN))),
    (90, 72, latent(3, 10, 4, 6, 20, 0.35)),
    (210, 128, latent(4, 48, 16, 64, 64, 0.13)),
    (250, 96, latent(8, 64, 32, 32, 128, 0.1, 5e5)),
    (70, 96, latent(1, 16, 16, 16, 16, 0.3, 50.0)),
    (140, 76, latent(3, 9, 6, 11, 33, 0.3, 2000.0)),
    (220, 80, latent(2, 32, 32, 48, 250, 0.15)),
    (220, 64, latent(16, 24, 8, 24, 40, 0.2)),
]


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("T, H, case", ATTENTION)
def test_attention_mixers_as_prompt_and_token_by_token(dtype, T, H, case):
    """Each attention alone as a prompt, and as a prompt followed by tokens one by one, from
    cuts at the first token, at a page border and elsewhere; biases and sinks that matter."""
    kind, m = case
    td = TD[dtype]
    W = _mixer_weights(kind, m, H, 600, td)
    h = rnd(T, H, seed=601).to(td)
    ref = _plain_of(kind, m, W)(h)
    part = _part(kind, W, m, H, td)
    tol = 5e-5 if dtype == "float32" else 4e-2
    for new in ([T], [1] * T, [T - 30] + [1] * 30, [64] + [1] * (T - 64)):
        assert rel_err(run_alone(part, h, new, td), ref) < tol, new[:2]
    for name, off in (("o.b", 0.0), ("v.b", 0.0), ("sink", -1e4)):
        if name in W:
            less = _plain_of(kind, m, {**W, name: torch.full_like(W[name], off)})(h)
            assert rel_err(less, ref) > 5e-2, name


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("case", [attention(4, 2, 32, 48, 0.25, rotation(16, 1e4, YARN)),
                                  latent(4, 32, 16, 24, 48, 0.2), latent(2, 10, 6, 10, 13, 0.3)])
def test_attention_unequal_batches_and_slots_used_again(dtype, case):
    kind, m = case
    td = TD[dtype]
    W = _mixer_weights(kind, m, 96, 900, td)
    run_batches(_part(kind, W, m, 96, td), _plain_of(kind, m, W), 96, td,
                5e-5 if dtype == "float32" else 4e-2, ROUNDS)


@pytest.mark.parametrize("dtype", DTYPES)
def test_a_far_key_among_hundreds_decides(dtype):
    """A key 900 tokens back outscores all others: prompt rows and decoded rows; every query
    reads axis 1 (set everywhere), only that token's key axis 0."""
    td = TD[dtype]
    H, T = 64, 930
    h = rnd(T, H, seed=801)
    h[:, 0], h[:, 1] = 0.0, 1.0
    h[11, 0] = 6.0
    h = h.to(td)
    cases = [attention(4, 1, 32, 48, 0.18, rotation(8, 1e4, YARN)), latent(4, 24, 8, 32, 40, 0.18)]
    for kind, m in cases:
        W = {k: v.double() for k, v in _mixer_weights(kind, m, H, 800, td).items()}
        d, s = m["dim"], 1.6 / m["scale"] ** 0.5
        if kind == "attention":
            for a in range(4):
                W["q"][a * d + d - 1] = 0.0
                W["q"][a * d + d - 1, 1] = s
            W["k"][d - 1] = 0.0
            W["k"][d - 1, 0] = s
            W["k.b"][d - 1] = 0.0
        else:
            # the latent's last value alone reads axis 0; the norm divides it by the rest
            r, R = m["rot_dim"], m["kv_rank"]
            W["dkv"][R - 1] = 0.0
            W["dkv"][R - 1, 0] = 1.5
            W["dkv.norm"][R - 1] = 1.0
            for a in range(4):
                W["q"][a * (d + r)] = 0.0
                W["q"][a * (d + r), 1] = 2 * s
                W["uk"][a * d] = 0.0
                W["uk"][a * d, R - 1] = s
        W = {k: v.to(td) for k, v in W.items()}
        plain = _plain_of(kind, m, W)
        ref = plain(h)
        h2 = h.clone()
        h2[11, 0] = 0
        assert (plain(h2)[-10:] - ref[-10:]).abs().max() > 0.3 * ref[-10:].abs().max(), kind
        part = _part(kind, W, m, H, td)
        tol = 1e-4 if dtype == "float32" else 5e-2
        assert rel_err(run_alone(part, h, [T], td), ref) < tol
        assert rel_err(run_alone(part, h, [900] + [1] * 30, td)[-30:], ref[-30:]) < tol


def test_the_output_bias_outside_a_joining_block():
    """A block that knows nothing of terms gets the sum with the bias in it."""
    td = torch.float32
    kind, m = attention(4, 2, 16, 24, 0.3, rotation(8, 1e3))
    W = _mixer_weights(kind, m, 64, 10, td)
    part = _part(kind, W, m, 64, td)
    h = rnd(20, 64, seed=11).float()
    terms = part.forward_terms(h.to(DEV), _Cache(part.cache_request(), 1, td).step([20]), 0, True)
    assert len(terms) == 2 and terms[1][0].shape == (64,)
    y = part.forward(h.to(DEV), _Cache(part.cache_request(), 1, td).step([20]), 0, True)
    ref = _plain_of(kind, m, W)(h)
    assert rel_err(summed(y), ref) < 5e-5
    assert rel_err(summed(terms[0][0]), ref - W["o.b"].double()) < 5e-5


# ------------------------------------------------------------ whole models
_ENGINES = {}


def engine_for(name, dtype, max_tokens=8192):
    key = (name, dtype)
    if key not in _ENGINES:
        from agave_b200.engine.api import Engine
        folder = folder_for(name, TD[dtype])
        _ENGINES[key] = (Engine(folder, dtype=dtype, max_tokens=max_tokens), folder)
    return _ENGINES[key]


def vocab(name):
    return CONFIGS[name]["vocab"]


NAMES = sorted(CONFIGS)


class RecordedRuns:
    """While active, every routed feed-forward's choice is kept in run order, step by step (a
    layer that runs several times chooses in every pass).  ``of_rows`` puts a request's rows
    together again from (step, first row, rows) pieces, as the plain model's ``choices`` wants
    them.  In bfloat16 a close call that falls the other way moves a row far more than rounding
    does, so the plain model takes the experts chosen in the very steps compared."""

    def __init__(self, eng):
        self.eng, self.steps, self._cur = eng, [], None

    def __enter__(self):
        from agave_b200.parts.moe import RoutedFeedForward
        self._cls, self._keep = RoutedFeedForward, RoutedFeedForward.route
        rec = self

        def route(part, x):
            ids, wts = rec._keep(part, x)
            rec._cur.append(ids.cpu().long())
            return ids, wts
        RoutedFeedForward.route = route
        return self

    def __exit__(self, *exc):
        self._cls.route = self._keep

    def step(self, entries, want):
        self._cur = []
        out = self.eng.step(entries, want)
        self.steps.append(self._cur)
        return out

    def of_rows(self, pieces):
        n = len(self.steps[pieces[0][0]])
        return [torch.cat([self.steps[k][i][a:a + m] for k, a, m in pieces]) for i in range(n)]


def reference(rec, folder, toks, pieces, dtype):
    if dtype == "float32":
        return plain_logits(folder, toks)
    return plain_logits(folder, toks, choices=rec.of_rows(pieces))


def recorded_alone(eng, folder, toks, cut, dtype):
    """(rows of a request run alone with ``cut`` tokens as the prompt, the plain model's)"""
    with RecordedRuns(eng) as rec:
        s = eng.acquire()
        got = [rec.step([(s, toks[:cut])], [list(range(cut))])]
        for p in range(cut, len(toks)):
            got.append(rec.step([(s, [toks[p]])], [[0]]))
        eng.release(s)
    pieces = [(0, 0, cut)] + [(k, 0, 1) for k in range(1, len(toks) - cut + 1)]
    return torch.cat(got), reference(rec, folder, toks, pieces, dtype)


def recorded_batch(eng, folder, seqs, lens, dtype):
    """Requests that start together with ``lens`` tokens each and go on one by one, the shorter
    ones ending first: per request its rows and the plain model's for it alone."""
    slots = [eng.acquire() for _ in seqs]
    got, pieces = [[] for _ in seqs], [[] for _ in seqs]
    with RecordedRuns(eng) as rec:
        out = rec.step([(sl, s[:n]) for sl, s, n in zip(slots, seqs, lens)],
                       [list(range(n)) for n in lens])
        o = 0
        for i, n in enumerate(lens):
            got[i].append(out[o:o + n])
            pieces[i].append((0, o, n))
            o += n
        at = list(lens)
        for i, s in enumerate(seqs):
            if at[i] == len(s):
                eng.release(slots[i])
        while any(a < len(s) for a, s in zip(at, seqs)):
            live = [i for i in range(len(seqs)) if at[i] < len(seqs[i])]
            out = rec.step([(slots[i], [seqs[i][at[i]]]) for i in live], [[0]] * len(live))
            for r, i in enumerate(live):
                got[i].append(out[r:r + 1])
                pieces[i].append((len(rec.steps) - 1, r, 1))
                at[i] += 1
                if at[i] == len(seqs[i]):
                    eng.release(slots[i])
    return [(torch.cat(g), reference(rec, folder, s, p, dtype))
            for g, s, p in zip(got, seqs, pieces)]


@pytest.mark.parametrize("name", NAMES)
def test_the_stream_after_every_layer_run(name):
    """32-bit: the residual stream after each layer run (a looped layer counts each time) against
    the plain model's, so that a fault names its run."""
    eng, folder = engine_for(name, "float32")
    toks = tokens(25, vocab(name), 9)
    streams = []
    plain_logits(folder, toks, streams)
    model = eng.model
    assert len(streams) == len(model.spec.schedule)
    for upto in range(1, len(model.spec.schedule) + 1):
        s = eng.acquire()
        ctx = eng.runner.context([(s, toks)])
        keep = model.spec
        model.spec = dataclasses.replace(keep, schedule=keep.schedule[:upto])
        try:
            h = model.hidden_states(ctx)
        finally:
            model.spec = keep
        eng.runner.cache.trim(s)
        eng.release(s)
        assert rel_err(h, streams[upto - 1]) < 2e-5, f"layer run {upto - 1}"


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("name", NAMES)
def test_whole_prompts_alone(name, dtype):
    eng, folder = engine_for(name, dtype)
    for n in (1, 2, 7, 8, 64, 65, 250):
        toks = tokens(n, vocab(name), 20 + n)
        rows_agree(*recorded_alone(eng, folder, toks, n, dtype), dtype, f"{name} {n} tokens")


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("name", NAMES)
def test_prompt_then_tokens_one_by_one(name, dtype):
    """Decoding starts after one token, before a convolution is full, at a page border."""
    eng, folder = engine_for(name, dtype)
    for n, cut in ((90, 60), (41, 1), (140, 127), (100, 64), (12, 2)):
        toks = tokens(n, vocab(name), 11 + n)
        rows_agree(*recorded_alone(eng, folder, toks, cut, dtype), dtype, f"{name} {n}/{cut}")


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("name", NAMES)
def test_unequal_batches_and_slots_used_again(name, dtype):
    """Requests of unequal lengths start together and are decoded together, the shorter ones
    ending earlier; then other requests take the freed slots, pages and states.  Every row
    against the plain model run on that request alone."""
    eng, folder = engine_for(name, dtype)
    V = vocab(name)
    for round_, lens in enumerate([(130, 3, 64, 1), (1, 65, 20), (63, 70, 5)]):
        seqs = [tokens(n + 6 + 3 * i, V, 50 + 10 * round_ + i) for i, n in enumerate(lens)]
        for i, (got, ref) in enumerate(recorded_batch(eng, folder, seqs, lens, dtype)):
            rows_agree(got, ref, dtype, f"{name} round {round_} request {i}")


@pytest.mark.parametrize("name", NAMES)
def test_lengths_round_page_borders_and_rounds(name):
    """32-bit: prompts that end just before, on and just after a page border and a round of the
    delta rule's scan, each followed by three decoded tokens."""
    eng, folder = engine_for(name, "float32")
    for n in (3, 4, 5, 8, 9, 15, 16, 17, 63, 64, 65, 127, 128, 129):
        toks = tokens(n + 3, vocab(name), n)
        ref = plain_logits(folder, toks)
        s = eng.acquire()
        got = [eng.step([(s, toks[:n])], [[0, n - 1]])]
        for p in range(n, n + 3):
            got.append(eng.step([(s, [toks[p]])], [[0]]))
        eng.release(s)
        rows_agree(torch.cat(got), ref[[0, n - 1, n, n + 1, n + 2]], "float32", f"{name} {n}")


@pytest.mark.parametrize("name", ["P1", "P2", "P4"])
def test_a_pass_has_a_cache_of_its_own(name):
    """32-bit: the same configuration with one pass more is another function, and one whose
    embedding is not added again yet another; the loop's passes share weights alone."""
    eng, folder = engine_for(name, "float32")
    toks = tokens(40, vocab(name), 3)
    ref = plain_logits(folder, toks)
    model = eng.model
    keep = model.spec
    s = eng.acquire()
    with_ = eng.step([(s, toks)], [list(range(40))])
    eng.release(s)
    model.spec = dataclasses.replace(keep, schedule=tuple(
        dataclasses.replace(c, add_embedding=False) for c in keep.schedule))
    try:
        s = eng.acquire()
        without = eng.step([(s, toks)], [list(range(40))])
        eng.release(s)
    finally:
        model.spec = keep
    rows_agree(with_, ref, "float32", name)
    assert rel_err(without, ref) > 5e-2


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("name", ["P1", "P5"])
def test_the_embedding_joins_without_a_block_that_knows_it(name, dtype):
    """Blocks that do not take the embedding as a term of their join get it in a launch of the
    decoder's own: the same rows, in prompts and while decoding."""
    from agave_b200.parts.parallel import ParallelBlock
    eng, folder = engine_for(name, dtype)
    toks = tokens(50, vocab(name), 8)
    a = alone(eng, toks, 30)
    ParallelBlock.joins_extra = False
    try:
        b = alone(eng, toks, 30)
    finally:
        ParallelBlock.joins_extra = True
    assert rel_err(b, a) < (1e-5 if dtype == "float32" else 1e-1)


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("name", ["P1", "P2"])
def test_long_decoding(name, dtype):
    """250 tokens decoded after a prompt of 5."""
    eng, folder = engine_for(name, dtype)
    toks = tokens(255, vocab(name), 77)
    rows_agree(*recorded_alone(eng, folder, toks, 5, dtype), dtype, name)


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("name", NAMES)
def test_greedy_generation_through_the_entry_point(name, dtype):
    """``Engine.generate`` (scheduler, CUDA graphs, the arg max in the head's epilogue): every
    generated token is the plain model's best, or within rounding of it."""
    eng, folder = engine_for(name, dtype)
    V = vocab(name)
    prompts = [tokens(n, V, 300 + n) for n in (4, 37, 70, 9, 130)]
    outs = eng.generate(prompts, max_new_tokens=12, stop_token_ids=[])
    slack = 2e-3 if dtype == "float32" else 8e-2
    misses = 0
    for p, g in zip(prompts, outs):
        assert len(g) == 12
        # (bfloat16: under the experts the library chooses when it is fed those tokens)
        ref = recorded_alone(eng, folder, p + g, len(p), dtype)[1]
        for k, t in enumerate(g):
            row = ref[len(p) - 1 + k]
            misses += float(row.max() - row[t]) > slack * float(row.abs().max())
    assert misses <= (0 if dtype == "float32" else 3), misses


@pytest.mark.parametrize("dtype", DTYPES)
def test_generation_in_batches_of_the_slot_limit(dtype):
    """More prompts than slots: slots and their states are used again; the tokens are the same
    as with room for all."""
    from agave_b200.engine.api import Engine
    folder = folder_for("P1", TD[dtype])
    V = vocab("P1")
    prompts = [tokens(n, V, 900 + n) for n in (5, 66, 17, 3, 40, 21, 8)]
    wide = Engine(folder, dtype=dtype, max_tokens=4096)
    narrow = Engine(folder, dtype=dtype, max_tokens=4096, max_batch=3)
    a = wide.generate(prompts, max_new_tokens=10, stop_token_ids=[])
    b = narrow.generate(prompts, max_new_tokens=10, stop_token_ids=[])
    same = sum(x == y for x, y in zip(a, b))
    assert same >= (len(prompts) if dtype == "float32" else len(prompts) - 3)


def test_sampling_runs_on_this_architecture():
    eng, _ = engine_for("P1", "bfloat16")
    V = vocab("P1")
    kw = dict(max_new_tokens=8, temperature=0.8, top_k=20, top_p=0.9, seed=5, stop_token_ids=[])
    outs = eng.generate([tokens(6, V, 1), tokens(30, V, 2)], **kw)
    again = eng.generate([tokens(6, V, 1), tokens(30, V, 2)], **kw)
    assert outs == again and all(len(o) == 8 and all(0 <= t < V for t in o) for o in outs)


def test_random_weights_from_a_configuration():
    from agave_b200.engine.api import Engine
    raw = CONFIGS["P1"]
    eng = Engine.from_config(raw, seed=3, max_tokens=1024)
    outs = eng.generate([tokens(9, raw["vocab"], 1)], max_new_tokens=5, stop_token_ids=[])
    assert len(outs[0]) == 5
    info = eng.model_info()
    assert info["architecture"] == "Pubunex" and info["weight_bytes"] > 0


@pytest.mark.parametrize("dtype", DTYPES)
def test_a_model_of_delta_layers_alone(dtype):
    """No layer keeps keys and values: the cache holds fixed-size states and nothing else."""
    from agave_b200.engine.api import Engine
    from pubunex_util import moe
    cfg = config(64, 90, [(delta(4, 2, 16, 24, 4), moe(3, 1, 16, 1.0, 16)),
                          (delta(2, 2, 8, 8, 2), None)], loop=(0, 2, 2))
    folder = write_folder(cfg, 4, TD[dtype])
    try:
        eng = Engine(folder, dtype=dtype, max_tokens=512)
        toks = tokens(90, 90, 3)
        rows_agree(*recorded_alone(eng, folder, toks, 40, dtype), dtype, "delta")
        outs = eng.generate([toks[:9], toks[:30]], max_new_tokens=4, stop_token_ids=[])
        assert [len(o) for o in outs] == [4, 4]
    finally:
        shutil.rmtree(folder, ignore_errors=True)


@pytest.mark.parametrize("dtype", DTYPES)
def test_trace_replay_as_a_process(dtype):
    name = "P2"
    eng, folder = engine_for(name, dtype)
    V = vocab(name)
    a, b = tokens(210, V, 5), tokens(33, V, 6)
    # (the same steps through the engine here, for the experts they choose)
    refs = {"a": recorded_alone(eng, folder, a, 195, dtype)[1],
            "b": recorded_alone(eng, folder, b, 30, dtype)[1]}
    steps = [{"step": 0, "entries": [{"id": "a", "tokens": a[:195], "want": [0, 100, 194]},
                                     {"id": "b", "tokens": b[:30], "want": [29]}], "end": []}]
    for k in range(15):
        ent, end = [{"id": "a", "tokens": [a[195 + k]], "want": [0]}], []
        if k < 3:
            ent.append({"id": "b", "tokens": [b[30 + k]], "want": [0] if k != 1 else []})
            if k == 2:
                end.append("b")
        if k == 14:
            end.append("a")
        steps.append({"step": k + 1, "entries": ent, "end": end})
    out = tempfile.mkdtemp(prefix="pubunex_trace_")
    try:
        r = subprocess.run([sys.executable, os.path.join(ROOT, "bin", "trace_run"), "--model",
                            folder, "--dtype", dtype, "--out", out, "--max-tokens", "300"],
                           input="\n".join(json.dumps(s) for s in steps) + "\n", text=True,
                           capture_output=True, timeout=900)
        assert r.returncode == 0, r.stderr[-2000:]
        assert [l for l in r.stdout.split("\n") if l.startswith("done")] == \
            [f"done {k}" for k in range(16)]
        got = torch.from_numpy(np.fromfile(os.path.join(out, "0.f32"), dtype="<f4").reshape(4, V))
        rows = [(got, torch.stack([refs["a"][0], refs["a"][100], refs["a"][194], refs["b"][29]]))]
        for k in range(15):
            want = [refs["a"][195 + k]]
            if k < 3 and k != 1:
                want.append(refs["b"][30 + k])
            g = np.fromfile(os.path.join(out, f"{k + 1}.f32"), dtype="<f4").reshape(len(want), V)
            rows.append((torch.from_numpy(g), torch.stack(want)))
        got, want = torch.cat([g for g, _ in rows]), torch.cat([w for _, w in rows])
        if dtype == "float32":
            rows_agree(got, want, dtype, "trace")
        else:
            err = (got.double() - want).abs().amax(1) / want.abs().amax(1)
            assert (err <= 0.12).sum() >= len(err) - 2, err
    finally:
        shutil.rmtree(out, ignore_errors=True)


def test_command_line_on_this_architecture():
    """``python -m agave_b200`` picks the model class from config.json: greedy tokens equal the
    plain model's, --model-info names the architecture, --profile lists this design's
    operations."""
    name = "P2"
    folder = folder_for(name, torch.float32)
    prompt = tokens(9, vocab(name), 31)

    def run(*args):
        env = dict(os.environ)
        env["PYTHONPATH"] = ROOT + os.pathsep + env.get("PYTHONPATH", "")
        return subprocess.run([sys.executable, "-m", "agave_b200", *args], capture_output=True,
                              text=True, timeout=900, env=env, cwd=ROOT)
    toks = ",".join(str(t) for t in prompt)
    r = run(folder, "--tokens", toks, "-n", "6", "--json", "--dtype", "float32")
    assert r.returncode == 0, r.stderr[-2000:]
    out = json.loads(r.stdout.strip().splitlines()[-1])["output_ids"]
    assert len(out) == 6
    ref = plain_logits(folder, prompt + out)
    for k, t in enumerate(out):
        row = ref[len(prompt) - 1 + k]
        assert float(row.max() - row[t]) <= 2e-3 * float(row.abs().max()), (k, t)
    r = run(folder, "--model-info", "--json")
    assert r.returncode == 0 and "Pubunex" in r.stdout, r.stderr[-2000:]
    r = run(folder, "--tokens", toks, "-n", "3", "--profile", "--dtype", "bfloat16")
    assert r.returncode == 0, r.stderr[-2000:]
    for op in ("norm", "qkv", "qk_norm_rope", "attention", "latent_attention", "q_absorb", "v_up",
               "ssm_conv", "delta_coef", "delta_scan", "delta_out", "router", "experts_gate_up",
               "experts_down", "shared_gate_up", "shared_down", "out_proj", "lm_head", "TOTAL"):
        assert op in r.stderr, (op, r.stderr[-1500:])


@pytest.mark.parametrize("name, room", [("P1", 60), ("P2", 90), ("P3", 64), ("P4", 100)])
def test_a_cache_of_one_or_two_pages(name, room):
    """32-bit: a request that fills the cache to its last row."""
    from agave_b200.engine.api import Engine
    folder = folder_for(name, torch.float32)
    eng = Engine(folder, dtype="float32", max_tokens=room, ctx_size=room, max_batch=1)
    toks = tokens(room, vocab(name), 5)
    rows_agree(alone(eng, toks, room - 15), plain_logits(folder, toks), "float32", name)


def test_the_library_kernels_run_without_errors_left_behind():
    from agave_b200 import kernels
    assert kernels.attention_tc_status() == 0
    assert kernels.attention_decode_status() == 0
    assert kernels.linear_tc_status() == 0
    assert kernels.moe_tc_status() == 0
    assert math.isfinite(float(torch.zeros(1, device=DEV)))
