"""Savovik on the GPU against the plain implementation (tests/plain/savovik_plain.py): each
mechanism alone, then whole models of four small configurations through the engine: the stream
after every layer, whole prompts, the last tokens one by one, unequal batches against each
request alone, slots, pages and states used again, lengths round page borders, window and chunk
edges, long decoding, greedy generation through the scheduler, and trace replay as a process.

Where random weights would hide a fault, the inputs are made so that it shows: one key (just
inside or just outside a window or a chunk, or far back among hundreds) gets a score that
stands out; scores reach well into the soft cap; the scans' decays are set next to one and one
far token writes much more than the others, so that what was written hundreds of tokens ago
still decides the read-out.
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

from plain import savovik_plain as P
from savovik_util import CONFIGS, folder_for, heads, mamba2, plain_logits, rotation, scan, tokens
from test_kadavik_gpu import _Cache, alone, rel_err, rnd, summed
from util import ROOT

pytestmark = pytest.mark.gpu
DEV = "cuda"
DTYPES = ["float32", "bfloat16"]
TD = {"float32": torch.float32, "bfloat16": torch.bfloat16}


def rows_agree(got, ref, dtype, what=""):
    """Logit rows against reference rows: max error over the row's greatest logit.  32-bit:
    every row within 3e-4.  bfloat16: every row within 0.3 and all but one in twenty-five (at
    least one) within 0.12 (several layers of strong weights between 8-bit mantissas, and norms
    of short parts, which turn round where all their values are small)."""
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


# ------------------------------------------------------------ joins and gates
@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("R, H, n_terms, n_gates, splits", [
    (1, 72, 1, 1, 1), (5, 128, 3, 2, 4), (300, 76, 2, 1, 1), (40, 1024, 3, 2, 1), (3, 4096, 4, 2, 8),
    (7, 33, 2, 0, 2)])
def test_branches_join_through_gates_and_the_next_norm(dtype, R, H, n_terms, n_gates, splits):
    from agave_b200 import kernels
    td = TD[dtype]
    h = rnd(R, H, seed=1).float()
    terms, want = [], h.double()
    part = rnd(splits, R, max(n_gates, 1) * H, seed=2, std=1.0 / splits ** 0.5).float()
    bias = rnd(max(n_gates, 1) * H, seed=3, std=0.5).float()
    logits = part.double().sum(0) + bias.double()
    for i in range(n_terms):
        gate = i % (n_gates + 1) - 1
        mult = (1.0, 0.6, -1.4, 2.0)[i]
        y = rnd(splits, R, H, seed=10 + i).float() if i % 2 == 0 else rnd(R, H, seed=10 + i).to(td)
        s = y.double().sum(0) if y.dim() == 3 else y.double()
        g = torch.sigmoid(logits[:, gate * H:(gate + 1) * H]) if gate >= 0 else 1.0
        want = want + mult * g * s
        terms.append((y.to(DEV), mult, gate))
    w = rnd(H, seed=4, std=0.3).float() + 1.0
    for form in ("partial", "rows", "no norm", "no stream"):
        hd = h.to(DEV).clone()
        x = torch.empty(R, H, dtype=td, device=DEV)
        row = part.sum(0).to(DEV) if form == "rows" else None
        kernels.gated_join(None if form == "no stream" else hd, terms,
                           row if n_gates else None,
                           None if form == "rows" or not n_gates else part.to(DEV),
                           bias.to(DEV) if n_gates else None,
                           None if form.startswith("no") else w.to(DEV), 1e-5,
                           x if form != "no norm" else None)
        if form != "no stream":
            assert rel_err(hd, want) < 2e-6
        tol = 5e-6 if dtype == "float32" else 6e-3
        if form == "no stream":
            assert rel_err(x, want - h.double()) < tol
        elif form != "no norm":
            assert rel_err(x, P.rms(want, 1e-5) * w.double()) < tol


def test_a_value_norm_a_bias_and_neighbouring_pairs_in_the_row_kernel():
    """The kernel between projection and attention on its own, both inputs it takes."""
    from agave_b200 import kernels
    T, A, G, d, dv, dims = 9, 3, 1, 12, 20, 8
    W = A * d + G * (d + dv)
    part = rnd(3, T, W, seed=5).float()
    bias = rnd(W, seed=6, std=0.5).float()
    wq, wk = rnd(d, seed=7).float(), rnd(d, seed=8).float()
    pos = torch.tensor([0, 1, 2, 3, 4, 77, 78, 900, 4000], dtype=torch.int32)
    f = torch.tensor(P.frequencies({"dims": dims, "base": 500.0}), dtype=torch.float64)
    a = pos.double()[:, None] * f
    x = part.double().sum(0) + bias.double()
    q = P.rms(x[:, :A * d].view(T, A, d), 1e-5) * wq.double()
    k = P.rms(x[:, A * d:(A + G) * d].view(T, G, d), 1e-5) * wk.double()
    v = P.rms(x[:, (A + G) * d:].view(T, G, dv), 3e-5)
    rot = {"dims": dims, "base": 500.0}
    want = torch.cat([P.rotate(q, pos, rot, True).reshape(T, -1),
                      P.rotate(k, pos, rot, True).reshape(T, -1), v.reshape(T, -1)], dim=1)
    for partial in (part.to(DEV), None):
        row = torch.empty(T, W, device=DEV) if partial is not None else part.sum(0).to(DEV)
        kernels.qk_norm_rope_store(row, A, G, d, wq.to(DEV), wk.to(DEV), 1e-5,
                                   torch.cos(a).float().to(DEV), torch.sin(a).float().to(DEV), dims,
                                   pos.to(DEV), partial=partial, value_dim=dv, bias=bias.to(DEV),
                                   interleaved=True, value_eps=3e-5)
        assert rel_err(row, want) < 5e-6


# ------------------------------------------------------------ attention kernels
def _qkv(lens, nh, nkv, hd, hdv, td, seed=5, std=1.6):
    n = sum(lens)
    return (rnd(n, nh * hd, seed=seed, std=std).to(td).to(DEV),
            rnd(n, nkv * hd, seed=seed + 1, std=std).to(td).to(DEV),
            rnd(n, nkv * hdv, seed=seed + 2).to(td).to(DEV))


def _seen(n, window):
    i, j = torch.arange(n)[:, None], torch.arange(n)[None, :]
    if window > 0:
        return (j <= i) & (i - j < window)
    if window < 0:
        return (j <= i) & (torch.div(i, -window, rounding_mode="floor") ==
                           torch.div(j, -window, rounding_mode="floor"))
    return j <= i


PROMPT = [(64, 64, 76, 20.0, 300), (64, 128, -70, 0.0, 260), (128, 64, 0, 3.0, 200),
          (48, 48, 100, 5.0, 330), (128, 256, 65, 30.0, 270), (32, 16, -64, 2.0, 200),
          (24, 40, 33, 4.0, 150), (256, 128, 0, 0.0, 210), (16, 144, -100, 8.0, 300)]


@pytest.mark.parametrize("hd, hdv, window, cap, T", PROMPT)
def test_a_soft_cap_and_wide_values_in_every_form_of_the_prompt_kernels(hd, hdv, window, cap, T):
    """bfloat16: the one-warp, the mma.sync and (head sizes in steps of 16) the tcgen05 prompt
    kernels on the same q, k, v: two sequences of unequal lengths, scores of several times the
    cap, sliding windows and chunks."""
    from agave_b200 import kernels
    nh, nkv, lens = 4, 2, [T, T // 3]
    q, k, v = _qkv(lens, nh, nkv, hd, hdv, torch.bfloat16)
    scale = 3.0 / hd ** 0.5
    i32 = dict(dtype=torch.int32, device=DEV)
    cu = torch.tensor([0, lens[0], sum(lens)], **i32)
    pos = torch.tensor(list(range(lens[0])) + list(range(lens[1])), **i32)
    seq = torch.tensor([0] * lens[0] + [1] * lens[1], **i32)
    refs, o = [], 0
    for n in lens:
        refs.append(P.attend(q[o:o + n].double().cpu().view(n, nh, hd),
                             k[o:o + n].double().cpu().view(n, nkv, hd),
                             v[o:o + n].double().cpu().view(n, nkv, hdv), scale, _seen(n, window),
                             cap or None))
        o += n
    ref = torch.cat(refs)
    if cap:
        plain = P.attend(q[:T].double().cpu().view(T, nh, hd), k[:T].double().cpu().view(T, nkv, hd),
                         v[:T].double().cpu().view(T, nkv, hdv), scale, _seen(T, window), None)
        assert (plain - ref[:T]).abs().max() > 0.05 * ref.abs().max()      # (the cap matters)
    out = torch.empty(sum(lens), nh * hdv, dtype=torch.bfloat16, device=DEV)
    kernels.attention_prefill_simt(q, k, v, out, pos, seq, cu, nh, nkv, hd, scale, window,
                                   value_dim=hdv, softcap=cap)
    assert rel_err(out, ref) < 2e-2
    out.zero_()
    kernels.attention_prefill_mma(q, k, v, out, cu, max(lens), nh, nkv, hd, scale, window,
                                  value_dim=hdv, softcap=cap)
    assert rel_err(out, ref) < 2e-2
    if hd % 16 == 0 and hdv % 16 == 0:
        out.zero_()
        kernels.attention_prefill_tc(q, k, v, out, cu, max(lens), nh, nkv, hd, scale, window,
                                     value_dim=hdv, softcap=cap)
        assert kernels.attention_tc_status() == 0
        assert rel_err(out, ref) < 2e-2


DECODE = [(64, 64, 76, 20.0), (64, 128, -70, 0.0), (128, 64, 0, 3.0), (48, 48, 100, 5.0),
          (128, 256, 65, 30.0), (32, 16, -64, 2.0), (256, 128, 0, 4.0), (16, 144, 90, 8.0),
          (320, 32, 0, 6.0), (24, 40, 33, 4.0)]


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("hd, hdv, window, cap", DECODE)
def test_a_soft_cap_and_wide_values_in_the_decode_kernels(dtype, hd, hdv, window, cap):
    """One query for each of several sequences (one of them padding) against the paged cache,
    the split kernel of the dtype and the one-warp kernel, with eight query heads a kv head."""
    from agave_b200 import kernels
    td = TD[dtype]
    nh, nkv, lens = 8, 1, [400, 1, 65, 128, 77]
    if hd % 16 or hdv % 16:
        nh, nkv = 4, 2
    B, PAGE = len(lens) + 1, 64
    pages = [(n + PAGE - 1) // PAGE for n in lens]
    total = sum(pages)
    perm = torch.randperm(total, generator=torch.Generator().manual_seed(3)).tolist()
    cap_rows = max(pages) * PAGE
    table = torch.zeros(B, max(pages), dtype=torch.int32)
    kp = rnd(total, PAGE, nkv, hd, seed=1, std=1.6).to(td)
    vp = rnd(total, PAGE, nkv, hdv, seed=2).to(td)
    q = rnd(B, nh * hd, seed=3, std=1.6).to(td)
    scale, refs, at = 3.0 / hd ** 0.5, [], 0
    for b, n in enumerate(lens):
        mine = perm[at:at + pages[b]]
        at += pages[b]
        table[b, :pages[b]] = torch.tensor(mine, dtype=torch.int32)
        k = kp[mine].reshape(-1, nkv, hd)[:n].double()
        v = vp[mine].reshape(-1, nkv, hdv)[:n].double()
        see = _seen(n, window)[n - 1:]
        refs.append(P.attend(q[b].double().view(1, nh, hd), k, v, scale, see, cap or None))
    refs.insert(2, torch.zeros(1, nh * hdv, dtype=torch.float64))           # the padding entry
    q = torch.cat([q[:2], q[-1:], q[2:-1]])
    slots = torch.tensor([0, 1, -1, 2, 3, 4], dtype=torch.int32, device=DEV)
    pos = torch.tensor([399, 0, 0, 64, 127, 76], dtype=torch.int32, device=DEV)
    seq = torch.arange(B, dtype=torch.int32, device=DEV)
    ref = torch.cat(refs)
    args = (kp.to(DEV), vp.to(DEV), table.to(DEV), slots, pos)
    tol = 3e-5 if dtype == "float32" else 2e-2
    out = torch.full((B, nh * hdv), float("nan"), dtype=td, device=DEV)
    if hd % 16 == 0 and hdv % 16 == 0:
        keys = min(abs(window), 400) if window else 400
        kernels.attention_decode_split(q.to(DEV), out, *args, PAGE, cap_rows, nh, nkv, hd, scale,
                                       window, keys, value_dim=hdv, softcap=cap)
        assert rel_err(out, ref) < tol
        out.fill_(float("nan"))
    kernels.attention_paged_simt(q.to(DEV), out, *args, seq, PAGE, cap_rows, nh, nkv, hd, scale,
                                 window, value_dim=hdv, softcap=cap)
    assert rel_err(out, ref) < tol


# ------------------------------------------------------------ attention mixers
def _attention_weights(m, H, seed, td, extras):
    A, G, d, dv = m["heads"], m["kv_heads"], m["dim"], m["vdim"]
    lin = 1.0 / H ** 0.5
    W = {"q": rnd(A * d, H, seed=seed, std=1.5 * lin), "k": rnd(G * d, H, seed=seed + 1, std=1.5 * lin),
         "v": rnd(G * dv, H, seed=seed + 2, std=lin),
         "o": rnd(H, A * dv, seed=seed + 3, std=1.0 / (A * dv) ** 0.5)}
    if extras:
        for i, n in enumerate("qkv"):
            W[n + ".b"] = rnd(W[n].shape[0], seed=seed + 4 + i, std=0.4)
        W["q.norm"] = rnd(d, seed=seed + 8, std=0.3) + 1.2
        W["k.norm"] = rnd(d, seed=seed + 9, std=0.3) + 1.2
    return {k: v.to(td) for k, v in W.items()}


NAMES_OF = {"q": "q_proj.weight", "k": "k_proj.weight", "v": "v_proj.weight", "o": "o_proj.weight",
            "q.b": "q_proj.bias", "k.b": "k_proj.bias", "v.b": "v_proj.bias",
            "q.norm": "q_norm.weight", "k.norm": "k_norm.weight"}


def _spec_of(kind, m, eps=1e-5):
    """The library's lowering of one mixer, through a configuration of one layer."""
    from agave_b200.config.savovik import SavovikConfig
    raw = {"layers": [{"type": kind, "mixer": m, "mlp": None}], "norm": {"eps": eps}, "vocab": 8,
           "width": 8}
    return SavovikConfig.from_dict(raw).to_model_spec().blocks[0].mixer


def _chunked_part(W, m, H, td):
    from agave_b200.parts.attention import AttentionMixer
    spec = _spec_of("parallel", {"left": m, "right": scan(4, 1, 1, 1), "left_scale": 1.0,
                                 "right_scale": 1.0}).left
    part = AttentionMixer(spec, H, td, torch.device(DEV))
    t = {NAMES_OF[k]: v for k, v in W.items()}
    assert set(t) == set(AttentionMixer.param_specs(spec, H))
    part.load(t, td, torch.device(DEV))
    return part


def _window_part(W, m, H, td):
    from agave_b200.parts.attention import AttentionMixer
    spec = _spec_of("attention", m)
    part = AttentionMixer(spec, H, td, torch.device(DEV))
    t = {NAMES_OF[k]: v for k, v in W.items()}
    assert set(t) == set(AttentionMixer.param_specs(spec, H))
    part.load(t, td, torch.device(DEV))
    return part


SC = (8.0, 1.0, 4.0, 16)
CHUNKED = [
    # T, H, mixer
    (90, 72, heads(4, 2, 10, 14, 0.4, size=7, rot=rotation(6, 1e4, SC))),
    (200, 128, heads(4, 1, 64, 128, 0.13, size=70, rot=rotation(32, 500.0, SC))),
    (150, 64, heads(2, 2, 24, 8, 0.3, size=64, rot=rotation(24, 50.0))),
    (70, 96, heads(1, 1, 16, 16, 0.3, size=1)),
    (300, 80, heads(6, 3, 128, 48, 0.09, size=130, rot=rotation(2, 1e5, 3.0))),
    (140, 64, heads(2, 1, 32, 32, 0.25)),
]
WINDOWED = [
    (90, 72, heads(3, 1, 12, 6, 0.35, size=9, rot=rotation(8, 300.0, 2.5), softcap=5.0)),
    (210, 128, heads(8, 2, 64, 64, 0.13, size=100, rot=rotation(64, 1e4, 4.0), softcap=20.0)),
    (250, 96, heads(4, 2, 128, 64, 0.09, size=64, rot=rotation(64, 1e4, 8.0), softcap=2.0)),
    (70, 96, heads(2, 2, 24, 24, 0.3, size=1)),
    (220, 80, heads(4, 4, 48, 48, 0.2, size=90, rot=rotation(40, 2e5), softcap=18.0)),
    (140, 64, heads(2, 1, 32, 16, 0.25, softcap=1.0)),
]


def _plain_of(fn, m, W):
    Wd = {k: v.double() for k, v in W.items()}
    return lambda h: fn(h.double(), m, Wd, "", 1e-5)


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("which, case", [("chunk", c) for c in CHUNKED] +
                         [("window", c) for c in WINDOWED])
def test_attention_mixers_as_prompt_and_token_by_token(dtype, which, case):
    """Each attention alone as a prompt, and as a prompt followed by tokens one by one, from
    cuts at the first token, inside a chunk or window and at a page border."""
    T, H, m = case
    td = TD[dtype]
    W = _attention_weights(m, H, 600, td, which == "chunk")
    fn, make = (P.chunked_attention, _chunked_part) if which == "chunk" else \
        (P.window_attention, _window_part)
    h = rnd(T, H, seed=601).to(td)
    ref = _plain_of(fn, m, W)(h)
    part = make(W, m, H, td)
    tol = 5e-5 if dtype == "float32" else 4e-2
    for new in ([T], [1] * T, [T - 30] + [1] * 30, [64] + [1] * (T - 64)):
        assert rel_err(run_alone(part, h, new, td), ref) < tol, new[:2]


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("which", ["chunk", "window"])
def test_attention_unequal_batches_and_slots_used_again(dtype, which):
    td = TD[dtype]
    m = heads(4, 2, 32, 48, 0.25, size=40, rot=rotation(16, 1e4, 2.0),
              softcap=None if which == "chunk" else 6.0)
    W = _attention_weights(m, 96, 900, td, which == "chunk")
    fn, make = (P.chunked_attention, _chunked_part) if which == "chunk" else \
        (P.window_attention, _window_part)
    run_batches(make(W, m, 96, td), _plain_of(fn, m, W), 96, td,
                5e-5 if dtype == "float32" else 4e-2, ROUNDS)


def _marked(T, H, marks, seed, amp=6.0):
    """A stream whose tokens ``marks`` alone have a component along axis 0, all tokens having one
    along axis 1: with the weights below, every query scores those tokens' keys highest."""
    h = rnd(T, H, seed=seed)
    h[:, 0] = 0.0
    h[:, 1] = 1.0
    for t in marks:
        h[t, 0] = amp
    return h


def _mark_weights(W, m, td, chunk, strength=1.6):
    """The last (unrotated) dimension of every q head reads axis 1, of every k head axis 0; under
    a per-head norm all other dimensions are made small instead."""
    d = m["dim"]
    for name, axis, n in (("q", 1, m["heads"]), ("k", 0, m["kv_heads"])):
        w = W[name].double()
        for a in range(n):
            w[a * d + d - 1] = 0.0
            w[a * d + d - 1, axis] = strength / m["scale"] ** 0.5
        W[name] = w.to(td)
        if chunk:
            W[name + ".b"] = torch.zeros_like(W[name + ".b"])
            nw = torch.full((d,), 0.2, dtype=torch.float64)
            nw[-1] = 2.0 / m["scale"] ** 0.5
            W[name + ".norm"] = nw.to(td)
    return W


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("size, d, dv", [(76, 64, 64), (20, 24, 16), (64, 32, 48), (100, 128, 64)])
def test_the_key_at_a_window_edge_decides(dtype, size, d, dv):
    """One key scores far above the rest: the row just inside its window is its value, the row
    just outside another one altogether, in a prompt and when decoding; a mask that is off by
    one shows.  The cap is above the marked score, but not by much."""
    td = TD[dtype]
    H, T = 64, 2 * size + 40
    m = heads(4, 2, d, dv, 0.2, size=size, rot=rotation(d // 2, 1e4, 2.0), softcap=25.0)
    tol = 1e-4 if dtype == "float32" else 5e-2
    for mark in (0, 3, min(64, T - size - 5), T - size - 2):
        W = _mark_weights(_attention_weights(m, H, 700, td, False), m, td, False)
        h = _marked(T, H, [mark], 701 + mark).to(td)
        ref = _plain_of(P.window_attention, m, W)(h)
        a, b = ref[mark + size - 1], ref[mark + size]
        assert (a - b).abs().max() > 0.3 * max(a.abs().max(), b.abs().max())
        part = _window_part(W, m, H, td)
        for new in ([T], [mark + 3] + [1] * (T - mark - 3), [T - 9] + [1] * 9):
            assert rel_err(run_alone(part, h, new, td), ref) < tol, (mark, new[:2])


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("size, d, dv", [(76, 64, 128), (20, 24, 16), (64, 32, 32), (100, 128, 64)])
def test_the_key_at_a_chunk_edge_decides(dtype, size, d, dv):
    """Marked keys at a chunk's first and last place and at the next chunk's first: the last row
    of the chunk sees them, the next row none of them."""
    td = TD[dtype]
    H, T = 64, 2 * size + 40
    m = heads(4, 2, d, dv, 0.2, size=size, rot=rotation(d // 2, 1e4, SC))
    tol = 1e-4 if dtype == "float32" else 5e-2
    for mark in (0, size - 1, size, size + 3, 2 * size - 2):
        W = _mark_weights(_attention_weights(m, H, 720, td, True), m, td, True)
        h = _marked(T, H, [mark], 721 + mark).to(td)
        ref = _plain_of(P.chunked_attention, m, W)(h)
        edge = (mark // size + 1) * size
        a, b = ref[edge - 1], ref[edge]
        assert (a - b).abs().max() > 0.3 * max(a.abs().max(), b.abs().max())
        part = _chunked_part(W, m, H, td)
        for new in ([T], [mark + 3] + [1] * (T - mark - 3), [edge] + [1] * (T - edge),
                    [edge - 1] + [1] * (T - edge + 1)):
            assert rel_err(run_alone(part, h, new, td), ref) < tol, (mark, new[:2])


@pytest.mark.parametrize("dtype", DTYPES)
def test_a_far_key_among_hundreds_decides(dtype):
    """No mask: a key 900 tokens back outscores all others; prompt rows and decoded rows."""
    td = TD[dtype]
    H, T = 64, 930
    m = heads(4, 1, 32, 48, 0.18, rot=rotation(8, 1e4, 4.0), softcap=30.0)
    W = _mark_weights(_attention_weights(m, H, 800, td, False), m, td, False)
    h = _marked(T, H, [11], 801).to(td)
    plain = _plain_of(P.window_attention, m, W)
    ref = plain(h)
    h2 = h.clone()
    h2[11, 0] = 0
    assert (plain(h2)[-10:] - ref[-10:]).abs().max() > 0.3 * ref[-10:].abs().max()
    part = _window_part(W, m, H, td)
    tol = 1e-4 if dtype == "float32" else 5e-2
    assert rel_err(run_alone(part, h, [T], td), ref) < tol
    assert rel_err(run_alone(part, h, [900] + [1] * 30, td)[-30:], ref[-30:]) < tol


# ------------------------------------------------------------ the scans
def _mamba_weights(m, H, seed, td):
    n, N, r = m["inner"], m["state"], m["dt_rank"]
    lin = 1.0 / H ** 0.5
    W = {"in": rnd(2 * n, H, seed=seed, std=1.3 * lin), "conv": rnd(n, m["conv"], seed=seed + 1, std=0.6) + 0.3,
         "conv.b": rnd(n, seed=seed + 2, std=0.2), "x": rnd(r + 2 * N, n, seed=seed + 3, std=1.5 / n ** 0.5),
         "dt": rnd(n, r, seed=seed + 4, std=0.6 / r ** 0.5), "dt.b": rnd(n, seed=seed + 5, std=0.8) - 2.0,
         "A_log": rnd(n, N, seed=seed + 6, std=2.0) - 1.5, "D": rnd(n, seed=seed + 7, std=0.3) + 0.8,
         "o": rnd(H, n, seed=seed + 8, std=1.0 / n ** 0.5)}
    return {k: v.to(td) for k, v in W.items()}


def _mamba_part(W, m, H, td):
    from agave_b200.config.base import SelectiveScanSpec
    from agave_b200.parts.state_space import SelectiveScanMixer
    spec = SelectiveScanSpec(inner=m["inner"], state=m["state"], dt_rank=m["dt_rank"],
                             conv_taps=m["conv"])
    part = SelectiveScanMixer(spec, H, td, torch.device(DEV))
    names = {"in": "in_proj.weight", "conv": "conv.weight", "conv.b": "conv.bias",
             "x": "x_proj.weight", "dt": "dt_proj.weight", "dt.b": "dt_proj.bias",
             "A_log": "a_log", "D": "d", "o": "o_proj.weight"}
    t = {names[k]: v for k, v in W.items()}
    assert set(t) == set(SelectiveScanMixer.param_specs(spec, H))
    part.load(t, td, torch.device(DEV))
    return part


def _mamba2_weights(m, H, seed, td):
    A, dv, N, G = m["heads"], m["vdim"], m["state"], m["groups"]
    C = A * dv + 2 * G * N
    lin = 1.0 / H ** 0.5
    W = {"in": rnd(A * dv + C + A, H, seed=seed, std=1.3 * lin),
         "conv": rnd(C, m["conv"], seed=seed + 1, std=0.6) + 0.3, "conv.b": rnd(C, seed=seed + 2, std=0.2),
         "dt_bias": rnd(A, seed=seed + 3) - 2.0, "A_log": rnd(A, seed=seed + 4, std=2.0) - 1.5,
         "D": rnd(A, seed=seed + 5, std=0.3) + 0.8, "norm": rnd(A * dv, seed=seed + 6, std=0.3) + 1.0,
         "o": rnd(H, A * dv, seed=seed + 7, std=1.0 / (A * dv) ** 0.5)}
    return {k: v.to(td) for k, v in W.items()}


def _mamba2_part(W, m, H, td):
    from agave_b200.parts.state_space import StateSpaceMixer
    spec = _spec_of("mamba2", m)
    part = StateSpaceMixer(spec, H, td, torch.device(DEV))
    names = {"in": "in_proj.weight", "conv": "conv.weight", "conv.b": "conv.bias",
             "dt_bias": "dt_bias", "A_log": "a_log", "D": "d", "norm": "out_norm.weight",
             "o": "o_proj.weight"}
    t = {names[k]: v for k, v in W.items()}
    assert set(t) == set(StateSpaceMixer.param_specs(spec, H))
    part.load(t, td, torch.device(DEV))
    return part


def _m2(*a):
    return mamba2(*a)[1]


MAMBA = [(72, scan(36, 5, 3, 2)), (128, scan(192, 16, 8, 4)), (96, scan(8, 1, 1, 1)),
         (76, scan(53, 24, 5, 7)), (64, scan(200, 33, 16, 3)), (48, scan(64, 8, 4, 8)),
         (40, scan(24, 128, 2, 4)), (40, scan(12, 200, 3, 2)), (64, scan(130, 3, 2, 4))]
MAMBA2 = [(72, _m2(6, 10, 12, 3, 2, 3)), (128, _m2(4, 64, 64, 1, 1, 4)), (96, _m2(1, 16, 1, 1, 1, 1)),
          (76, _m2(5, 33, 18, 5, 1, 6)), (64, _m2(2, 7, 130, 2, 7, 2)), (48, _m2(6, 40, 44, 2, 3, 8)),
          (64, _m2(2, 128, 256, 1, 2, 4)), (80, _m2(3, 8, 8, 3, 3, 2)),
          # (enough heads for the scan's form with two columns a lane, its last ones partly empty)
          (32, _m2(100, 41, 20, 50, 4, 2))]


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("kind, H, m", [("mamba", *c) for c in MAMBA] + [("mamba2", *c) for c in MAMBA2])
def test_scans_as_prompt_and_token_by_token(dtype, kind, H, m):
    """Each scan alone: the whole sequence in one step; a prompt and then tokens one by one,
    from cuts at the first token, before the convolution is full, and at a border of the scan's
    chunks of tokens."""
    td = TD[dtype]
    T = 90
    if kind == "mamba":
        W = _mamba_weights(m, H, 70, td)
        part, plain = _mamba_part(W, m, H, td), lambda h, w: P.mamba(h, m, w, "")
    else:
        W = _mamba2_weights(m, H, 80, td)
        part, plain = _mamba2_part(W, m, H, td), lambda h, w: P.mamba2(h, m, w, "", 1e-5)
    h = rnd(T, H, seed=71).to(td)
    ref = plain(h.double(), {k: v.double() for k, v in W.items()})
    tol = 5e-5 if dtype == "float32" else 4e-2
    for new in ([T], [50] + [1] * 40, [1] * T, [2] + [1] * 88, [16] + [1] * 74, [33] + [1] * 57):
        assert rel_err(run_alone(part, h, new, td), ref) < tol, new[:2]


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("kind", ["mamba", "mamba2"])
def test_scans_unequal_batches_and_slots_used_again(dtype, kind):
    """A freed slot's state and stored convolution inputs must start at zero again; the last
    round's prompt is long enough for the convolution's form with several tokens a thread, whose
    tiles straddle the sequences."""
    td = TD[dtype]
    H = 96
    if kind == "mamba":
        m = scan(120, 16, 6, 4)
        W = _mamba_weights(m, H, 90, td)
        part, plain = _mamba_part(W, m, H, td), lambda h, w: P.mamba(h, m, w, "")
    else:
        m = _m2(4, 24, 40, 2, 2, 4)
        W = _mamba2_weights(m, H, 95, td)
        part, plain = _mamba2_part(W, m, H, td), lambda h, w: P.mamba2(h, m, w, "", 1e-5)
    Wd = {k: v.double() for k, v in W.items()}
    run_batches(part, lambda h: plain(h, Wd), H, td, 5e-5 if dtype == "float32" else 4e-2, ROUNDS)


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("kind", ["mamba", "mamba2"])
def test_what_a_scan_took_in_hundreds_of_tokens_ago_decides(dtype, kind):
    """Decays next to one and a step size that only one early token makes large: the read-out
    600 tokens later is mostly what that token wrote, and decoding must still have it.  The
    convolution passes the current token, D is zero."""
    td = TD[dtype]
    H, T, far = 64, 640, 9
    h = rnd(T, H, seed=501)
    h[:, 5] = 0.0
    h[far, 5] = 3.0
    if kind == "mamba":
        m = scan(48, 8, 2, 3)
        W = {k: v.double() for k, v in _mamba_weights(m, H, 500, td).items()}
        # u's last channel reads axis 5; the step sizes come from it alone
        W["in"][47] = 0.0
        W["in"][47, 5] = 2.0
        W["conv.b"][:] = 0.0
        W["x"][:2] = 0.0
        W["x"][:2, 47] = 1.0
        W["dt"] = torch.full_like(W["dt"], 0.6)
        W["dt.b"][:] = -6.0
        W["A_log"] = rnd(48, 8, seed=502) - 7.0
    else:
        m = _m2(4, 12, 16, 2, 1, 3)
        W = {k: v.double() for k, v in _mamba2_weights(m, H, 510, td).items()}
        W["in"][-4:] = 0.0
        W["in"][-4:, 5] = 2.5
        W["conv.b"][:] = 0.0
        W["dt_bias"][:] = -6.0
        W["A_log"] = rnd(4, seed=512) - 7.0
    W["conv"][:] = 0.0
    W["conv"][:, -1] = 1.0
    W["D"][:] = 0.0
    W = {k: v.to(td) for k, v in W.items()}
    h = h.to(td)
    Wd = {k: v.double() for k, v in W.items()}
    plain = (lambda x: P.mamba(x, m, Wd, "")) if kind == "mamba" else \
        (lambda x: P.mamba2(x, m, Wd, "", 1e-5))
    part = _mamba_part(W, m, H, td) if kind == "mamba" else _mamba2_part(W, m, H, td)
    ref = plain(h.double())
    h2 = h.clone()
    h2[far, 5] = 0
    other = plain(h2.double())
    assert (other[-20:] - ref[-20:]).abs().max() > 0.3 * ref[-20:].abs().max()
    got = run_alone(part, h, [600] + [1] * 40, td)
    tol = 2e-4 if dtype == "float32" else 5e-2
    assert rel_err(got[-40:], ref[-40:]) < tol
    assert rel_err(got[20:], ref[20:]) < 2 * tol


@pytest.mark.parametrize("dtype", DTYPES)
def test_two_mixers_side_by_side(dtype):
    """The sum a block that knows nothing of the two gets, and the terms one that joins them
    itself gets; decoding through one cache entry that holds keys, values and a state."""
    from agave_b200.parts.parallel import SideBySideMixer
    td = TD[dtype]
    H, T = 96, 70
    m = {"left": heads(4, 2, 16, 24, 0.3, size=20, rot=rotation(8, 1e3)), "right": scan(40, 6, 3, 3),
         "left_scale": 1.7, "right_scale": -0.4}
    Wl = _attention_weights(m["left"], H, 10, td, True)
    Wr = _mamba_weights(m["right"], H, 30, td)
    spec = _spec_of("parallel", m)
    part = SideBySideMixer(spec, H, td, torch.device(DEV))
    left, right = _chunked_part(Wl, m["left"], H, td), _mamba_part(Wr, m["right"], H, td)
    part.left, part.right = left, right
    h = rnd(T, H, seed=40).to(td)
    w = {**{f"left.{k}": v.double() for k, v in Wl.items()},
         **{f"right.{k}": v.double() for k, v in Wr.items()}}
    ref = P.mixer("parallel", h.double(), m, w, "", 1e-5)
    tol = 5e-5 if dtype == "float32" else 4e-2
    for new in ([T], [30] + [1] * 40):
        assert rel_err(run_alone(part, h, new, td), ref) < tol
    terms = part.forward_terms(h.to(DEV), _Cache(part.cache_request(), 1, td).step([T]), 0, True)
    assert [s for _, s in terms] == pytest.approx([1.7, -0.4])
    assert rel_err(sum(s * summed(y) for y, s in terms), ref) < tol


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


@pytest.mark.parametrize("name", NAMES)
def test_the_stream_after_every_layer(name):
    """32-bit: the residual stream after each layer run against the plain model's, so that a
    fault names its layer."""
    eng, folder = engine_for(name, "float32")
    toks = tokens(25, vocab(name), 9)
    streams = []
    plain_logits(folder, toks, streams)
    model = eng.model
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
        assert rel_err(h, streams[upto - 1]) < 2e-5, f"layer {upto - 1}"


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("name", NAMES)
def test_whole_prompts_alone(name, dtype):
    eng, folder = engine_for(name, dtype)
    for n in (1, 2, 7, 8, 64, 65, 300):
        toks = tokens(n, vocab(name), 20 + n)
        s = eng.acquire()
        got = eng.step([(s, toks)], [list(range(n))])
        eng.release(s)
        rows_agree(got, plain_logits(folder, toks), dtype, f"{name} {n} tokens")


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("name", NAMES)
def test_prompt_then_tokens_one_by_one(name, dtype):
    """Decoding starts after one token, inside the first window and chunk, at a page border, and
    runs past several edges."""
    eng, folder = engine_for(name, dtype)
    for n, cut in ((100, 60), (41, 1), (200, 127), (140, 64), (12, 2)):
        toks = tokens(n, vocab(name), 11 + n)
        rows_agree(alone(eng, toks, cut), plain_logits(folder, toks), dtype, f"{name} {n}/{cut}")


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
                if at[i] == len(seqs[i]):
                    eng.release(slots[i])
        for i in range(len(seqs)):
            rows_agree(torch.cat(got[i]), plain_logits(folder, seqs[i]), dtype,
                       f"{name} round {round_} request {i}")


@pytest.mark.parametrize("name", NAMES)
def test_lengths_round_page_borders_window_and_chunk_edges(name):
    """32-bit: prompts that end just before, on and just after a page border and every window's
    and chunk's edge, each followed by three decoded tokens."""
    eng, folder = engine_for(name, "float32")
    edges = {63, 64, 65, 127, 128, 129}
    for l in CONFIGS[name]["layers"]:
        m = l["mixer"].get("left", l["mixer"])
        if m.get("mask"):
            w = m["mask"]["size"]
            edges |= {max(1, w - 1), w, w + 1, 2 * w - 1, 2 * w, 2 * w + 1}
    for n in sorted(edges):
        toks = tokens(n + 3, vocab(name), n)
        ref = plain_logits(folder, toks)
        s = eng.acquire()
        got = [eng.step([(s, toks[:n])], [[0, n - 1]])]
        for p in range(n, n + 3):
            got.append(eng.step([(s, [toks[p]])], [[0]]))
        eng.release(s)
        rows_agree(torch.cat(got), ref[[0, n - 1, n, n + 1, n + 2]], "float32", f"{name} {n}")


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("name", ["S1", "S2"])
def test_long_decoding(name, dtype):
    """300 tokens decoded after a prompt of 5: the rings of windows and chunks wrap more than
    once, the states go through 300 updates."""
    eng, folder = engine_for(name, dtype)
    toks = tokens(305, vocab(name), 77)
    rows_agree(alone(eng, toks, 5), plain_logits(folder, toks), dtype, name)


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
        ref = plain_logits(folder, p + g)
        for k, t in enumerate(g):
            row = ref[len(p) - 1 + k]
            misses += float(row.max() - row[t]) > slack * float(row.abs().max())
    assert misses <= (0 if dtype == "float32" else 2), misses


@pytest.mark.parametrize("dtype", DTYPES)
def test_generation_in_batches_of_the_slot_limit(dtype):
    """More prompts than slots: slots and their states are used again; the tokens are the same
    as with room for all."""
    from agave_b200.engine.api import Engine
    folder = folder_for("S1", TD[dtype])
    V = vocab("S1")
    prompts = [tokens(n, V, 900 + n) for n in (5, 66, 17, 3, 40, 21, 8)]
    wide = Engine(folder, dtype=dtype, max_tokens=4096)
    narrow = Engine(folder, dtype=dtype, max_tokens=4096, max_batch=3)
    a = wide.generate(prompts, max_new_tokens=10, stop_token_ids=[])
    b = narrow.generate(prompts, max_new_tokens=10, stop_token_ids=[])
    same = sum(x == y for x, y in zip(a, b))
    assert same >= (len(prompts) if dtype == "float32" else len(prompts) - 2)


def test_sampling_runs_on_this_architecture():
    eng, _ = engine_for("S1", "bfloat16")
    V = vocab("S1")
    kw = dict(max_new_tokens=8, temperature=0.8, top_k=20, top_p=0.9, seed=5, stop_token_ids=[])
    outs = eng.generate([tokens(6, V, 1), tokens(30, V, 2)], **kw)
    again = eng.generate([tokens(6, V, 1), tokens(30, V, 2)], **kw)
    assert outs == again and all(len(o) == 8 and all(0 <= t < V for t in o) for o in outs)


def test_random_weights_from_a_configuration():
    from agave_b200.engine.api import Engine
    raw = CONFIGS["S1"]
    eng = Engine.from_config(raw, seed=3, max_tokens=1024)
    outs = eng.generate([tokens(9, raw["vocab"], 1)], max_new_tokens=5, stop_token_ids=[])
    assert len(outs[0]) == 5
    info = eng.model_info()
    assert info["architecture"] == "Savovik" and info["weight_bytes"] > 0


@pytest.mark.parametrize("dtype", DTYPES)
def test_a_model_of_scans_alone(dtype):
    """No layer keeps keys and values: the cache holds fixed-size states and nothing else."""
    from agave_b200.engine.api import Engine
    from savovik_util import config, write_folder
    cfg = config(64, 90, [(mamba2(4, 16, 24, 2, 1, 4), 48), (mamba2(2, 8, 8, 1, 2, 2), None), 0])
    folder = write_folder(cfg, 4, TD[dtype])
    try:
        eng = Engine(folder, dtype=dtype, max_tokens=512)
        toks = tokens(90, 90, 3)
        rows_agree(alone(eng, toks, 40), plain_logits(folder, toks), dtype, "scans")
        outs = eng.generate([toks[:9], toks[:30]], max_new_tokens=4, stop_token_ids=[])
        assert [len(o) for o in outs] == [4, 4]
    finally:
        shutil.rmtree(folder, ignore_errors=True)


@pytest.mark.parametrize("dtype", DTYPES)
def test_trace_replay_as_a_process(dtype):
    name = "S2"
    folder = folder_for(name, TD[dtype])
    V = vocab(name)
    a, b = tokens(210, V, 5), tokens(33, V, 6)
    refs = {"a": plain_logits(folder, a), "b": plain_logits(folder, b)}
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
    out = tempfile.mkdtemp(prefix="savovik_trace_")
    try:
        r = subprocess.run([sys.executable, os.path.join(ROOT, "bin", "trace_run"), "--model",
                            folder, "--dtype", dtype, "--out", out, "--max-tokens", "300"],
                           input="\n".join(json.dumps(s) for s in steps) + "\n", text=True,
                           capture_output=True, timeout=900)
        assert r.returncode == 0, r.stderr[-2000:]
        assert [l for l in r.stdout.split("\n") if l.startswith("done")] == \
            [f"done {k}" for k in range(16)]
        got = torch.from_numpy(np.fromfile(os.path.join(out, "0.f32"), dtype="<f4").reshape(4, V))
        rows_agree(got, torch.stack([refs["a"][0], refs["a"][100], refs["a"][194], refs["b"][29]]),
                   dtype, "step 0")
        rows = []
        for k in range(15):
            want = [refs["a"][195 + k]]
            if k < 3 and k != 1:
                want.append(refs["b"][30 + k])
            g = np.fromfile(os.path.join(out, f"{k + 1}.f32"), dtype="<f4").reshape(len(want), V)
            rows.append((torch.from_numpy(g), torch.stack(want)))
        rows_agree(torch.cat([g for g, _ in rows]), torch.cat([w for _, w in rows]), dtype,
                   "decoded")
    finally:
        shutil.rmtree(out, ignore_errors=True)


def test_command_line_on_this_architecture():
    """``python -m agave_b200`` picks the model class from config.json: greedy tokens equal the
    plain model's, --model-info names the architecture, --profile lists this design's
    operations."""
    name = "S2"
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
    assert r.returncode == 0 and "Savovik" in r.stdout, r.stderr[-2000:]
    r = run(folder, "--tokens", toks, "-n", "3", "--profile", "--dtype", "bfloat16")
    assert r.returncode == 0, r.stderr[-2000:]
    for op in ("norm", "qkv", "qk_norm_rope", "attention", "ssm_conv", "selective_scan", "head_scan",
               "ssd_out", "x_proj", "dt_proj", "gates", "up", "out_proj", "down", "lm_head", "TOTAL"):
        assert op in r.stderr, (op, r.stderr[-1500:])


@pytest.mark.parametrize("name, room", [("S1", 60), ("S2", 90), ("S3", 64), ("S4", 100)])
def test_a_cache_shorter_than_a_page_or_a_window(name, room):
    """32-bit: a cache of one or two pages.  A window or chunk that still fits a sequence keeps
    its edge; one that no sequence can outgrow is none."""
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
    assert math.isfinite(float(torch.zeros(1, device=DEV)))
