"""Small Savovik configurations and a writer of model folders for the tests.

The writer makes every tensor under its checkpoint name from the configuration dictionary
alone (it does not ask the library which names it expects), with scales chosen so that faults
show: scores of order one, decays from fast ones to some so close to one that a state lost
hundreds of tokens ago is missed, gates spread round one half.
"""
import atexit
import json
import os
import shutil
import tempfile

import torch


def rotation(dims, base, scaling=None):
    """``scaling``: a factor, or (factor, low, high, original)."""
    r = {"base": base, "dims": dims}
    if scaling is not None:
        r["scaling"] = ({"factor": scaling} if not isinstance(scaling, tuple) else
                        dict(zip(("factor", "low", "high", "original"), scaling)))
    return r


def heads(n, kv_heads, dim, vdim, scale, size=None, rot=None, softcap=None):
    """The part of a layer entry both attentions share."""
    m = {"dim": dim, "heads": n, "kv_heads": kv_heads, "scale": scale, "vdim": vdim}
    if size is not None:
        m["mask"] = {"size": size}
    if rot is not None:
        m["rot"] = rot
    if softcap is not None:
        m["softcap"] = softcap
    return m


def scan(inner, state, dt_rank, conv):
    return {"conv": conv, "dt_rank": dt_rank, "inner": inner, "state": state}


def parallel(left, right, left_scale=1.0, right_scale=1.0):
    return "parallel", {"left": left, "left_scale": left_scale, "right": right,
                        "right_scale": right_scale}


def attention(*a, **k):
    return "attention", heads(*a, **k)


def mamba2(n, vdim, state, groups, norm_groups, conv):
    return "mamba2", {"conv": conv, "groups": groups, "heads": n, "norm_groups": norm_groups,
                      "state": state, "vdim": vdim}


def config(width, vocab, layers, eps=1e-5):
    """``layers``: ((type, mixer), feed-forward width or None), or the number of an earlier layer
    whose weights this one runs."""
    out = []
    for entry in layers:
        if isinstance(entry, int):
            out.append({**{k: v for k, v in out[entry].items() if k != "weights_of"},
                        "weights_of": entry})
        else:
            (kind, m), ff = entry
            out.append({"mixer": m, "type": kind,
                        "mlp": None if ff is None else {"ff": ff, "kind": "dense"}})
    return {"architecture": "Savovik", "layers": out, "norm": {"eps": eps}, "vocab": vocab,
            "width": width}


# S1: small odd sizes (every kernel's general form): a chunk and a window shorter than a page,
# part of the head rotated with both kinds of scaled frequencies, value heads wider and narrower
# than the keys, more norm parts than groups and the other way round, a layer without a
# feed-forward, layers that run another's weights (each kind of mixer).
S1 = config(72, 210, [
    (parallel(heads(4, 2, 10, 14, 0.4, size=7, rot=rotation(6, 10000.0, (8.0, 1.0, 4.0, 16))),
              scan(36, 5, 3, 2), 1.3, 0.7), 40),
    (mamba2(6, 10, 12, 3, 2, 3), None),
    (attention(3, 1, 12, 6, 0.35, size=9, rot=rotation(8, 300.0, 2.5), softcap=5.0), 56),
    0,
    (mamba2(4, 6, 20, 1, 4, 4), 24),
    1,
    2,
], eps=1e-5)

# S2: the sizes that take the tensor-core kernels (head sizes 64 and 128, groups of four query
# heads, a window and a chunk that cross pages).
S2 = config(128, 320, [
    (attention(8, 2, 64, 64, 0.13, size=100, rot=rotation(64, 10000.0, 4.0), softcap=20.0), 192),
    (parallel(heads(4, 1, 64, 128, 0.12, size=70, rot=rotation(32, 500.0, (4.0, 2.0, 8.0, 64))),
              scan(192, 16, 8, 4), 0.6, 1.4), 128),
    (mamba2(4, 64, 64, 1, 1, 4), 256),
    (attention(4, 2, 128, 64, 0.09, size=70, rot=rotation(64, 10000.0, 8.0), softcap=3.0), None),
    1,
    2,
], eps=1e-6)

# S3: values the other two make unequal are equal here or 1, and what may be absent is: one head,
# as many kv heads as heads, one state, a rank of one, one tap, a chunk of one, a window of
# exactly a page, no mask, no rotation, no cap, scales of one, one group of each kind and as many
# groups as heads.
S3 = config(96, 150, [
    (parallel(heads(1, 1, 16, 16, 0.3, size=1), scan(8, 1, 1, 1)), 32),
    (mamba2(1, 16, 1, 1, 1, 1), None),
    (attention(2, 2, 24, 24, 0.3, size=64), 48),
    (mamba2(3, 8, 8, 3, 3, 2), 96),
    (parallel(heads(2, 2, 32, 32, 0.25, size=64, rot=rotation(32, 50.0)), scan(96, 4, 6, 5)), None),
    (attention(2, 1, 32, 32, 0.25, rot=rotation(32, 50.0)), 16),
    (parallel(heads(2, 1, 16, 48, 0.25), scan(40, 33, 2, 3), 1.0, 2.0), 24),
], eps=3e-6)

# S4: a width, a vocabulary and inner sizes that are no multiples of 8 (no product takes the
# tensor cores), states no power of two, the order turned round.
S4 = config(76, 211, [
    (mamba2(5, 33, 18, 5, 1, 6), 36),
    (attention(6, 3, 20, 12, 0.3, size=33, rot=rotation(10, 2000.0, 3.0), softcap=30.0), 44),
    (mamba2(2, 7, 130, 2, 7, 2), None),
    (parallel(heads(3, 3, 18, 22, 0.3, size=50, rot=rotation(18, 2000.0, (2.0, 1.0, 2.0, 40))),
              scan(53, 24, 5, 7), 0.9, 1.1), 20),
    1,
], eps=2e-5)

CONFIGS = {"S1": S1, "S2": S2, "S3": S3, "S4": S4}


def make_tensors(cfg, seed, dtype):
    g = torch.Generator().manual_seed(seed)

    def rnd(*shape, std=1.0, mean=0.0):
        return (torch.randn(*shape, generator=g) * std + mean).to(dtype)

    H, V = cfg["width"], cfg["vocab"]
    lin = 1.0 / H ** 0.5                                   # unit outputs from a unit stream
    t = {"embed": rnd(V, H), "head": rnd(V, H, std=lin), "final.norm": rnd(H, std=0.3)}

    def attn(p, m, extras):
        A, G, d, dv = m["heads"], m["kv_heads"], m["dim"], m["vdim"]
        for n, rows, std in (("q", A * d, 1.5), ("k", G * d, 1.5), ("v", G * dv, 1.0)):
            t[p + n] = rnd(rows, H, std=std * lin)
            if extras:
                t[p + n + ".b"] = rnd(rows, std=0.4)
        if extras:
            t[p + "q.norm"] = rnd(d, std=0.3, mean=1.2)
            t[p + "k.norm"] = rnd(d, std=0.3, mean=1.2)
        t[p + "o"] = rnd(H, A * dv, std=1.0 / (A * dv) ** 0.5)

    for i, layer in enumerate(cfg["layers"]):
        if layer.get("weights_of") is not None:
            continue
        p, m = f"l{i}.", layer["mixer"]
        t[p + "norm1"] = rnd(H, std=0.2)
        if layer["type"] == "attention":
            attn(p + "mix.", m, False)
        elif layer["type"] == "parallel":
            attn(p + "mix.left.", m["left"], True)
            r, q = m["right"], p + "mix.right."
            n, N, rank = r["inner"], r["state"], r["dt_rank"]
            t[q + "in"] = rnd(2 * n, H, std=1.3 * lin)
            t[q + "conv"] = rnd(n, r["conv"], std=0.6, mean=0.3)
            t[q + "conv.b"] = rnd(n, std=0.2)
            t[q + "x"] = rnd(rank + 2 * N, n, std=1.5 / n ** 0.5)
            t[q + "dt"] = rnd(n, rank, std=0.6 / rank ** 0.5)
            t[q + "dt.b"] = rnd(n, std=0.8, mean=-2.0)
            t[q + "A_log"] = rnd(n, N, std=2.0, mean=-1.5)
            t[q + "D"] = rnd(n, std=0.3, mean=0.8)
            t[q + "o"] = rnd(H, n, std=1.0 / n ** 0.5)
        else:
            A, dv, N, G = m["heads"], m["vdim"], m["state"], m["groups"]
            C = A * dv + 2 * G * N
            t[p + "mix.in"] = rnd(A * dv + C + A, H, std=1.3 * lin)
            t[p + "mix.conv"] = rnd(C, m["conv"], std=0.6, mean=0.3)
            t[p + "mix.conv.b"] = rnd(C, std=0.2)
            t[p + "mix.dt_bias"] = rnd(A, std=1.0, mean=-2.0)
            t[p + "mix.A_log"] = rnd(A, std=2.0, mean=-1.5)
            t[p + "mix.D"] = rnd(A, std=0.3, mean=0.8)
            t[p + "mix.norm"] = rnd(A * dv, std=0.3, mean=1.0)
            t[p + "mix.o"] = rnd(H, A * dv, std=1.0 / (A * dv) ** 0.5)
        t[p + "rg1"] = rnd(H, H, std=1.5 * lin)
        t[p + "rg1.b"] = rnd(H, std=0.5)
        if layer["mlp"] is not None:
            ff = layer["mlp"]["ff"]
            t[p + "mlp.up"] = rnd(ff, H, std=1.5 * lin)
            t[p + "mlp.down"] = rnd(H, ff, std=1.0 / ff ** 0.5)
            t[p + "rg2"] = rnd(H, H, std=1.5 * lin)
            t[p + "rg2.b"] = rnd(H, std=0.5)
    return t


_FOLDERS = {}


def write_folder(cfg, seed, dtype, prefix="savovik_"):
    from safetensors.torch import save_file
    d = tempfile.mkdtemp(prefix=prefix)
    with open(os.path.join(d, "config.json"), "w") as f:
        json.dump(cfg, f)
    save_file({k: v.contiguous() for k, v in make_tensors(cfg, seed, dtype).items()},
              os.path.join(d, "model.safetensors"))
    return d


def folder_for(name, dtype=torch.float32, seed=0):
    """A temporary model folder of configuration ``name`` (made once per run)."""
    key = (name, dtype, seed)
    if key not in _FOLDERS:
        _FOLDERS[key] = write_folder(CONFIGS[name], seed, dtype, prefix=f"savovik_{name}_")
    return _FOLDERS[key]


def _cleanup():
    for d in _FOLDERS.values():
        shutil.rmtree(d, ignore_errors=True)


atexit.register(_cleanup)


def tokens(n, vocab, seed):
    g = torch.Generator().manual_seed(seed)
    return torch.randint(0, vocab, (n,), generator=g).tolist()


_READ = {}
_DONE = {}


def plain_logits(folder, toks, streams=None):
    from plain import savovik_plain as P
    from safetensors.torch import load_file
    if folder not in _READ:
        with open(os.path.join(folder, "config.json")) as f:
            _READ[folder] = (json.load(f), load_file(os.path.join(folder, "model.safetensors")))
    cfg, w = _READ[folder]
    key = (folder, tuple(toks))
    if streams is not None or key not in _DONE:
        out = P.forward(cfg, w, toks, layers_out=streams)
        if len(_DONE) > 200:
            _DONE.clear()
        _DONE[key] = out
    return _DONE[key]
