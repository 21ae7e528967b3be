"""Small Pubunex configurations and a writer of model folders for the tests.

The writer makes every tensor under its checkpoint name from the configuration dictionary
alone (it does not ask the library which names it expects), with scales chosen so that faults
show: scores of order one, sinks that take a good share, decays from fast ones to some so close
to one that a state lost hundreds of tokens ago is missed, expert gates and inputs on both sides
of their bounds, router scores spread over (0, 1).
"""
import atexit
import json
import os
import shutil
import tempfile

import torch


def rotation(dims, base, scaling=None):
    """``scaling``: (factor, original, fast, slow)."""
    r = {"base": base, "dims": dims}
    if scaling is not None:
        r["scaling"] = dict(zip(("factor", "original", "fast", "slow"), scaling))
    return r


def delta(heads, kv_heads, dim, vdim, conv):
    return "delta", {"conv": conv, "dim": dim, "heads": heads, "kv_heads": kv_heads, "vdim": vdim}


def attention(heads, kv_heads, dim, vdim, scale, rot=None):
    m = {"dim": dim, "heads": heads, "kv_heads": kv_heads, "scale": scale, "vdim": vdim}
    if rot is not None:
        m["rot"] = rot
    return "attention", m


def latent(heads, dim, rot_dim, vdim, kv_rank, scale, base=10000.0):
    return "latent_attention", {"dim": dim, "heads": heads, "kv_rank": kv_rank,
                                "rot": rotation(rot_dim, base), "rot_dim": rot_dim,
                                "scale": scale, "vdim": vdim}


def moe(experts, top, ff, limit, shared=None, shared_limit=None):
    f = {"expert": {"ff": ff, "limit": limit}, "kind": "moe",
         "router": {"experts": experts, "top": top}}
    if shared is not None:
        f["shared"] = {"ff": shared, "limit": limit if shared_limit is None else shared_limit}
    return f


def config(width, vocab, layers, loop=None, eps=1e-5):
    """``layers``: ((type, mixer), feed-forward or None); ``loop``: (start, stop, times)."""
    d = {"architecture": "Pubunex",
         "layers": [{"mixer": m, "mlp": f, "type": kind} for (kind, m), f in layers],
         "norm": {"eps": eps}, "vocab": vocab, "width": width}
    if loop is not None:
        d["loop"] = dict(zip(("start", "stop", "times"), loop))
    return d


# P1: small odd sizes (every kernel's general form): value heads wider and narrower than the
# keys, part of the head rotated, a layer without a feed-forward inside the loop, layers before
# and behind it, three passes, experts and their shared one with bounds of their own.
P1 = config(72, 210, [
    (attention(4, 2, 10, 14, 0.4, rotation(6, 1000.0, (8.0, 64, 4.0, 0.5))), moe(5, 2, 24, 0.8, 20, 2.5)),
    (delta(4, 2, 10, 14, 3), moe(3, 1, 20, 1.5, 12)),
    (latent(3, 10, 4, 6, 20, 0.35), None),
    (delta(6, 1, 18, 7, 2), moe(4, 3, 16, 0.6, 24)),
    (latent(2, 6, 8, 12, 14, 0.4, 300.0), moe(6, 2, 12, 3.0)),
], loop=(1, 4, 3))

# P2: the sizes that take the tensor-core kernels.
P2 = config(128, 320, [
    (latent(4, 48, 16, 64, 64, 0.13), moe(8, 2, 64, 1.2, 128, 0.7)),
    (attention(8, 2, 64, 128, 0.12, rotation(32, 20000.0, (4.0, 256, 16.0, 1.0))), moe(8, 3, 64, 2.0, 64)),
    (delta(4, 2, 64, 64, 4), moe(4, 1, 128, 0.9, 64)),
    (delta(2, 2, 128, 64, 4), None),
], loop=(0, 3, 2), eps=1e-6)

# P3: values the others make unequal are equal here or 1, and what may be absent is: one head,
# as many kv heads as heads, one tap, one expert, every expert chosen, no shared expert, no
# loop, no rotation, no scaling, the whole head rotated.
P3 = config(96, 150, [
    (delta(1, 1, 16, 16, 1), moe(1, 1, 16, 1.0)),
    (attention(2, 2, 24, 24, 0.3), moe(4, 4, 16, 1.0, 16)),
    (latent(1, 16, 16, 16, 16, 0.3, 50.0), moe(2, 1, 32, 1.0, 32, 1.0)),
    (attention(1, 1, 32, 32, 0.25, rotation(32, 50.0)), None),
    (delta(3, 3, 8, 8, 4), moe(2, 2, 8, 1.0)),
], eps=3e-6)

# P4: a width, a vocabulary and inner sizes that are no multiples of 8 (no product takes the
# tensor cores), a delta head beyond 128, every layer in the loop, one layer a loop's whole body.
P4 = config(76, 211, [
    (delta(2, 1, 130, 33, 6), moe(3, 2, 18, 1.1, 26, 0.5)),
    (attention(6, 3, 20, 12, 0.3, rotation(10, 2000.0, (2.0, 40, 8.0, 1.0))), moe(5, 1, 22, 0.7, 14)),
    (latent(3, 9, 6, 11, 33, 0.3, 2000.0), moe(7, 5, 10, 1.4, 9)),
], loop=(0, 3, 2), eps=2e-5)
P5 = config(64, 130, [
    (attention(4, 1, 16, 16, 0.3, rotation(8, 1000.0)), moe(4, 2, 16, 1.0, 16)),
    (delta(8, 4, 16, 16, 4), moe(4, 2, 32, 1.5, 32)),
], loop=(1, 2, 4))

CONFIGS = {"P1": P1, "P2": P2, "P3": P3, "P4": P4, "P5": P5}


def make_tensors(cfg, seed, dtype):
    g = torch.Generator().manual_seed(seed)

    def rnd(*shape, std=1.0, mean=0.0):
        return (torch.randn(*shape, generator=g) * std + mean).to(dtype)

    H, V = cfg["width"], cfg["vocab"]
    lin = 1.0 / H ** 0.5                                   # unit outputs from a unit stream
    t = {"embed": rnd(V, H), "head": rnd(V, H, std=lin), "final.norm": rnd(H, std=0.3)}
    for i, layer in enumerate(cfg["layers"]):
        p, m = f"l{i}.", layer["mixer"]
        q = p + "mix."
        t[p + "norm1"] = rnd(H, std=0.2)
        A, d, dv = m["heads"], m["dim"], m["vdim"]
        if layer["type"] == "delta":
            G = m["kv_heads"]
            for n, rows in (("q", G * d), ("k", G * d), ("v", A * dv)):
                t[q + n] = rnd(rows, H, std=1.3 * lin)
                t[f"{q}{n}.conv"] = rnd(rows, m["conv"], std=0.6, mean=0.3)
            t[q + "b"] = rnd(A, H, std=1.5 * lin)
            t[q + "a"] = rnd(A, H, std=lin)
            t[q + "A_log"] = rnd(A, std=2.0, mean=-1.5)
            t[q + "dt_bias"] = rnd(A, std=1.0, mean=-2.0)
            t[q + "g"] = rnd(A * dv, H, std=1.3 * lin)
            t[q + "norm"] = rnd(dv, std=0.3, mean=1.0)
            t[q + "o"] = rnd(H, A * dv, std=1.0 / (A * dv) ** 0.5)
        elif layer["type"] == "attention":
            G = m["kv_heads"]
            for n, rows, std in (("q", A * d, 1.5), ("k", G * d, 1.5), ("v", G * dv, 1.0)):
                t[q + n] = rnd(rows, H, std=std * lin)
                t[q + n + ".b"] = rnd(rows, std=0.4)
            t[q + "o"] = rnd(H, A * dv, std=1.0 / (A * dv) ** 0.5)
            t[q + "o.b"] = rnd(H, std=0.3)
        else:
            r, R = m["rot_dim"], m["kv_rank"]
            t[q + "q"] = rnd(A * (d + r), H, std=1.5 * lin)
            t[q + "dkv"] = rnd(R + r, H, std=1.3 * lin)
            t[q + "dkv.norm"] = rnd(R, std=0.3, mean=1.2)
            t[q + "uk"] = rnd(A * d, R, std=1.3 / R ** 0.5)
            t[q + "uv"] = rnd(A * dv, R, std=1.0 / R ** 0.5)
            t[q + "sink"] = rnd(A, std=1.0, mean=1.5)
            t[q + "o"] = rnd(H, A * dv, std=1.0 / (A * dv) ** 0.5)
        f = layer["mlp"]
        if f is None:
            continue
        q = p + "mlp."
        t[q + "router"] = rnd(f["router"]["experts"], H, std=2.0 * lin)
        for n, ff in [(f"e{e}", f["expert"]["ff"]) for e in range(f["router"]["experts"])] + \
                ([("shared", f["shared"]["ff"])] if f.get("shared") else []):
            t[f"{q}{n}.gate"] = rnd(ff, H, std=1.6 * lin)
            t[f"{q}{n}.up"] = rnd(ff, H, std=1.6 * lin)
            t[f"{q}{n}.down"] = rnd(H, ff, std=1.0 / ff ** 0.5)
    return t


_FOLDERS = {}


def write_folder(cfg, seed, dtype, prefix="pubunex_"):
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
        _FOLDERS[key] = write_folder(CONFIGS[name], seed, dtype, prefix=f"pubunex_{name}_")
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


def plain_logits(folder, toks, streams=None, choices=None):
    from plain import pubunex_plain as P
    from safetensors.torch import load_file
    if folder not in _READ:
        with open(os.path.join(folder, "config.json")) as f:
            _READ[folder] = (json.load(f), load_file(os.path.join(folder, "model.safetensors")))
    cfg, w = _READ[folder]
    if streams is not None or choices is not None:
        return P.forward(cfg, w, toks, layers_out=streams, choices=choices)
    key = (folder, tuple(toks))
    if key not in _DONE:
        if len(_DONE) > 200:
            _DONE.clear()
        _DONE[key] = P.forward(cfg, w, toks)
    return _DONE[key]
