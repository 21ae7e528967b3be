"""Pubunex, written out plainly: one function per mechanism, 64-bit, the recurrence token by
token.  Nothing here is shared with the library; the tests compare the two.

``cfg`` is the parsed ``config.json`` of a model; ``w`` maps checkpoint names to tensors.
"""
from __future__ import annotations

import math
from typing import Dict, List, Optional

import torch

F = torch.float64


def silu(z):
    return z * torch.sigmoid(z)


def softplus(z):
    return torch.log1p(torch.exp(-z.abs())) + z.clamp(min=0.0)


def rms(x, eps):
    """x over the root of its mean square, eps under the root, along the last axis."""
    return x / torch.sqrt((x * x).mean(-1, keepdim=True) + eps)


def norm_around_zero(x, weight, eps):
    return rms(x, eps) * (1.0 + weight.to(F))


def lin(x, w, name, bias: bool = False):
    y = x @ w[name].to(F).T
    return y + w[name + ".b"].to(F) if bias else y


# ------------------------------------------------------------------ positions
def frequencies(rot: dict):
    """(the frequencies of the pairs, the factor on cos and sin).  A pair that turns often
    within the original context keeps its frequency, one that hardly turns has it divided, a
    ramp over the pair's number between."""
    dims, base = rot["dims"], rot["base"]
    f = [base ** (-2.0 * i / dims) for i in range(dims // 2)]
    sc = rot.get("scaling")
    if sc is None:
        return f, 1.0

    def pair(turns):
        return dims * math.log(sc["original"] / (2.0 * math.pi * turns)) / (2.0 * math.log(base))
    lo = max(math.floor(pair(sc["fast"])), 0)
    hi = min(math.ceil(pair(sc["slow"])), dims - 1)
    out = []
    for i, fi in enumerate(f):
        ramp = (i - lo) / max(hi - lo, 0.001)
        ramp = 0.0 if ramp < 0.0 else 1.0 if ramp > 1.0 else ramp
        out.append(ramp * fi / sc["factor"] + (1.0 - ramp) * fi)
    return out, 1.0 + 0.1 * math.log(sc["factor"])


def rotate(x, positions, rot: dict, neighbours: bool):
    """x [T, heads, dim]: pairs (2i, 2i + 1) or (i, i + dims / 2) of the first rot.dims
    dimensions of every head turn by position * f_i."""
    dims = rot["dims"]
    f, mult = frequencies(rot)
    a = positions.to(F)[:, None] * torch.tensor(f, dtype=F)[None, :]
    c, s = (torch.cos(a) * mult)[:, None, :], (torch.sin(a) * mult)[:, None, :]
    y = x.clone()
    if neighbours:
        u, v = x[..., 0:dims:2], x[..., 1:dims:2]
        y[..., 0:dims:2] = u * c - v * s
        y[..., 1:dims:2] = v * c + u * s
    else:
        half = dims // 2
        u, v = x[..., :half], x[..., half:dims]
        y[..., :half] = u * c - v * s
        y[..., half:dims] = v * c + u * s
    return y


# ------------------------------------------------------------------ attention
def attend(q, k, v, scale: float, sink=None):
    """q [T, H, dim], k [T, G, dim], v [T, G, vdim] -> [T, H * vdim]; causal.  ``sink`` [H]: a
    logit whose exponential is one more term of the denominator."""
    T, H, _ = q.shape
    G = k.shape[1]
    see = torch.tril(torch.ones(T, T, dtype=torch.bool))
    out = torch.zeros(T, H, v.shape[2], dtype=F)
    for a in range(H):
        g = a // (H // G)
        s = (q[:, a] @ k[:, g].T) * scale
        s = torch.where(see, s, torch.full_like(s, -math.inf))
        if sink is not None:
            s = torch.cat([s, sink[a].to(F).expand(T, 1)], dim=1)
        out[:, a] = torch.softmax(s, -1)[:, :T] @ v[:, g]
    return out.reshape(T, -1)


def attention(h, m: dict, w: Dict[str, torch.Tensor], p: str):
    """Grouped heads, biases on every projection, split halves rotated."""
    T = h.shape[0]
    H, G = m["heads"], m["kv_heads"]
    q = lin(h, w, p + "q", True).view(T, H, m["dim"])
    k = lin(h, w, p + "k", True).view(T, G, m["dim"])
    v = lin(h, w, p + "v", True).view(T, G, m["vdim"])
    if m.get("rot") is not None:
        q = rotate(q, torch.arange(T), m["rot"], False)
        k = rotate(k, torch.arange(T), m["rot"], False)
    return lin(attend(q, k, v, m["scale"]), w, p + "o", True)


def latent_attention(h, m: dict, w: Dict[str, torch.Tensor], p: str, eps: float):
    """Keys and values rebuilt from a normed latent, one rotated key part (neighbouring pairs)
    for all heads, a sink per head."""
    T = h.shape[0]
    H, d, r, dv, R = m["heads"], m["dim"], m["rot_dim"], m["vdim"], m["kv_rank"]
    q = lin(h, w, p + "q").view(T, H, d + r)
    row = lin(h, w, p + "dkv")
    c = rms(row[:, :R], eps) * w[p + "dkv.norm"].to(F)
    kr = rotate(row[:, R:].view(T, 1, r), torch.arange(T), m["rot"], True)
    q = torch.cat([q[..., :d], rotate(q[..., d:], torch.arange(T), m["rot"], True)], dim=-1)
    k = torch.cat([lin(c, w, p + "uk").view(T, H, d), kr.expand(T, H, r)], dim=-1)
    v = lin(c, w, p + "uv").view(T, H, dv)
    return lin(attend(q, k, v, m["scale"], w[p + "sink"]), w, p + "o")


# ------------------------------------------------------------------ the delta rule
def causal_conv(u, weight):
    """u [T, C], weight [C, taps]: y_t = sum_j weight[:, j] * u_(t - taps + 1 + j), zeros
    before the sequence's first token."""
    T = u.shape[0]
    taps = weight.shape[1]
    y = torch.zeros_like(u)
    for j in range(taps):
        back = taps - 1 - j
        if back < T:
            y[back:] += weight[:, j] * u[:T - back]
    return y


def unit(x):
    return x / torch.sqrt((x * x).sum(-1, keepdim=True) + 1e-6)


def head_decay(pre, dt_bias, a_log):
    """pre [T, H] -> exp(-exp(a_log) * softplus(pre + dt_bias)), one per head and token."""
    return torch.exp(-torch.exp(a_log.to(F)) * softplus(pre + dt_bias.to(F)))


def delta_recurrence(q, k, v, beta, g):
    """q, k [T, G, d], v [T, H, dv], beta, g [T, H] -> [T, H, dv], token by token."""
    T, H, dv = v.shape
    G, d = k.shape[1:]
    o = torch.zeros(T, H, dv, dtype=F)
    for a in range(H):
        kv = a // (H // G)
        S = torch.zeros(d, dv, dtype=F)
        for t in range(T):
            S = g[t, a] * S
            u = beta[t, a] * (v[t, a] - S.T @ k[t, kv])
            S = S + torch.outer(k[t, kv], u)
            o[t, a] = S.T @ q[t, kv]
    return o


def delta(h, m: dict, w: Dict[str, torch.Tensor], p: str, eps: float):
    T = h.shape[0]
    H, G, d, dv = m["heads"], m["kv_heads"], m["dim"], m["vdim"]
    x = {n: silu(causal_conv(lin(h, w, p + n), w[f"{p}{n}.conv"].to(F))) for n in ("q", "k", "v")}
    q = unit(x["q"].view(T, G, d)) * d ** -0.5
    k = unit(x["k"].view(T, G, d))
    o = delta_recurrence(q, k, x["v"].view(T, H, dv), torch.sigmoid(lin(h, w, p + "b")),
                         head_decay(lin(h, w, p + "a"), w[p + "dt_bias"], w[p + "A_log"]))
    o = rms(o, eps) * w[p + "norm"].to(F) * silu(lin(h, w, p + "g")).view(T, H, dv)
    return lin(o.reshape(T, -1), w, p + "o")


# ------------------------------------------------------------------ feed-forward
def clamped_expert(h, w, p: str, limit: float):
    g = lin(h, w, p + "gate").clamp(max=limit)
    u = lin(h, w, p + "up").clamp(min=-limit, max=limit)
    return lin(g * torch.sigmoid(1.702 * g) * (u + 1.0), w, p + "down")


def route(h, w, p: str, top: int):
    """(ids [T, top], weights [T, top]): sigmoid scores choose and weigh as they are."""
    s = torch.sigmoid(lin(h, w, p + "router"))
    val, ids = torch.topk(s, top, dim=-1)
    return ids, val


def experts(h, f: dict, w, p: str, ids=None):
    """``ids`` [T, top]: take these experts (and their own scores) instead of choosing."""
    top = f["router"]["top"]
    chosen, wts = route(h, w, p, top)
    if ids is not None:
        chosen = ids
        wts = torch.sigmoid(lin(h, w, p + "router")).gather(1, ids)
    out = torch.zeros_like(h)
    for t in range(h.shape[0]):
        for c in range(top):
            e = int(chosen[t, c])
            out[t] += clamped_expert(wts[t, c] * h[t:t + 1], w, f"{p}e{e}.",
                                     f["expert"]["limit"])[0]
    if f.get("shared") is not None:
        out = out + clamped_expert(h, w, p + "shared.", f["shared"]["limit"])
    return out


# ------------------------------------------------------------------ the model
def mixer(kind: str, h, m: dict, w, p: str, eps: float):
    if kind == "attention":
        return attention(h, m, w, p)
    if kind == "latent_attention":
        return latent_attention(h, m, w, p, eps)
    assert kind == "delta", kind
    return delta(h, m, w, p, eps)


def run_order(cfg: dict) -> List[tuple]:
    """(layer, whether the embedding output is added right before it) in the order they run."""
    n = len(cfg["layers"])
    lp = cfg.get("loop")
    if lp is None:
        return [(i, False) for i in range(n)]
    out = [(i, False) for i in range(lp["start"])]
    for t in range(lp["times"]):
        for i in range(lp["start"], lp["stop"]):
            out.append((i, t > 0 and i == lp["start"]))
    return out + [(i, False) for i in range(lp["stop"], n)]


def forward(cfg: dict, w: Dict[str, torch.Tensor], tokens, layers_out: Optional[list] = None,
            choices: Optional[list] = None):
    """Logits [T, vocab] of one sequence from position 0.  ``layers_out``: a list that receives
    the stream after every layer run.  ``choices``: the experts every run of a layer with
    experts takes ([T, top] each, in run order), instead of its own choice."""
    tokens = torch.as_tensor(tokens, dtype=torch.long)
    eps = cfg["norm"]["eps"]
    x = start = w["embed"].to(F)[tokens]
    given = iter(choices) if choices is not None else None
    for i, again in run_order(cfg):
        layer, p = cfg["layers"][i], f"l{i}."
        if again:
            x = x + start
        h = norm_around_zero(x, w[p + "norm1"], eps)
        y = mixer(layer["type"], h, layer["mixer"], w, p + "mix.", eps)
        if layer.get("mlp") is not None:
            y = y + experts(h, layer["mlp"], w, p + "mlp.",
                            next(given) if given is not None else None)
        x = x + y
        if layers_out is not None:
            layers_out.append(x.clone())
    return norm_around_zero(x, w["final.norm"], eps) @ w["head"].to(F).T
