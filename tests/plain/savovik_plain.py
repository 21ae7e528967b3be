"""Savovik, written out plainly: one function per mechanism, 64-bit, token by token where the
design is a recurrence.  Nothing here is shared with the library; the tests compare the two.

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


def gelu_erf(z):
    return 0.5 * z * (1.0 + torch.erf(z / math.sqrt(2.0)))


def rms(x, eps):
    """x over the root of its mean square, eps under the root, along the last axis."""
    return x / torch.sqrt((x * x).mean(-1, keepdim=True) + eps)


def lin(x, w, name):
    """W x, plus the bias stored under the name with '.b' where there is one."""
    y = x @ w[name].to(F).T
    if name + ".b" in w:
        y = y + w[name + ".b"].to(F)
    return y


# ------------------------------------------------------------------ positions
def frequencies(rot: dict) -> List[float]:
    """A scaling with a factor alone divides every frequency; one with bounds keeps short
    wavelengths, divides long ones and blends between."""
    sc = rot.get("scaling")
    out = []
    for i in range(rot["dims"] // 2):
        f = rot["base"] ** (-2.0 * i / rot["dims"])
        if sc is not None and "original" not in sc:
            f = f / sc["factor"]
        elif sc is not None:
            wavelength = 2.0 * math.pi / f
            if wavelength > sc["original"] / sc["low"]:
                f = f / sc["factor"]
            elif not wavelength < sc["original"] / sc["high"]:
                s = (sc["original"] / wavelength - sc["low"]) / (sc["high"] - sc["low"])
                f = (1.0 - s) * f / sc["factor"] + s * f
        out.append(f)
    return out


def rotate(x, positions, rot: dict, neighbours: bool):
    """x [T, heads, dim]: pairs (2i, 2i + 1) or (i, i + dims / 2) of the first rot.dims
    dimensions of every head turn by position * f_i."""
    dims = rot["dims"]
    f = torch.tensor(frequencies(rot), dtype=F)
    a = positions.to(F)[:, None] * f[None, :]
    c, s = torch.cos(a)[:, None, :], torch.sin(a)[:, None, :]
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


# ------------------------------------------------------------------ convolution
def causal_conv(u, weight, bias):
    """u [T, C], weight [C, taps]: y_t = bias + sum_j weight[:, j] * u_(t - taps + 1 + j), zeros
    before the sequence's first token."""
    T, C = u.shape
    taps = weight.shape[1]
    y = bias[None, :].repeat(T, 1)
    for j in range(taps):
        back = taps - 1 - j
        if back < T:
            y[back:] += weight[:, j] * u[:T - back]
    return y


# ------------------------------------------------------------------ attention
def in_chunk(i: int, j: int, size: int) -> bool:
    return j <= i and i // size == j // size


def in_window(i: int, j: int, size: int) -> bool:
    return 0 <= i - j < size


def attend(q, k, v, scale: float, see, softcap: Optional[float]):
    """q [T, H, dim], k [T, G, dim], v [T, G, vdim], see [T, T] -> [T, H * vdim]."""
    T, H, _ = q.shape
    G = k.shape[1]
    out = torch.zeros(T, H, v.shape[2], dtype=F)
    for a in range(H):
        g = a // (H // G)
        s = (q[:, a] @ k[:, g].T) * scale
        if softcap is not None:
            s = softcap * torch.tanh(s / softcap)
        s = torch.where(see, s, torch.full_like(s, -math.inf))
        out[:, a] = torch.softmax(s, -1) @ v[:, g]
    return out.reshape(T, -1)


def _heads(h, m: dict, w, p: str):
    T = h.shape[0]
    H, G = m["heads"], m.get("kv_heads", m["heads"])
    return (lin(h, w, p + "q").view(T, H, m["dim"]), lin(h, w, p + "k").view(T, G, m["dim"]),
            lin(h, w, p + "v").view(T, G, m["vdim"]))


def mask(T: int, fn, m: dict):
    if m.get("mask") is None:
        return torch.tril(torch.ones(T, T, dtype=torch.bool))
    size = m["mask"]["size"]
    i, j = torch.arange(T)[:, None], torch.arange(T)[None, :]
    if fn is in_chunk:
        return (j <= i) & (i // size == j // size)
    return (i - j >= 0) & (i - j < size)


def chunked_attention(h, m: dict, w: Dict[str, torch.Tensor], p: str, eps: float):
    """Biases on q, k and v, a per-head norm of q and k, neighbouring pairs rotated, a mask of
    chunks counted from position 0."""
    T = h.shape[0]
    q, k, v = _heads(h, m, w, p)
    q = rms(q, eps) * w[p + "q.norm"].to(F)
    k = rms(k, eps) * w[p + "k.norm"].to(F)
    if m.get("rot") is not None:
        q = rotate(q, torch.arange(T), m["rot"], True)
        k = rotate(k, torch.arange(T), m["rot"], True)
    return lin(attend(q, k, v, m["scale"], mask(T, in_chunk, m), None), w, p + "o")


def window_attention(h, m: dict, w: Dict[str, torch.Tensor], p: str, eps: float):
    """Split halves rotated, every value over its root mean square, capped scores, a sliding
    window."""
    T = h.shape[0]
    q, k, v = _heads(h, m, w, p)
    if m.get("rot") is not None:
        q = rotate(q, torch.arange(T), m["rot"], False)
        k = rotate(k, torch.arange(T), m["rot"], False)
    v = rms(v, eps)
    return lin(attend(q, k, v, m["scale"], mask(T, in_window, m), m.get("softcap")), w, p + "o")


# ------------------------------------------------------------------ state-space mixers
def selective_scan(x, dt, A, B, C, D):
    """x, dt [T, inner], A [inner, N], B, C [T, N], D [inner]: the state of every channel token
    by token, and what is read from it."""
    S = torch.zeros_like(A)
    y = torch.zeros_like(x)
    for t in range(x.shape[0]):
        S = torch.exp(dt[t][:, None] * A) * S + (dt[t] * x[t])[:, None] * B[t][None, :]
        y[t] = (S * C[t][None, :]).sum(-1) + D * x[t]
    return y


def mamba(h, m: dict, w: Dict[str, torch.Tensor], p: str):
    inner, N, r = m["inner"], m["state"], m["dt_rank"]
    xz = lin(h, w, p + "in")
    x, z = xz[:, :inner], xz[:, inner:]
    x = silu(causal_conv(x, w[p + "conv"].to(F), w[p + "conv.b"].to(F)))
    dbc = lin(x, w, p + "x")
    dt = softplus(lin(dbc[:, :r], w, p + "dt"))
    y = selective_scan(x, dt, -torch.exp(w[p + "A_log"].to(F)), dbc[:, r:r + N], dbc[:, r + N:],
                       w[p + "D"].to(F))
    return lin(y * silu(z), w, p + "o")


def ssd(x, dt, a, B, C, D):
    """x [T, H, dv], dt [T, H], a [H] (positive), B, C [T, G, N], D [H]."""
    T, H, dv = x.shape
    G = B.shape[1]
    y = torch.zeros_like(x)
    for i in range(H):
        g = i // (H // G)
        S = torch.zeros(B.shape[2], dv, dtype=F)
        for t in range(T):
            S = torch.exp(-a[i] * dt[t, i]) * S + dt[t, i] * torch.outer(B[t, g], x[t, i])
            y[t, i] = S.T @ C[t, g] + D[i] * x[t, i]
    return y


def mamba2(h, m: dict, w: Dict[str, torch.Tensor], p: str, eps: float):
    T = h.shape[0]
    H, dv, N, G = m["heads"], m["vdim"], m["state"], m["groups"]
    inner = H * dv
    zxbcdt = lin(h, w, p + "in")
    z, xbc, dt = zxbcdt.split([inner, inner + 2 * G * N, H], dim=1)
    xbc = silu(causal_conv(xbc, w[p + "conv"].to(F), w[p + "conv.b"].to(F)))
    x, B, C = xbc.split([inner, G * N, G * N], dim=1)
    dt = softplus(dt + w[p + "dt_bias"].to(F))
    y = ssd(x.view(T, H, dv), dt, torch.exp(w[p + "A_log"].to(F)), B.view(T, G, N),
            C.view(T, G, N), w[p + "D"].to(F)).reshape(T, inner)
    y = y * silu(z)
    y = rms(y.view(T, m["norm_groups"], -1), eps).reshape(T, inner) * w[p + "norm"].to(F)
    return lin(y, w, p + "o")


# ------------------------------------------------------------------ the model
def mixer(kind: str, h, m: dict, w, p: str, eps: float):
    if kind == "parallel":
        return (m["left_scale"] * chunked_attention(h, m["left"], w, p + "left.", eps) +
                m["right_scale"] * mamba(h, m["right"], w, p + "right."))
    if kind == "mamba2":
        return mamba2(h, m, w, p, eps)
    assert kind == "attention", kind
    return window_attention(h, m, w, p, eps)


def feed_forward(h, w, p: str):
    return lin(gelu_erf(lin(h, w, p + "up")), w, p + "down")


def forward(cfg: dict, w: Dict[str, torch.Tensor], tokens, layers_out=None):
    """Logits [T, vocab] of one sequence from position 0.  ``layers_out``: a list that receives
    the stream after every layer."""
    tokens = torch.as_tensor(tokens, dtype=torch.long)
    eps = cfg["norm"]["eps"]
    x = w["embed"].to(F)[tokens]
    for i, layer in enumerate(cfg["layers"]):
        while layer.get("weights_of") is not None:
            i = layer["weights_of"]
            layer = cfg["layers"][i]
        p = f"l{i}."
        h = rms(x, eps) * (1.0 + w[p + "norm1"].to(F))
        y = mixer(layer["type"], h, layer["mixer"], w, p + "mix.", eps) * \
            torch.sigmoid(lin(h, w, p + "rg1"))
        if layer.get("mlp") is not None:
            y = y + feed_forward(h, w, p + "mlp.") * torch.sigmoid(lin(h, w, p + "rg2"))
        x = x + y
        if layers_out is not None:
            layers_out.append(x.clone())
    return (rms(x, eps) * (1.0 + w["final.norm"].to(F))) @ w["head"].to(F).T
