"""Two state-space mixers: the selective scan of Mamba and the head-wise form of Mamba-2.

Both begin with one input product, a causal convolution over time with a bias on some of its
columns (the last taps - 1 inputs of a sequence are part of its state, a ring by position) and
silu, and end with a gate silu(z) from the same input product and an output product.

"selective_scan": W_in x = [u | z]; after convolution and silu, W_x u = [r | B | C] and dt =
softplus(W_dt r + b) per channel; per channel c and state n, with A = -exp(A_log):

    S[c, n] <- exp(dt_c A[c, n]) S[c, n] + dt_c u_c B_n;      y_c = sum_n S[c, n] C_n + D_c u_c

Flow of a step: input product; convolution kernel (u in 32-bit for the scan and rounded for its
product); the product W_x; a row kernel (r rounded for its product, B and C padded); the product
W_dt; the scan, which takes the softplus of the step sizes and finishes y * silu(z); the output
product.

"state_space": W_in x = [z | u | B | C | dt]; u, B and C pass the convolution; dt = softplus(dt +
bias) per head; with B and C of the head's group

    S <- exp(-exp(A_log_h) dt) S + dt B u^T;      y = S^T C + D_h u

then (y * silu(z)) / rms in equal parts of the row, times a weight.  Flow: input product;
convolution kernel (which also makes the pair (decay, dt) of every head); the scan, which is the
matrix memory's without its normaliser; the read-out kernel; the output product.

A prompt and a decoded token run the same kernels.  The state of a sequence (S, then the ring of
the convolution's inputs) lives in 32-bit in its slot of the cache's fixed-size state, zero when
the slot is taken, read at the start of a step and written at its end.
"""
from __future__ import annotations

import math
from typing import Dict, Optional

import torch

from .. import kernels
from ..config.base import SelectiveScanSpec, StateSpaceSpec
from .base import ParamSpec, StateRequest, register_mixer
from .linear import Linear
from .matrix_memory import project_f32

MAX_TAPS = 8


def _loaders(tensors, dtype, device):
    def mat(name):
        return tensors[name].to(device=device, dtype=dtype).contiguous()

    def f32(name):
        return tensors[name].to(device=device, dtype=torch.float32).contiguous()
    return mat, f32


class SelectiveScanMixer:
    def __init__(self, spec: SelectiveScanSpec, hidden_size: int, dtype: torch.dtype,
                 device: torch.device):
        s = spec
        if min(s.inner, s.state, s.dt_rank, s.conv_taps) < 1:
            raise ValueError("the sizes of a selective scan must be positive")
        if s.state > kernels.SELECTIVE_MAX_STATE or s.conv_taps > MAX_TAPS:
            raise ValueError(f"a selective scan holds at most {kernels.SELECTIVE_MAX_STATE} states "
                             f"a channel and {MAX_TAPS} taps")
        self.spec, self.hidden_size, self.dtype, self.device = spec, hidden_size, dtype, device
        self.conv_off = s.inner * s.state                      # behind S
        self.in_proj: Optional[Linear] = None
        self.x_proj: Optional[Linear] = None
        self.dt_proj: Optional[Linear] = None
        self.out: Optional[Linear] = None
        self.conv_w = self.conv_b = self.dt_bias = self.a2 = self.d = None

    @classmethod
    def param_specs(cls, spec: SelectiveScanSpec, hidden_size: int) -> Dict[str, ParamSpec]:
        s = spec
        return {
            "in_proj.weight": ParamSpec((2 * s.inner, hidden_size)),
            "conv.weight": ParamSpec((s.inner, s.conv_taps), "float32"),
            "conv.bias": ParamSpec((s.inner,), "float32"),
            "x_proj.weight": ParamSpec((s.dt_rank + 2 * s.state, s.inner)),
            "dt_proj.weight": ParamSpec((s.inner, s.dt_rank)),
            "dt_proj.bias": ParamSpec((s.inner,), "float32"),
            "a_log": ParamSpec((s.inner, s.state), "float32"),
            "d": ParamSpec((s.inner,), "float32"),
            "o_proj.weight": ParamSpec((hidden_size, s.inner)),
        }

    def cache_request(self):
        s = self.spec
        return StateRequest(s.inner * s.state + (s.conv_taps - 1) * s.inner)

    def load(self, tensors: Dict[str, torch.Tensor], dtype: torch.dtype,
             device: torch.device) -> None:
        mat, f32 = _loaders(tensors, dtype, device)
        self.in_proj = Linear(mat("in_proj.weight"), role="qkv")
        self.x_proj = Linear(mat("x_proj.weight"), role="x_proj")
        self.dt_proj = Linear(mat("dt_proj.weight"), role="dt_proj")
        self.out = Linear(mat("o_proj.weight"), role="out_proj")
        self.conv_w, self.conv_b = f32("conv.weight"), f32("conv.bias")
        self.dt_bias, self.d = f32("dt_proj.bias"), f32("d")
        # A = -exp(A_log) on the base-2 scale of the kernel's exponential, formed in 64-bit
        a = -torch.exp(tensors["a_log"].to(torch.float64)) / math.log(2.0)
        self.a2 = a.to(device=device, dtype=torch.float32).contiguous()

    def forward(self, x: torch.Tensor, ctx, cache_entry: int, writes_cache: bool) -> torch.Tensor:
        if not writes_cache:
            raise ValueError("a recurrent mixer owns the state of its cache entry")
        s = self.spec
        T, f32 = x.shape[0], torch.float32
        state = ctx.cache.state_view(cache_entry).state
        row, part = project_f32(self.in_proj, x)
        u = ctx.new(T, s.inner, dtype=f32)
        rounded = u if self.dtype == f32 else ctx.new(T, s.inner)
        kernels.ssm_conv(row, part, T, 2 * s.inner, 0, s.conv_taps, self.conv_w, self.conv_b, u,
                         None if rounded is u else rounded, state, self.conv_off, ctx)
        proj = self.x_proj.partial(rounded)
        split = proj.dim() == 3
        low = ctx.new(T, s.dt_rank)
        bc = ctx.new(T, 2 * kernels.selective_pad(s.state), dtype=f32)
        kernels.selective_low(None if split else proj, proj if split else None, s.dt_rank, s.state,
                              low, bc)
        dt = self.dt_proj(low, out=ctx.new(T, s.inner, dtype=f32))
        y = ctx.new(T, s.inner)
        kernels.selective_scan(u, dt, self.dt_bias, bc, self.a2, self.d, row, part, 2 * s.inner,
                               s.inner, y, ctx, state, 0)
        return self.out.partial(y)


register_mixer("selective_scan", SelectiveScanMixer)


class StateSpaceMixer:
    def __init__(self, spec: StateSpaceSpec, hidden_size: int, dtype: torch.dtype,
                 device: torch.device):
        s = spec
        if min(s.n_heads, s.value_dim, s.state, s.n_groups, s.norm_groups, s.conv_taps) < 1:
            raise ValueError("the sizes of a state-space mixer must be positive")
        if s.n_heads % s.n_groups or (s.n_heads * s.value_dim) % s.norm_groups:
            raise ValueError("a state-space mixer's groups must divide its heads, and the parts of "
                             "its norm its width")
        if s.state > 256 or s.conv_taps > MAX_TAPS:
            raise ValueError(f"a state-space mixer's state is at most 256 wide, with {MAX_TAPS} taps")
        self.spec, self.hidden_size, self.dtype, self.device = spec, hidden_size, dtype, device
        self.inner = s.n_heads * s.value_dim
        self.channels = self.inner + 2 * s.n_groups * s.state   # what the convolution runs over
        self.width = self.inner + self.channels + s.n_heads
        self.conv_off = s.n_heads * s.state * s.value_dim        # behind S
        self.in_proj: Optional[Linear] = None
        self.out: Optional[Linear] = None
        self.conv_w = self.conv_b = self.dt_bias = self.neg_a = self.d = self.out_norm = None

    @classmethod
    def param_specs(cls, spec: StateSpaceSpec, hidden_size: int) -> Dict[str, ParamSpec]:
        s = spec
        inner = s.n_heads * s.value_dim
        channels = inner + 2 * s.n_groups * s.state
        return {
            "in_proj.weight": ParamSpec((inner + channels + s.n_heads, hidden_size)),
            "conv.weight": ParamSpec((channels, s.conv_taps), "float32"),
            "conv.bias": ParamSpec((channels,), "float32"),
            "dt_bias": ParamSpec((s.n_heads,), "float32"),
            "a_log": ParamSpec((s.n_heads,), "float32"),
            "d": ParamSpec((s.n_heads,), "float32"),
            "out_norm.weight": ParamSpec((inner,), "norm"),
            "o_proj.weight": ParamSpec((hidden_size, inner)),
        }

    def cache_request(self):
        return StateRequest(self.conv_off + (self.spec.conv_taps - 1) * self.channels)

    def load(self, tensors: Dict[str, torch.Tensor], dtype: torch.dtype,
             device: torch.device) -> None:
        mat, f32 = _loaders(tensors, dtype, device)
        self.in_proj = Linear(mat("in_proj.weight"), role="qkv")
        self.out = Linear(mat("o_proj.weight"), role="out_proj")
        self.conv_w, self.conv_b = f32("conv.weight"), f32("conv.bias")
        self.dt_bias, self.d, self.out_norm = f32("dt_bias"), f32("d"), f32("out_norm.weight")
        self.neg_a = (-torch.exp(tensors["a_log"].to(torch.float64))).to(
            device=device, dtype=torch.float32).contiguous()

    def forward(self, x: torch.Tensor, ctx, cache_entry: int, writes_cache: bool) -> torch.Tensor:
        if not writes_cache:
            raise ValueError("a recurrent mixer owns the state of its cache entry")
        s = self.spec
        T, f32 = x.shape[0], torch.float32
        H, dv, N, G = s.n_heads, s.value_dim, s.state, s.n_groups
        inner = self.inner
        state = ctx.cache.state_view(cache_entry).state
        row, part = project_f32(self.in_proj, x)
        ubc = ctx.new(T, self.channels, dtype=f32)
        coef = ctx.new(T, H, 2, dtype=f32)
        kernels.ssm_conv(row, part, T, self.width, inner, s.conv_taps, self.conv_w, self.conv_b,
                         ubc, None, state, self.conv_off, ctx, dt_offset=inner + self.channels,
                         dt_bias=self.dt_bias, neg_a=self.neg_a, coef=coef)
        u, b, c = ubc[:, :inner], ubc[:, inner:inner + G * N], ubc[:, inner + G * N:]
        num = ctx.new(T, inner, dtype=f32)
        kernels.head_scan(c, b, u, coef, num, ctx, state, 0, H, G, N, dv)
        y = ctx.new(T, inner)
        kernels.ssd_out(num, u, self.d, row, part, self.width, 0, self.out_norm, float(s.eps),
                        s.norm_groups, dv, y)
        return self.out.partial(y)


register_mixer("state_space", StateSpaceMixer)
