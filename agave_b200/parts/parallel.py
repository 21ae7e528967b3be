"""Parts that stand side by side: two mixers on one input, and a block whose mixer and
feed-forward read one norm.

"side_by_side" (a mixer): left_scale * left(x) + right_scale * right(x).  Each of the two is any
mixer of the registry; together they use one cache entry, so at most one of them may keep keys
and values and at most one a fixed-size state.

"parallel" (a block): with x = norm(h),

    h += sigmoid(W_m x + b_m) * mixer(x) + sigmoid(W_f x + b_f) * ffn(x)

element by element, or without the gates.  The two gates' projections are one stacked product;
the gates, the branches' sums over ranges of K, the scales of mixers side by side, the bias of a
mixer's output product, what the run order adds to the stream after the block, the residual sum
and the norm that feeds the next block are one launch.
"""
from __future__ import annotations

from typing import Dict, List, Optional, Tuple

import torch

from .. import kernels
from ..config.base import ParallelBlockSpec, SideBySideSpec
from .base import (KVRequest, ParamSpec, StateRequest, feed_forward_class, mixer_class, norm_class,
                   register_block, register_mixer)
from .linear import Linear
from .matrix_memory import project_f32
from .norm import RMSNorm


def _under(tensors: Dict[str, torch.Tensor], prefix: str) -> Dict[str, torch.Tensor]:
    n = len(prefix) + 1
    return {k[n:]: v for k, v in tensors.items() if k.startswith(prefix + ".")}


class SideBySideMixer:
    def __init__(self, spec: SideBySideSpec, hidden_size: int, dtype: torch.dtype,
                 device: torch.device):
        self.spec, self.hidden_size, self.dtype, self.device = spec, hidden_size, dtype, device
        self.left = mixer_class(spec.left.kind)(spec.left, hidden_size, dtype, device)
        self.right = mixer_class(spec.right.kind)(spec.right, hidden_size, dtype, device)
        self.cache_request()                   # (two requests that cannot share an entry raise here)

    @classmethod
    def param_specs(cls, spec: SideBySideSpec, hidden_size: int) -> Dict[str, ParamSpec]:
        out: Dict[str, ParamSpec] = {}
        for side in ("left", "right"):
            s = getattr(spec, side)
            for k, v in mixer_class(s.kind).param_specs(s, hidden_size).items():
                out[f"{side}.{k}"] = v
        return out

    def cache_request(self):
        asked: List[object] = []
        for m in (self.left, self.right):
            r = m.cache_request()
            asked += list(r) if isinstance(r, (tuple, list)) else [] if r is None else [r]
        for kind, what in ((KVRequest, "keys and values"), (StateRequest, "a fixed-size state")):
            if sum(isinstance(r, kind) for r in asked) > 1:
                raise ValueError(f"two mixers side by side cannot both keep {what}")
        return tuple(asked) if len(asked) > 1 else asked[0] if asked else None

    def load(self, tensors: Dict[str, torch.Tensor], dtype: torch.dtype,
             device: torch.device) -> None:
        self.left.load(_under(tensors, "left"), dtype, device)
        self.right.load(_under(tensors, "right"), dtype, device)

    def forward_terms(self, x: torch.Tensor, ctx, cache_entry: int,
                      writes_cache: bool) -> List[Tuple[torch.Tensor, float]]:
        """The two results and their scales, for a block that joins them itself."""
        return [(self.left.forward(x, ctx, cache_entry, writes_cache), float(self.spec.left_scale)),
                (self.right.forward(x, ctx, cache_entry, writes_cache),
                 float(self.spec.right_scale))]

    def forward(self, x: torch.Tensor, ctx, cache_entry: int, writes_cache: bool) -> torch.Tensor:
        y = ctx.new(x.shape[0], self.hidden_size, dtype=torch.float32)
        kernels.gated_join(None, [(t, m, -1) for t, m in
                                  self.forward_terms(x, ctx, cache_entry, writes_cache)],
                           None, None, None, None, 0.0, y)
        return y.unsqueeze(0)


register_mixer("side_by_side", SideBySideMixer)


class ParallelBlock:
    def __init__(self, spec: ParallelBlockSpec, hidden_size: int, dtype: torch.dtype,
                 device: torch.device):
        self.spec, self.hidden_size, self.dtype, self.device = spec, hidden_size, dtype, device
        self.norm = norm_class(spec.norm.kind)(spec.norm, hidden_size, dtype, device)
        self.mixer = mixer_class(spec.mixer.kind)(spec.mixer, hidden_size, dtype, device)
        self.ffn = None
        if spec.feed_forward is not None:
            self.ffn = feed_forward_class(spec.feed_forward.kind)(spec.feed_forward, hidden_size,
                                                                  dtype, device)
        self.gated = bool(spec.gated)
        self.gates: Optional[Linear] = None
        self.gate_bias: Optional[torch.Tensor] = None

    @classmethod
    def param_specs(cls, spec: ParallelBlockSpec, hidden_size: int) -> Dict[str, ParamSpec]:
        out: Dict[str, ParamSpec] = {}
        for k, v in norm_class(spec.norm.kind).param_specs(spec.norm, hidden_size).items():
            out[f"norm.{k}"] = v
        for k, v in mixer_class(spec.mixer.kind).param_specs(spec.mixer, hidden_size).items():
            out[f"mixer.{k}"] = v
        ff = spec.feed_forward
        if ff is not None:
            for k, v in feed_forward_class(ff.kind).param_specs(ff, hidden_size).items():
                out[f"ffn.{k}"] = v
        if spec.gated:
            for name in ("mixer_gate", "ffn_gate")[:1 if ff is None else 2]:
                out[f"{name}.weight"] = ParamSpec((hidden_size, hidden_size))
                out[f"{name}.bias"] = ParamSpec((hidden_size,), "float32")
        return out

    # the block adds ``ctx.join_extra`` (a 32-bit [T, H] or None) to the stream in its own join
    joins_extra = True

    @property
    def entry_norm(self):
        return self.norm

    def cache_request(self):
        return self.mixer.cache_request()

    def state_request(self):
        ask = getattr(self.mixer, "state_request", None)
        return ask() if ask is not None else None

    def load(self, tensors: Dict[str, torch.Tensor], dtype: torch.dtype,
             device: torch.device) -> None:
        self.norm.load(_under(tensors, "norm"), device)
        self.mixer.load(_under(tensors, "mixer"), dtype, device)
        if self.ffn is not None:
            self.ffn.load(_under(tensors, "ffn"), dtype, device)
        if self.gated:
            names = ("mixer_gate", "ffn_gate")[:1 if self.ffn is None else 2]
            self.gates = Linear(torch.cat([tensors[f"{n}.weight"].to(device=device, dtype=dtype)
                                           for n in names], dim=0).contiguous(), role="gates")
            self.gate_bias = torch.cat([tensors[f"{n}.bias"].to(device=device, dtype=torch.float32)
                                        for n in names]).contiguous()

    def forward(self, h: torch.Tensor, x: torch.Tensor, ctx, cache_entry: int,
                writes_cache: bool, next_norm) -> Optional[torch.Tensor]:
        """h: [T, H] 32-bit stream (updated in place); x = norm(h)."""
        many = getattr(self.mixer, "forward_terms", None)
        if many is not None:
            branches = many(x, ctx, cache_entry, writes_cache)
        else:
            branches = [(self.mixer.forward(x, ctx, cache_entry, writes_cache), 1.0)]
        terms = [(y, m, 0 if self.gated else -1) for y, m in branches]
        if self.ffn is not None:
            terms.append((self.ffn.forward(x, ctx), 1.0, 1 if self.gated else -1))
        extra = getattr(ctx, "join_extra", None)
        if extra is not None:
            terms.append((extra, 1.0, -1))
        row = part = None
        if self.gated:
            row, part = project_f32(self.gates, x)
        fused = type(next_norm) is RMSNorm
        x_next = ctx.new(*x.shape) if next_norm is not None else None
        kernels.gated_join(h, terms, row, part, self.gate_bias,
                           next_norm.weight if fused else None, next_norm.eps if fused else 0.0,
                           x_next if fused else None)
        if next_norm is not None and not fused:
            next_norm.forward(h, x_next)
        return x_next


register_block("parallel", ParallelBlock)
