"""Savovik: the registry entry and the names of its tensors.

The layer structure is data (``SavovikConfig.to_model_spec``): attention over chunks of
positions beside a selective scan, a scan with one decay per head, or windowed attention with
capped scores and normed values; a dense erf-GELU feed-forward; both branches from one norm,
each joining the stream through a gate; layers that run another layer's weights.  What is left
to say here is how the generic decoder's tensor names map to a checkpoint's: ``embed``,
``head``, ``final.norm`` and per layer with tensors of its own ``l<i>.norm1``, ``l<i>.rg1`` and
``rg2``, ``l<i>.mix.*`` (``l<i>.mix.left.*`` and ``.right.*`` for the two mixers side by side)
and ``l<i>.mlp.{up,down}``; a bias is its tensor's name with ``.b``.
"""
from __future__ import annotations

from dataclasses import dataclass
from typing import Tuple

from ..config.registry import register_architecture
from ..config.savovik import SavovikConfig
from ..parts import parallel as _parallel            # registers the block and the mixer
from ..parts import state_space as _state_space      # registers the mixers

_BLOCK = {"norm.weight": "norm1", "mixer_gate.weight": "rg1", "mixer_gate.bias": "rg1.b",
          "ffn_gate.weight": "rg2", "ffn_gate.bias": "rg2.b"}
_MIXER = {
    # attention
    "q_proj.weight": "q", "k_proj.weight": "k", "v_proj.weight": "v", "o_proj.weight": "o",
    "q_proj.bias": "q.b", "k_proj.bias": "k.b", "v_proj.bias": "v.b",
    "q_norm.weight": "q.norm", "k_norm.weight": "k.norm",
    # the scans
    "in_proj.weight": "in", "conv.weight": "conv", "conv.bias": "conv.b", "x_proj.weight": "x",
    "dt_proj.weight": "dt", "dt_proj.bias": "dt.b", "dt_bias": "dt_bias", "a_log": "A_log",
    "d": "D", "out_norm.weight": "norm",
}
_FFN = {"up_proj.weight": "up", "down_proj.weight": "down"}


@dataclass(frozen=True)
class SavovikWeightNames:
    owners: Tuple[int, ...]            # layer number of each block
    prefixes: Tuple[str, ...] = ("",)
    ignore_prefixes: Tuple[str, ...] = ()

    def checkpoint_name(self, internal: str, prefix: str) -> str:
        if internal == "embed.weight":
            return prefix + "embed"
        if internal == "lm_head.weight":
            return prefix + "head"
        if internal == "final_norm.weight":
            return prefix + "final.norm"
        parts = internal.split(".", 2)
        if parts[0] == "blocks" and len(parts) == 3 and int(parts[1]) < len(self.owners):
            layer, rest = f"{prefix}l{self.owners[int(parts[1])]}.", parts[2]
            if rest in _BLOCK:
                return layer + _BLOCK[rest]
            head, _, leaf = rest.partition(".")
            if head == "mixer":
                side, _, inner = leaf.partition(".")
                if side in ("left", "right") and inner in _MIXER:
                    return f"{layer}mix.{side}.{_MIXER[inner]}"
                if leaf in _MIXER:
                    return f"{layer}mix.{_MIXER[leaf]}"
            if head == "ffn" and leaf in _FFN:
                return f"{layer}mlp.{_FFN[leaf]}"
        raise KeyError(f"Savovik has no checkpoint name for '{internal}'")


def _weight_names(config: SavovikConfig) -> SavovikWeightNames:
    return SavovikWeightNames(owners=config.owners())


register_architecture("Savovik", SavovikConfig, _weight_names, model_types=("savovik",))
