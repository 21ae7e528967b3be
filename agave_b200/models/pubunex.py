"""Pubunex: the registry entry and the names of its tensors.

The layer structure is data (``PubunexConfig.to_model_spec``): the gated delta rule with one
decay per head, attention with biases, latent attention with a sink per head; routed experts
whose weight multiplies their input beside a shared one; both branches from one norm; layers
that run several times in a row with the embedding added before each further pass.  What is left
to say here is how the generic decoder's tensor names map to a checkpoint's: ``embed``, ``head``,
``final.norm`` and per layer ``l<i>.norm1``, ``l<i>.mix.*`` and ``l<i>.mlp.*`` (experts
``e<j>.{gate,up,down}``, ``router``, ``shared.{gate,up,down}``).  The biases of an attention
layer and the convolutions of a delta layer are their projection's name with ``.b`` and
``.conv``; a delta layer's ``b``, ``a`` and ``g`` are projections.
"""
from __future__ import annotations

import re
from dataclasses import dataclass
from typing import Tuple

from ..config.pubunex import PubunexConfig
from ..config.registry import register_architecture
from ..parts import parallel as _parallel            # registers the block

_MIXERS = {
    "delta": {
        "q_proj.weight": "q", "k_proj.weight": "k", "v_proj.weight": "v", "o_proj.weight": "o",
        "q_conv.weight": "q.conv", "k_conv.weight": "k.conv", "v_conv.weight": "v.conv",
        "beta_proj.weight": "b", "decay_proj.weight": "a", "gate_proj.weight": "g",
        "a_log": "A_log", "dt_bias": "dt_bias", "out_norm.weight": "norm",
    },
    "attention": {
        "q_proj.weight": "q", "k_proj.weight": "k", "v_proj.weight": "v", "o_proj.weight": "o",
        "q_proj.bias": "q.b", "k_proj.bias": "k.b", "v_proj.bias": "v.b", "o_proj.bias": "o.b",
    },
    "latent_attention": {
        "q_proj.weight": "q", "kv_down.weight": "dkv", "kv_down_norm.weight": "dkv.norm",
        "k_up.weight": "uk", "v_up.weight": "uv", "sink": "sink", "o_proj.weight": "o",
    },
}
_FFN = {
    "router.weight": "router", "shared.gate_proj.weight": "shared.gate",
    "shared.up_proj.weight": "shared.up", "shared.down_proj.weight": "shared.down",
}
_EXPERT = re.compile(r"^experts\.(\d+)\.(gate|up|down)_proj\.weight$")


@dataclass(frozen=True)
class PubunexWeightNames:
    kinds: Tuple[str, ...]             # the mixer of each layer
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
        if parts[0] == "blocks" and len(parts) == 3 and int(parts[1]) < len(self.kinds):
            layer, rest = f"{prefix}l{int(parts[1])}.", parts[2]
            if rest == "norm.weight":
                return layer + "norm1"
            head, _, leaf = rest.partition(".")
            if head == "mixer" and leaf in _MIXERS[self.kinds[int(parts[1])]]:
                return f"{layer}mix.{_MIXERS[self.kinds[int(parts[1])]][leaf]}"
            if head == "ffn":
                if leaf in _FFN:
                    return f"{layer}mlp.{_FFN[leaf]}"
                e = _EXPERT.match(leaf)
                if e:
                    return f"{layer}mlp.e{e.group(1)}.{e.group(2)}"
        raise KeyError(f"Pubunex has no checkpoint name for '{internal}'")


def _weight_names(config: PubunexConfig) -> PubunexWeightNames:
    return PubunexWeightNames(kinds=tuple(layer.kind for layer in config.layers))


register_architecture("Pubunex", PubunexConfig, _weight_names, model_types=("pubunex",))
