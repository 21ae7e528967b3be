"""Typed configuration of the Pubunex decoder, read from its own ``config.json`` keys.

A Pubunex model is a list of layers.  Each entry names its mixer (``type``: ``delta``,
``attention`` or ``latent_attention``), the mixer's sizes and constants (``mixer``) and its
feed-forward (``mlp``: a mixture of experts with the sizes and the bound of an expert, of the
router and of the shared expert, or null for a layer without).  ``loop`` names the layers that
run several times in a row.  The top level gives the width, the vocabulary and the norms' eps
(``norm.eps``).  Every size and every constant that can differ between two models of the design
is read from there.

What the design fixes, and what therefore stands in the lowering below: mixer and feed-forward
of a layer read one zero-centred RMS norm of the stream side by side and both join it; a pass of
the loop but the first begins with the embedding added to the stream, and every pass has caches
and states of its own; ``delta`` is the gated delta rule with one decay per head, unit q and k
with eps 1e-6, q times dim ** -0.5 and a silu gate; ``attention`` has biases on its four
projections and rotates split halves; ``latent_attention`` rotates neighbouring pairs, takes its
queries straight from the layer's input and has a learned sink per head; an expert bounds its
gate from above and its up projection on both sides, with a sigmoid of 1.702 times the gate;
sigmoid scores choose the experts and multiply their inputs; a shared expert of the same form
runs for every token; the head is a table of its own.
"""
from __future__ import annotations

from dataclasses import dataclass
from typing import Any, Dict, Optional, Tuple

from .base import (AttentionSpec, ClampedGateSpec, ConfigError, HeadDeltaSpec,
                   LatentAttentionSpec, ModelSpec, NormSpec, ParallelBlockSpec, RotarySpec,
                   RoutedFeedForwardSpec, WavelengthScalingSpec, default_schedule,
                   looped_schedule)

MIXERS = ("delta", "attention", "latent_attention")
UNIT_EPS = 1e-6
GATE_ALPHA = 1.702


def _get(d: Any, key: str, where: str, typ=int):
    if not isinstance(d, dict) or key not in d or d[key] is None:
        raise ConfigError(f"config.json: required key '{where}{key}' is missing")
    v = d[key]
    if typ is int:
        if isinstance(v, bool) or not isinstance(v, int):
            if isinstance(v, float) and v.is_integer():
                return int(v)
            raise ConfigError(f"config.json: '{where}{key}' must be an integer, got {v!r}")
        return v
    if typ is float:
        if isinstance(v, bool) or not isinstance(v, (int, float)):
            raise ConfigError(f"config.json: '{where}{key}' must be a number, got {v!r}")
        return float(v)
    return v


def _positive(record: Any, keys, where: str) -> None:
    for k in keys:
        if getattr(record, k) <= 0:
            raise ConfigError(f"config.json: '{where}{k}' must be positive")


@dataclass(frozen=True)
class PubunexScaling:
    factor: float
    original: float
    fast: float
    slow: float


@dataclass(frozen=True)
class PubunexRotation:
    dims: int
    base: float
    scaling: Optional[PubunexScaling] = None


@dataclass(frozen=True)
class PubunexDelta:
    heads: int
    kv_heads: int
    dim: int
    vdim: int
    conv: int


@dataclass(frozen=True)
class PubunexAttention:
    heads: int
    kv_heads: int
    dim: int
    vdim: int
    scale: float
    rot: Optional[PubunexRotation] = None


@dataclass(frozen=True)
class PubunexLatent:
    heads: int
    dim: int
    rot_dim: int
    vdim: int
    kv_rank: int
    scale: float
    rot: PubunexRotation = None


@dataclass(frozen=True)
class PubunexExpert:
    ff: int
    limit: float


@dataclass(frozen=True)
class PubunexExperts:
    experts: int
    top: int
    expert: PubunexExpert
    shared: Optional[PubunexExpert] = None


@dataclass(frozen=True)
class PubunexLayer:
    kind: str
    mixer: object                             # the record of the kind
    mlp: Optional[PubunexExperts]             # None: there is no feed-forward


@dataclass(frozen=True)
class PubunexLoop:
    start: int
    stop: int
    times: int


def _read_rotation(r: Any, where: str) -> Optional[PubunexRotation]:
    if r is None:
        return None
    sc = r.get("scaling")
    if sc is not None:
        sc = PubunexScaling(**{k: _get(sc, k, where + "scaling.", float)
                               for k in ("factor", "original", "fast", "slow")})
    return PubunexRotation(_get(r, "dims", where), _get(r, "base", where, float), sc)


def _read_mixer(kind: str, m: dict, where: str):
    def ints(*keys):
        return {k: _get(m, k, where) for k in keys}

    def kv_heads():
        return _get(m, "kv_heads", where) if m.get("kv_heads") is not None else \
            _get(m, "heads", where)
    if kind == "delta":
        return PubunexDelta(kv_heads=kv_heads(), **ints("heads", "dim", "vdim", "conv"))
    rot = _read_rotation(m.get("rot"), where + "rot.")
    scale = _get(m, "scale", where, float)
    if kind == "attention":
        return PubunexAttention(kv_heads=kv_heads(), scale=scale, rot=rot,
                                **ints("heads", "dim", "vdim"))
    if rot is None:
        raise ConfigError(f"config.json: required key '{where}rot' is missing")
    return PubunexLatent(scale=scale, rot=rot,
                         **ints("heads", "dim", "rot_dim", "vdim", "kv_rank"))


def _read_expert(d: Any, where: str) -> PubunexExpert:
    return PubunexExpert(_get(d, "ff", where), _get(d, "limit", where, float))


def _read_mlp(f: Any, where: str) -> Optional[PubunexExperts]:
    if f is None:
        return None
    if _get(f, "kind", where, typ=None) != "moe":
        raise ConfigError(f"config.json: '{where}kind' = {f['kind']!r} is not a feed-forward of "
                          "this design (known: moe)")
    r = _get(f, "router", where, typ=None)
    return PubunexExperts(
        experts=_get(r, "experts", where + "router."), top=_get(r, "top", where + "router."),
        expert=_read_expert(_get(f, "expert", where, typ=None), where + "expert."),
        shared=None if f.get("shared") is None else _read_expert(f["shared"], where + "shared."))


def _check_rotation(rot: PubunexRotation, size: int, where: str) -> None:
    if rot.dims <= 0 or rot.dims % 2 or rot.dims > size:
        raise ConfigError(f"config.json: '{where}dims' ({rot.dims}) must be even and at most "
                          f"{size}")
    if rot.base <= 0 or (rot.scaling is not None and rot.base == 1.0):
        raise ConfigError(f"config.json: '{where}base' must be positive (and not 1 where "
                          "frequencies are scaled)")
    if rot.scaling is not None:
        _positive(rot.scaling, ("factor", "original", "fast", "slow"), where + "scaling.")


def _check_mixer(kind: str, m: Any, where: str) -> None:
    if kind == "latent_attention":
        _positive(m, ("heads", "dim", "rot_dim", "vdim", "kv_rank", "scale"), where)
        if m.rot.dims != m.rot_dim:
            raise ConfigError(f"config.json: '{where}rot.dims' ({m.rot.dims}) must equal "
                              f"'rot_dim' ({m.rot_dim})")
        _check_rotation(m.rot, m.rot_dim, where + "rot.")
        return
    _positive(m, ("heads", "kv_heads", "dim", "vdim"), where)
    if m.heads % m.kv_heads:
        raise ConfigError(f"config.json: '{where}heads' ({m.heads}) must be a multiple of "
                          f"'kv_heads' ({m.kv_heads})")
    if kind == "delta":
        _positive(m, ("conv",), where)
        return
    _positive(m, ("scale",), where)
    if m.rot is not None:
        _check_rotation(m.rot, m.dim, where + "rot.")


def _write_rotation(rot: PubunexRotation) -> Dict[str, Any]:
    d: Dict[str, Any] = {"base": rot.base, "dims": rot.dims}
    if rot.scaling is not None:
        d["scaling"] = {k: getattr(rot.scaling, k) for k in ("factor", "fast", "original", "slow")}
    return d


@dataclass(frozen=True)
class PubunexConfig:
    vocab: int
    width: int
    norm_eps: float
    layers: Tuple[PubunexLayer, ...]
    loop: Optional[PubunexLoop] = None
    bos_token_id: Optional[int] = None
    eos_token_ids: Tuple[int, ...] = ()

    architecture = "Pubunex"

    # ------------------------------------------------------------------ read
    @classmethod
    def from_dict(cls, raw: Dict[str, Any]) -> "PubunexConfig":
        layers_raw = _get(raw, "layers", "", typ=None)
        if not isinstance(layers_raw, list):
            raise ConfigError("config.json: 'layers' must be a list")
        layers = []
        for i, entry in enumerate(layers_raw):
            where = f"layers[{i}]."
            kind = _get(entry, "type", where, typ=None)
            if kind not in MIXERS:
                raise ConfigError(f"config.json: '{where}type' = {kind!r} is not a mixer of this "
                                  f"design (known: {', '.join(MIXERS)})")
            layers.append(PubunexLayer(
                kind, _read_mixer(kind, _get(entry, "mixer", where, typ=None), where + "mixer."),
                _read_mlp(entry.get("mlp"), where + "mlp.")))
        loop = raw.get("loop")
        if loop is not None:
            loop = PubunexLoop(**{k: _get(loop, k, "loop.") for k in ("start", "stop", "times")})
        eos = raw.get("eos_token_id")
        eos_ids = () if eos is None else tuple(int(e) for e in eos) if isinstance(eos, list) \
            else (int(eos),)
        bos = raw.get("bos_token_id")
        cfg = cls(vocab=_get(raw, "vocab", ""), width=_get(raw, "width", ""),
                  norm_eps=_get(_get(raw, "norm", "", typ=None), "eps", "norm.", float),
                  layers=tuple(layers), loop=loop,
                  bos_token_id=None if bos is None else int(bos), eos_token_ids=eos_ids)
        cfg.validate()
        return cfg

    def validate(self) -> None:
        if self.vocab <= 0 or self.width <= 0:
            raise ConfigError("config.json: 'vocab' and 'width' must be positive")
        if self.norm_eps <= 0:
            raise ConfigError("config.json: 'norm.eps' must be positive")
        for i, layer in enumerate(self.layers):
            _check_mixer(layer.kind, layer.mixer, f"layers[{i}].mixer.")
            f, where = layer.mlp, f"layers[{i}].mlp."
            if f is not None:
                if not 0 < f.top <= f.experts:
                    raise ConfigError(f"config.json: '{where}router.top' ({f.top}) must be "
                                      f"between 1 and 'experts' ({f.experts})")
                _positive(f.expert, ("ff", "limit"), where + "expert.")
                if f.shared is not None:
                    _positive(f.shared, ("ff", "limit"), where + "shared.")
        lp = self.loop
        if lp is not None and not (0 <= lp.start < lp.stop <= len(self.layers) and lp.times >= 1):
            raise ConfigError(f"config.json: 'loop' must name layers start < stop of the "
                              f"{len(self.layers)} there are and run them at least once")

    # ----------------------------------------------------------------- write
    def to_dict(self) -> Dict[str, Any]:
        layers = []
        for layer in self.layers:
            m, f = layer.mixer, layer.mlp
            keys = {"delta": ("conv", "dim", "heads", "kv_heads", "vdim"),
                    "attention": ("dim", "heads", "kv_heads", "scale", "vdim"),
                    "latent_attention": ("dim", "heads", "kv_rank", "rot_dim", "scale",
                                         "vdim")}[layer.kind]
            mixer = {k: getattr(m, k) for k in keys}
            if layer.kind != "delta" and m.rot is not None:
                mixer["rot"] = _write_rotation(m.rot)
            mlp = None
            if f is not None:
                mlp = {"expert": {"ff": f.expert.ff, "limit": f.expert.limit}, "kind": "moe",
                       "router": {"experts": f.experts, "top": f.top}}
                if f.shared is not None:
                    mlp["shared"] = {"ff": f.shared.ff, "limit": f.shared.limit}
            layers.append({"mixer": mixer, "mlp": mlp, "type": layer.kind})
        d: Dict[str, Any] = {"architecture": self.architecture, "layers": layers,
                             "norm": {"eps": self.norm_eps}, "vocab": self.vocab,
                             "width": self.width}
        if self.loop is not None:
            d["loop"] = {k: getattr(self.loop, k) for k in ("start", "stop", "times")}
        if self.bos_token_id is not None:
            d["bos_token_id"] = self.bos_token_id
        if self.eos_token_ids:
            d["eos_token_id"] = list(self.eos_token_ids)
        return d

    # ----------------------------------------------------------------- lower
    @staticmethod
    def _rotary(rot: PubunexRotation, size: int, interleaved: bool) -> RotarySpec:
        sc = rot.scaling
        if sc is not None:
            sc = WavelengthScalingSpec(factor=sc.factor, original=sc.original, fast=sc.fast,
                                       slow=sc.slow)
        return RotarySpec(theta=rot.base, rotary_dim=0 if rot.dims == size else rot.dims,
                          interleaved=interleaved, scaling=sc)

    def _mixer_spec(self, layer: PubunexLayer):
        m = layer.mixer
        if layer.kind == "delta":
            return HeadDeltaSpec(n_heads=m.heads, n_qk_heads=m.kv_heads, head_dim=m.dim,
                                 value_dim=m.vdim, conv_taps=m.conv, eps=self.norm_eps,
                                 unit_eps=UNIT_EPS, gate_activation="silu")
        if layer.kind == "attention":
            return AttentionSpec(
                n_heads=m.heads, n_kv_heads=m.kv_heads, head_dim=m.dim, scale=m.scale,
                value_dim=0 if m.vdim == m.dim else m.vdim, qkv_bias=True, out_bias=True,
                position=None if m.rot is None else self._rotary(m.rot, m.dim, False))
        return LatentAttentionSpec(
            n_heads=m.heads, head_dim=m.dim, rot_dim=m.rot_dim, value_dim=m.vdim,
            kv_rank=m.kv_rank, q_rank=0, scale=m.scale, eps=self.norm_eps, gate=None, sink=True,
            position=self._rotary(m.rot, m.rot_dim, True))

    @staticmethod
    def _ffn_spec(f: Optional[PubunexExperts]) -> Optional[RoutedFeedForwardSpec]:
        if f is None:
            return None
        return RoutedFeedForwardSpec(
            n_experts=f.experts, top=f.top, intermediate_size=f.expert.ff,
            activation=ClampedGateSpec(limit=f.expert.limit, alpha=GATE_ALPHA), n_groups=1,
            keep_groups=1, correction=False, weighting="sigmoid", weigh_input=True,
            shared_size=0 if f.shared is None else f.shared.ff, shared_gate=False,
            shared_activation=None if f.shared is None else
            ClampedGateSpec(limit=f.shared.limit, alpha=GATE_ALPHA))

    def to_model_spec(self) -> ModelSpec:
        norm = NormSpec(eps=self.norm_eps, zero_centered=True)
        blocks = tuple(ParallelBlockSpec(mixer=self._mixer_spec(layer),
                                         feed_forward=self._ffn_spec(layer.mlp), norm=norm,
                                         gated=False) for layer in self.layers)
        lp, n = self.loop, len(self.layers)
        schedule = (default_schedule(n) if lp is None else
                    looped_schedule(n, lp.start, lp.stop, lp.times, add_embedding=True))
        return ModelSpec(
            hidden_size=self.width, vocab_size=self.vocab, embed_scale=1.0, blocks=blocks,
            schedule=schedule, final_norm=norm, tie_embeddings=False, max_positions=0,
            bos_token_id=self.bos_token_id, eos_token_ids=self.eos_token_ids)
