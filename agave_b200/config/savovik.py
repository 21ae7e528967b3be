"""Typed configuration of the Savovik decoder, read from its own ``config.json`` keys.

A Savovik model is a list of layers.  Each entry names its mixer (``type``: ``parallel``,
``mamba2`` or ``attention``), the mixer's sizes and constants (``mixer``) and its feed-forward
(``mlp``: a dense one, or null for a layer without).  An entry with ``weights_of: j`` has no
tensors of its own: it runs layer j's mixer, feed-forward and norm with a cache and state of
its own.  The top level gives the width, the vocabulary and the norms' eps (``norm.eps``).
Every size and every constant that can differ between two models of the design is read from
there.

What the design fixes, and what therefore stands in the lowering below: mixer and feed-forward
of a layer read one zero-centred RMS norm of the stream side by side, and each result joins it
times a sigmoid of a biased projection of that norm; ``parallel`` is two mixers on one input,
their outputs weighted by ``left_scale`` and ``right_scale`` and added: attention over chunks of
positions (biases on q, k and v, a per-head norm of q and k, neighbouring dimensions rotated,
frequencies scaled in three bands of wavelength) and a selective scan; ``mamba2`` is the scan
with one decay per head and token; ``attention`` rotates split halves with frequencies divided
by a factor, divides every value head by its root mean square, caps its scores and sees a
sliding window; the feed-forward is dense with the erf GELU and no gate; the head is a table of
its own.
"""
from __future__ import annotations

from dataclasses import dataclass
from typing import Any, Dict, Optional, Tuple

from .base import (AttentionSpec, BandScalingSpec, ConfigError, DenseFeedForwardSpec, LayerCall,
                   ModelSpec, NormSpec, ParallelBlockSpec, RotarySpec, SelectiveScanSpec,
                   SideBySideSpec, StateSpaceSpec)

MIXERS = ("parallel", "mamba2", "attention")


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


@dataclass(frozen=True)
class SavovikScaling:
    """``factor`` alone divides every frequency; with the three bounds the frequencies are
    scaled in bands of wavelength."""
    factor: float
    bounds: Optional[Tuple[float, float, float]] = None      # (low, high, original)


@dataclass(frozen=True)
class SavovikRotation:
    dims: int
    base: float
    scaling: Optional[SavovikScaling] = None


@dataclass(frozen=True)
class SavovikAttention:
    heads: int
    kv_heads: int
    dim: int
    vdim: int
    scale: float
    mask: Optional[int] = None                # chunk or window size; None: every earlier key
    rot: Optional[SavovikRotation] = None
    softcap: Optional[float] = None


@dataclass(frozen=True)
class SavovikScan:
    inner: int
    state: int
    dt_rank: int
    conv: int


@dataclass(frozen=True)
class SavovikParallel:
    left: SavovikAttention
    right: SavovikScan
    left_scale: float
    right_scale: float


@dataclass(frozen=True)
class SavovikMamba2:
    heads: int
    vdim: int
    state: int
    groups: int
    norm_groups: int
    conv: int


@dataclass(frozen=True)
class SavovikLayer:
    kind: str
    mixer: object                             # the record of the kind
    ff: Optional[int]                         # width of the feed-forward; None: there is none
    weights_of: Optional[int] = None


def _read_attention(m: dict, where: str) -> SavovikAttention:
    heads = _get(m, "heads", where)
    rot = None
    if m.get("rot") is not None:
        r, w = m["rot"], where + "rot."
        sc = r.get("scaling")
        if sc is not None:
            ws = w + "scaling."
            bounds = None
            if any(sc.get(k) is not None for k in ("low", "high", "original")):
                bounds = tuple(_get(sc, k, ws, float) for k in ("low", "high", "original"))
            sc = SavovikScaling(_get(sc, "factor", ws, float), bounds)
        rot = SavovikRotation(_get(r, "dims", w), _get(r, "base", w, float), sc)
    mask = m.get("mask")
    return SavovikAttention(
        heads=heads, kv_heads=_get(m, "kv_heads", where) if m.get("kv_heads") is not None else heads,
        dim=_get(m, "dim", where), vdim=_get(m, "vdim", where), scale=_get(m, "scale", where, float),
        mask=_get(mask, "size", where + "mask.") if mask is not None else None, rot=rot,
        softcap=_get(m, "softcap", where, float) if m.get("softcap") is not None else None)


def _read_mixer(kind: str, m: dict, where: str):
    if kind == "attention":
        return _read_attention(m, where)
    if kind == "mamba2":
        return SavovikMamba2(**{k: _get(m, k, where) for k in
                                ("heads", "vdim", "state", "groups", "norm_groups", "conv")})
    return SavovikParallel(
        left=_read_attention(_get(m, "left", where, typ=None), where + "left."),
        right=SavovikScan(**{k: _get(_get(m, "right", where, typ=None), k, where + "right.")
                             for k in ("inner", "state", "dt_rank", "conv")}),
        left_scale=_get(m, "left_scale", where, float),
        right_scale=_get(m, "right_scale", where, float))


def _check_attention(m: SavovikAttention, where: str) -> None:
    for k in ("heads", "kv_heads", "dim", "vdim"):
        if getattr(m, k) <= 0:
            raise ConfigError(f"config.json: '{where}{k}' must be positive")
    if m.heads % m.kv_heads:
        raise ConfigError(f"config.json: '{where}heads' ({m.heads}) must be a multiple of "
                          f"'kv_heads' ({m.kv_heads})")
    if m.scale <= 0:
        raise ConfigError(f"config.json: '{where}scale' must be positive")
    if m.mask is not None and m.mask <= 0:
        raise ConfigError(f"config.json: '{where}mask.size' must be positive")
    if m.softcap is not None and m.softcap <= 0:
        raise ConfigError(f"config.json: '{where}softcap' must be positive")
    if m.rot is not None:
        if m.rot.dims <= 0 or m.rot.dims % 2 or m.rot.dims > m.dim:
            raise ConfigError(f"config.json: '{where}rot.dims' ({m.rot.dims}) must be even and at "
                              f"most 'dim' ({m.dim})")
        if m.rot.base <= 0:
            raise ConfigError(f"config.json: '{where}rot.base' must be positive")
        sc = m.rot.scaling
        if sc is not None:
            if sc.factor <= 0:
                raise ConfigError(f"config.json: '{where}rot.scaling.factor' must be positive")
            if sc.bounds is not None:
                low, high, original = sc.bounds
                if original <= 0 or low <= 0 or high <= low:
                    raise ConfigError(f"config.json: '{where}rot.scaling' needs a positive "
                                      "'original' and 0 < 'low' < 'high'")


def _check_mixer(kind: str, m, where: str) -> None:
    if kind == "attention":
        _check_attention(m, where)
    elif kind == "parallel":
        _check_attention(m.left, where + "left.")
        for k in ("inner", "state", "dt_rank", "conv"):
            if getattr(m.right, k) <= 0:
                raise ConfigError(f"config.json: '{where}right.{k}' must be positive")
    else:
        for k in ("heads", "vdim", "state", "groups", "norm_groups", "conv"):
            if getattr(m, k) <= 0:
                raise ConfigError(f"config.json: '{where}{k}' must be positive")
        if m.heads % m.groups:
            raise ConfigError(f"config.json: '{where}heads' ({m.heads}) must be a multiple of "
                              f"'groups' ({m.groups})")
        if (m.heads * m.vdim) % m.norm_groups:
            raise ConfigError(f"config.json: '{where}norm_groups' ({m.norm_groups}) must divide "
                              f"heads * vdim ({m.heads * m.vdim})")


def _write_attention(m: SavovikAttention) -> Dict[str, Any]:
    d: Dict[str, Any] = {"dim": m.dim, "heads": m.heads, "kv_heads": m.kv_heads,
                         "scale": m.scale, "vdim": m.vdim}
    if m.mask is not None:
        d["mask"] = {"size": m.mask}
    if m.rot is not None:
        d["rot"] = {"base": m.rot.base, "dims": m.rot.dims}
        if m.rot.scaling is not None:
            d["rot"]["scaling"] = {"factor": m.rot.scaling.factor}
            if m.rot.scaling.bounds is not None:
                d["rot"]["scaling"].update(zip(("low", "high", "original"), m.rot.scaling.bounds))
    if m.softcap is not None:
        d["softcap"] = m.softcap
    return d


@dataclass(frozen=True)
class SavovikConfig:
    vocab: int
    width: int
    norm_eps: float
    layers: Tuple[SavovikLayer, ...]
    bos_token_id: Optional[int] = None
    eos_token_ids: Tuple[int, ...] = ()

    architecture = "Savovik"

    # ------------------------------------------------------------------ read
    @classmethod
    def from_dict(cls, raw: Dict[str, Any]) -> "SavovikConfig":
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
            mixer = _read_mixer(kind, _get(entry, "mixer", where, typ=None), where + "mixer.")
            ff = None                          # (no 'mlp' key reads as null: no feed-forward)
            if entry.get("mlp") is not None:
                f = entry["mlp"]
                if _get(f, "kind", where + "mlp.", typ=None) != "dense":
                    raise ConfigError(f"config.json: '{where}mlp.kind' = {f['kind']!r} is not a "
                                      "feed-forward of this design (known: dense)")
                ff = _get(f, "ff", where + "mlp.")
            wo = entry.get("weights_of")
            layers.append(SavovikLayer(kind, mixer, ff,
                                       None if wo is None else _get(entry, "weights_of", where)))
        eos = raw.get("eos_token_id")
        eos_ids = () if eos is None else tuple(int(e) for e in eos) if isinstance(eos, list) \
            else (int(eos),)
        bos = raw.get("bos_token_id")
        cfg = cls(vocab=_get(raw, "vocab", ""), width=_get(raw, "width", ""),
                  norm_eps=_get(_get(raw, "norm", "", typ=None), "eps", "norm.", float),
                  layers=tuple(layers), bos_token_id=None if bos is None else int(bos),
                  eos_token_ids=eos_ids)
        cfg.validate()
        return cfg

    def validate(self) -> None:
        if self.vocab <= 0 or self.width <= 0:
            raise ConfigError("config.json: 'vocab' and 'width' must be positive")
        if self.norm_eps <= 0:
            raise ConfigError("config.json: 'norm.eps' must be positive")
        for i, layer in enumerate(self.layers):
            _check_mixer(layer.kind, layer.mixer, f"layers[{i}].mixer.")
            if layer.ff is not None and layer.ff <= 0:
                raise ConfigError(f"config.json: 'layers[{i}].mlp.ff' must be positive")
            if layer.weights_of is not None:
                src = self.layers[self.owner(i)]
                if (src.kind, src.mixer, src.ff) != (layer.kind, layer.mixer, layer.ff):
                    raise ConfigError(f"config.json: 'layers[{i}]' must equal the layer whose "
                                      f"weights it uses (layers[{layer.weights_of}])")

    # ----------------------------------------------------------------- write
    def to_dict(self) -> Dict[str, Any]:
        layers = []
        for layer in self.layers:
            m = layer.mixer
            if layer.kind == "attention":
                mixer = _write_attention(m)
            elif layer.kind == "mamba2":
                mixer = {k: getattr(m, k) for k in
                         ("conv", "groups", "heads", "norm_groups", "state", "vdim")}
            else:
                mixer = {"left": _write_attention(m.left), "left_scale": m.left_scale,
                         "right": {k: getattr(m.right, k) for k in
                                   ("conv", "dt_rank", "inner", "state")},
                         "right_scale": m.right_scale}
            e: Dict[str, Any] = {"mixer": mixer, "type": layer.kind,
                                 "mlp": None if layer.ff is None else {"ff": layer.ff,
                                                                       "kind": "dense"}}
            if layer.weights_of is not None:
                e["weights_of"] = layer.weights_of
            layers.append(e)
        d: Dict[str, Any] = {"architecture": self.architecture, "layers": layers,
                             "norm": {"eps": self.norm_eps}, "vocab": self.vocab,
                             "width": self.width}
        if self.bos_token_id is not None:
            d["bos_token_id"] = self.bos_token_id
        if self.eos_token_ids:
            d["eos_token_id"] = list(self.eos_token_ids)
        return d

    # ----------------------------------------------------------------- lower
    def owner(self, i: int) -> int:
        """The layer whose tensors layer i runs (itself, or what ``weights_of`` leads to)."""
        seen = {i}
        while self.layers[i].weights_of is not None:
            j = self.layers[i].weights_of
            if not 0 <= j < len(self.layers) or j in seen:
                raise ConfigError(f"config.json: 'layers[{i}].weights_of' = {j} must name another "
                                  "layer, and lead to one with tensors of its own")
            seen.add(j)
            i = j
        return i

    def owners(self) -> Tuple[int, ...]:
        """Layer numbers that have tensors of their own, in order: block b of the lowered
        model is layer ``owners()[b]``."""
        return tuple(i for i, layer in enumerate(self.layers) if layer.weights_of is None)

    def _attention_spec(self, m: SavovikAttention, chunked: bool) -> AttentionSpec:
        position = None
        if m.rot is not None:
            sc, band, factor = m.rot.scaling, None, 1.0
            if sc is not None and sc.bounds is not None:
                low, high, original = sc.bounds
                band = BandScalingSpec(factor=sc.factor, original=original, low=low, high=high)
            elif sc is not None:
                factor = sc.factor             # (dividing the position divides every frequency)
            position = RotarySpec(theta=m.rot.base, factor=factor, interleaved=chunked,
                                  rotary_dim=0 if m.rot.dims == m.dim else m.rot.dims, scaling=band)
        return AttentionSpec(
            n_heads=m.heads, n_kv_heads=m.kv_heads, head_dim=m.dim, scale=m.scale,
            value_dim=0 if m.vdim == m.dim else m.vdim, position=position, softcap=m.softcap,
            window=None if chunked else m.mask, chunk=m.mask if chunked else None,
            qk_norm=NormSpec(eps=self.norm_eps, zero_centered=False) if chunked else None,
            qkv_bias=chunked, value_norm_eps=None if chunked else self.norm_eps)

    def _mixer_spec(self, layer: SavovikLayer):
        m = layer.mixer
        if layer.kind == "attention":
            return self._attention_spec(m, chunked=False)
        if layer.kind == "mamba2":
            return StateSpaceSpec(n_heads=m.heads, value_dim=m.vdim, state=m.state,
                                  n_groups=m.groups, norm_groups=m.norm_groups,
                                  conv_taps=m.conv, eps=self.norm_eps)
        return SideBySideSpec(
            left=self._attention_spec(m.left, chunked=True),
            right=SelectiveScanSpec(inner=m.right.inner, state=m.right.state,
                                    dt_rank=m.right.dt_rank, conv_taps=m.right.conv),
            left_scale=m.left_scale, right_scale=m.right_scale)

    def to_model_spec(self) -> ModelSpec:
        norm = NormSpec(eps=self.norm_eps, zero_centered=True)
        owners = self.owners()
        block_of = {layer: b for b, layer in enumerate(owners)}
        blocks = []
        for i in owners:
            layer = self.layers[i]
            ffn = None if layer.ff is None else DenseFeedForwardSpec(intermediate_size=layer.ff,
                                                                     activation="gelu_erf")
            blocks.append(ParallelBlockSpec(mixer=self._mixer_spec(layer), feed_forward=ffn,
                                            norm=norm, gated=True))
        schedule = tuple(LayerCall(block=block_of[self.owner(i)], cache=i)
                         for i in range(len(self.layers)))
        return ModelSpec(
            hidden_size=self.width, vocab_size=self.vocab, embed_scale=1.0,
            blocks=tuple(blocks), schedule=schedule, final_norm=norm, tie_embeddings=False,
            max_positions=0, bos_token_id=self.bos_token_id, eos_token_ids=self.eos_token_ids)
