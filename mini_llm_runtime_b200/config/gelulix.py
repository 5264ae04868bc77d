"""Typed configuration of the Gelulix decoder, read from its config.json.

    {"architecture": "Gelulix", "vocab": V, "width": W, "norm": {"eps"}, "postln_alpha": a,
     "layers": [{"type": "gla" | "latent_attention" | "channel_delta", "mixer": {...}, "mlp": {"kind": "dense", "ff": F} | null}, ...]}

A "gla" mixer has heads, dim, vdim and tau; a "latent_attention" mixer has heads, dim (plain query/key values per head), rot_dim
(rotated ones), vdim, kv_rank, scale and rot = {base, dims, optionally scaling = {factor, original, fast, slow}}; a "channel_delta" mixer
has heads, kv_heads (heads of q and k), dim, vdim and conv (taps).  A missing required key is an error, not a default.

The rows of the first matrices of the low-rank products ("a1", "g1") are sizes that only the stored tensors give: `with_stored_shapes`
takes them from there.  Where no tensors exist (random weights) the optional mixer keys decay_rank and gate_rank say them, else they
are a quarter of the head size, at least 8.  The design names no largest position; `max_positions` is this engine's bound on a
request's length.
"""
from __future__ import annotations

from dataclasses import dataclass, replace
from typing import Any, Dict, Optional, Tuple

from .base import ConfigError
from .gopevik import MAX_POSITIONS, _get, _integer, _number


@dataclass(frozen=True)
class YarnScaling:
    factor: float
    original: float
    fast: float
    slow: float


@dataclass(frozen=True)
class YarnRotation:
    base: float
    dims: int
    scaling: Optional[YarnScaling]


@dataclass(frozen=True)
class GatedLinearConfig:
    heads: int
    dim: int
    vdim: int
    tau: float
    decay_rank: int


@dataclass(frozen=True)
class LatentConfig:
    heads: int
    dim: int
    rot_dim: int
    vdim: int
    kv_rank: int
    scale: float
    rot: YarnRotation


@dataclass(frozen=True)
class ChannelDeltaConfig:
    heads: int
    qk_heads: int
    dim: int
    vdim: int
    conv: int
    decay_rank: int
    gate_rank: int


@dataclass(frozen=True)
class GelulixLayer:
    type: str
    mixer: Any
    ff: Optional[int]            # None: the layer has no feed-forward


def _rank(m: dict, key: str, where: str, size: int) -> int:
    return _integer(m, key, where) if m.get(key) is not None else max(8, size // 4)


def _rotation(raw: dict, where: str, size: int) -> YarnRotation:
    dims = _integer(raw, "dims", where)
    if dims % 2 or dims > size:
        raise ConfigError(f"config.json key {where}'dims' = {dims} must be even and at most the rotated size {size}")
    base = _number(raw, "base", where)
    s = raw.get("scaling")
    if s is None:
        return YarnRotation(base, dims, None)
    if base == 1.0:
        raise ConfigError(f"config.json key {where}'base' = 1 has no scaled frequencies")
    sw = where + "scaling."
    return YarnRotation(base, dims, YarnScaling(_number(s, "factor", sw), _number(s, "original", sw), _number(s, "fast", sw), _number(s, "slow", sw)))


@dataclass(frozen=True)
class GelulixConfig:
    architecture: str
    vocab_size: int
    width: int
    norm_eps: float
    alpha: float
    layers: Tuple[GelulixLayer, ...]
    max_position_embeddings: int = MAX_POSITIONS
    eos_token_ids: Tuple[int, ...] = ()
    stored_dtype: str = "bfloat16"

    @property
    def hidden_size(self) -> int:
        return self.width

    @property
    def num_hidden_layers(self) -> int:
        return len(self.layers)

    @classmethod
    def from_dict(cls, raw: dict) -> "GelulixConfig":
        listed = _get(raw, "layers", "")
        if not isinstance(listed, list) or not listed:
            raise ConfigError("config.json key 'layers' must be a non-empty list")
        layers = []
        for i, layer in enumerate(listed):
            where = f"layers[{i}]."
            kind = _get(layer, "type", where)
            m = _get(layer, "mixer", where)
            mw = where + "mixer."
            heads, dim, vdim = (_integer(m, key, mw) for key in ("heads", "dim", "vdim"))
            if kind == "gla":
                mixer = GatedLinearConfig(heads, dim, vdim, _number(m, "tau", mw), _rank(m, "decay_rank", mw, dim))
            elif kind == "latent_attention":
                rot_dim = _integer(m, "rot_dim", mw)
                mixer = LatentConfig(heads, dim, rot_dim, vdim, _integer(m, "kv_rank", mw), _number(m, "scale", mw),
                                     _rotation(_get(m, "rot", mw), mw + "rot.", rot_dim))
            elif kind == "channel_delta":
                qk = _integer(m, "kv_heads", mw) if m.get("kv_heads") is not None else heads
                if heads % qk:
                    raise ConfigError(f"config.json key {mw}'kv_heads' = {qk} does not divide the {heads} heads")
                mixer = ChannelDeltaConfig(heads, qk, dim, vdim, _integer(m, "conv", mw), _rank(m, "decay_rank", mw, dim),
                                           _rank(m, "gate_rank", mw, vdim))
            else:
                raise ConfigError(f"config.json key {where}'type' = {kind!r} is not one of 'gla', 'latent_attention', 'channel_delta'")
            mlp = layer.get("mlp")
            ff = None
            if mlp is not None:
                if _get(mlp, "kind", where + "mlp.") != "dense":
                    raise ConfigError(f"config.json key {where}mlp.'kind' = {mlp['kind']!r}; this design has 'dense'")
                ff = _integer(mlp, "ff", where + "mlp.")
            layers.append(GelulixLayer(kind, mixer, ff))
        eos = raw.get("eos_token_id", ())
        eos = (eos,) if isinstance(eos, int) else tuple(eos or ())
        return cls(architecture=_get(raw, "architecture", ""), vocab_size=_integer(raw, "vocab", ""), width=_integer(raw, "width", ""),
                   norm_eps=_number(_get(raw, "norm", ""), "eps", "norm."), alpha=_number(raw, "postln_alpha", "", positive=False),
                   layers=tuple(layers), max_position_embeddings=int(raw.get("max_positions", MAX_POSITIONS)), eos_token_ids=eos)

    def with_stored_shapes(self, shapes: Dict[str, Tuple[int, ...]]) -> "GelulixConfig":
        """The configuration with the ranks that the stored tensors have (a missing tensor is the loader's to report)."""
        def rows(name: str, otherwise: int) -> int:
            shape = shapes.get(name)
            return int(shape[0]) if shape is not None and len(shape) == 2 else otherwise

        layers = []
        for i, layer in enumerate(self.layers):
            m, p = layer.mixer, f"l{i}.mix."
            if isinstance(m, GatedLinearConfig):
                m = replace(m, decay_rank=rows(p + "a1", m.decay_rank))
            elif isinstance(m, ChannelDeltaConfig):
                m = replace(m, decay_rank=rows(p + "a1", m.decay_rank), gate_rank=rows(p + "g1", m.gate_rank))
            layers.append(replace(layer, mixer=m))
        return replace(self, layers=tuple(layers))
