"""Typed configuration of the Repolix decoder, read from its config.json.

    {"architecture": "Repolix", "vocab": V, "width": W, "norm": {"eps"}, "embedding": {"scale"},
     "layers": [{"type": "attention" | "mamba2" | "channel_delta", "mixer": {...}, "mlp": {...} | null}, ...]}

An "attention" mixer (differential attention) has heads, dim (of a query or key of ONE of a head's two maps), vdim, scale, diff, conv
(taps) and optionally kv_heads, mask.size (a sliding window) and rot = {base, dims, optionally scaling = {factor, original, fast, slow}}.
A "mamba2" mixer has heads, vdim, state, groups, conv and norm_groups; a "channel_delta" mixer has heads, dim, vdim, conv and optionally
kv_heads (heads of q and k).  A feed-forward is {"kind": "moe", "expert": {ff, limit}, "router": {experts, top, optionally groups =
{count, keep} and identity}, optionally "shared": {ff, limit}}; groups are formed over the experts and the identity experts together.
Every size and constant comes from the file; a missing required key is an error, and what the file leaves out does not exist.

The rows of the first matrices of the low-rank products of a "channel_delta" mixer are sizes that only the stored tensors give:
`with_stored_shapes` takes them from there (where no tensors exist, the optional mixer keys decay_rank and gate_rank or a default).  The
design names no largest position; `max_positions` is this engine's bound on a request's length.
"""
from __future__ import annotations

from dataclasses import dataclass, replace
from typing import Any, Dict, Optional, Tuple

from .base import ConfigError
from .gelulix import ChannelDeltaConfig, YarnRotation, _rank, _rotation
from .gopevik import MAX_POSITIONS, _get, _integer, _number
from .sokolorn import ExpertShape, _expert


@dataclass(frozen=True)
class DifferentialConfig:
    heads: int
    kv_heads: int
    dim: int
    vdim: int
    scale: float
    diff: float
    conv: int
    window: Optional[int]
    rot: Optional[YarnRotation]


@dataclass(frozen=True)
class StateSpaceConfig:
    heads: int
    groups: int
    state: int
    vdim: int
    conv: int
    norm_groups: int


@dataclass(frozen=True)
class RoutedConfig:
    expert: ExpertShape
    experts: int
    identity: int
    top: int
    groups: int
    keep: int
    shared: Optional[ExpertShape]


@dataclass(frozen=True)
class RepolixLayer:
    type: str
    mixer: Any
    mlp: Optional[RoutedConfig]


def _shared_by(m: dict, key: str, heads: int, where: str) -> int:
    n = _integer(m, key, where) if m.get(key) is not None else heads
    if heads % n:
        raise ConfigError(f"config.json key {where}{key!r} = {n} does not divide the {heads} heads")
    return n


@dataclass(frozen=True)
class RepolixConfig:
    architecture: str
    vocab_size: int
    width: int
    norm_eps: float
    embedding_scale: float
    layers: Tuple[RepolixLayer, ...]
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
    def from_dict(cls, raw: dict) -> "RepolixConfig":
        listed = _get(raw, "layers", "")
        if not isinstance(listed, list) or not listed:
            raise ConfigError("config.json key 'layers' must be a non-empty list")
        layers = []
        for i, layer in enumerate(listed):
            where = f"layers[{i}]."
            kind = _get(layer, "type", where)
            m = _get(layer, "mixer", where)
            mw = where + "mixer."
            heads, vdim, conv = (_integer(m, key, mw) for key in ("heads", "vdim", "conv"))
            if kind == "attention":
                dim = _integer(m, "dim", mw)
                mask = m.get("mask")
                window = _integer(mask, "size", mw + "mask.") if mask is not None and mask.get("size") is not None else None
                rot = _rotation(m["rot"], mw + "rot.", dim) if m.get("rot") is not None else None
                mixer = DifferentialConfig(heads, _shared_by(m, "kv_heads", heads, mw), dim, vdim, _number(m, "scale", mw, positive=False),
                                           _number(m, "diff", mw, positive=False), conv, window, rot)
            elif kind == "mamba2":
                parts = _integer(m, "norm_groups", mw)
                if heads * vdim % parts:
                    raise ConfigError(f"config.json key {mw}'norm_groups' = {parts} does not divide the {heads * vdim} values of all heads")
                _get(m, "groups", mw)
                mixer = StateSpaceConfig(heads, _shared_by(m, "groups", heads, mw), _integer(m, "state", mw), vdim, conv, parts)
            elif kind == "channel_delta":
                dim = _integer(m, "dim", mw)
                mixer = ChannelDeltaConfig(heads, _shared_by(m, "kv_heads", heads, mw), dim, vdim, conv, _rank(m, "decay_rank", mw, dim),
                                           _rank(m, "gate_rank", mw, vdim))
            else:
                raise ConfigError(f"config.json key {where}'type' = {kind!r} is not one of 'attention', 'mamba2', 'channel_delta'")
            layers.append(RepolixLayer(kind, mixer, cls._mlp(layer.get("mlp"), where + "mlp.")))
        eos = raw.get("eos_token_id", ())
        eos = (eos,) if isinstance(eos, int) else tuple(eos or ())
        return cls(architecture=_get(raw, "architecture", ""), vocab_size=_integer(raw, "vocab", ""), width=_integer(raw, "width", ""),
                   norm_eps=_number(_get(raw, "norm", ""), "eps", "norm."),
                   embedding_scale=_number(_get(raw, "embedding", ""), "scale", "embedding.", positive=False), layers=tuple(layers),
                   max_position_embeddings=int(raw.get("max_positions", MAX_POSITIONS)), eos_token_ids=eos)

    @staticmethod
    def _mlp(mlp: Optional[dict], where: str) -> Optional[RoutedConfig]:
        if mlp is None:
            return None
        if _get(mlp, "kind", where) != "moe":
            raise ConfigError(f"config.json key {where}'kind' = {mlp['kind']!r}; this design has 'moe'")
        router, rw = _get(mlp, "router", where), where + "router."
        experts, top = _integer(router, "experts", rw), _integer(router, "top", rw)
        identity = _integer(router, "identity", rw) if router.get("identity") else 0
        groups = keep = 1
        if router.get("groups") is not None:
            groups, keep = _integer(router["groups"], "count", rw + "groups."), _integer(router["groups"], "keep", rw + "groups.")
        everyone = experts + identity
        if everyone % groups or keep > groups or top > keep * (everyone // groups):
            raise ConfigError(f"config.json {where}router: {experts} experts and {identity} identity experts in {groups} 'groups' of which "
                              f"{keep} are kept cannot give {top}")
        shared = mlp.get("shared")
        return RoutedConfig(_expert(_get(mlp, "expert", where), where + "expert."), experts, identity, top, groups, keep,
                            _expert(shared, where + "shared.") if shared is not None else None)

    def with_stored_shapes(self, shapes: Dict[str, Tuple[int, ...]]) -> "RepolixConfig":
        """The configuration with the ranks that the stored tensors have (a missing tensor is the loader's to report)."""
        def rows(name: str, otherwise: int) -> int:
            shape = shapes.get(name)
            return int(shape[0]) if shape is not None and len(shape) == 2 else otherwise

        layers = []
        for i, layer in enumerate(self.layers):
            m, p = layer.mixer, f"l{i}.mix."
            if isinstance(m, ChannelDeltaConfig):
                layer = replace(layer, mixer=replace(m, decay_rank=rows(p + "a1", m.decay_rank), gate_rank=rows(p + "g1", m.gate_rank)))
            layers.append(layer)
        return replace(self, layers=tuple(layers))
