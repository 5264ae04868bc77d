"""Rotary position encoding as a table of cosines and sines.

`freq_j = theta^(-2j/D)`, `angle = float(position) * freq_j`, all in float32, as
src/minillm/runtime.cpp:231-241 computes them for each step and
src/minillm/cuda/storage.cpp:261-287 tabulates them once ([positions, D], cosines
in the first half of a row, sines in the second).  The table is made on the host
with float32 `pow`, multiply, `cos` and `sin`, then uploaded; the mixer's kernel
rotates `(x[j], x[j + D/2])` pairs with it.
Parameters: theta, rotary_dim, max_positions.  No weights.
"""
from __future__ import annotations

import math
from typing import Optional, Tuple

import numpy as np
import torch

from ..config.base import ConfigError
from ..config.registry import register_part
from .base import PositionEncoding


def rotation_table(theta: float, rotary_dim: int, max_positions: int) -> torch.Tensor:
    half = rotary_dim // 2
    j = np.arange(half, dtype=np.float32)
    exponent = (np.float32(-2.0) * j / np.float32(rotary_dim)).astype(np.float32)
    freq = np.power(np.float32(theta), exponent).astype(np.float32)
    pos = np.arange(max_positions, dtype=np.float32)[:, None]
    angle = (pos * freq[None, :]).astype(np.float32)
    table = np.concatenate([np.cos(angle), np.sin(angle)], axis=1).astype(np.float32)
    return torch.from_numpy(table)


class Rope(PositionEncoding):
    def __init__(self, spec):
        super().__init__(spec)
        self.theta = float(spec.params["theta"])
        self.rotary_dim = int(spec.params["rotary_dim"])
        self.max_positions = int(spec.params["max_positions"])
        if self.rotary_dim % 2:
            raise ValueError(f"rotary_dim {self.rotary_dim} must be even")
        self._table: Optional[torch.Tensor] = None

    def bind(self, tensors, rt) -> None:
        self._table = rotation_table(self.theta, self.rotary_dim, self.max_positions).to(rt.device)

    def rotation_table(self) -> Optional[torch.Tensor]:
        return self._table


register_part("position", "rope", Rope)


def scaled_frequencies(freq: np.ndarray, factor: float, low: float, high: float, original: float) -> np.ndarray:
    """Frequencies whose long wavelengths are slowed down, as a model does that was trained on `original` positions and
    is to read `factor` times as many: with the wavelength l = 2 pi / f, a frequency stays where l < original / high,
    becomes f / factor where l > original / low, and in between is the blend (1 - s) f / factor + s f with
    s = (original / l - low) / (high - low).  float64 in, float64 out."""
    freq = np.asarray(freq, dtype=np.float64)
    length = 2.0 * np.pi / freq
    s = (original / length - low) / (high - low)
    blend = (1.0 - s) * freq / factor + s * freq
    return np.where(length < original / high, freq, np.where(length > original / low, freq / factor, blend))


def yarn_frequencies(base: float, dims: int, factor: float, original: float, fast: float, slow: float) -> Tuple[np.ndarray, float]:
    """YaRN: frequencies that turn fewer than `slow` times within `original` positions are divided by `factor`, those that turn more than
    `fast` times stay, with a ramp over the pair index in between; and the factor 0.1 ln(factor) + 1 on every cosine and sine.
    The pair whose frequency turns t times is dims ln(original / (2 pi t)) / (2 ln base); the ramp's ends are those of `fast`, rounded
    down and at least 0, and of `slow`, rounded up and at most dims - 1.  float64."""
    i = np.arange(dims // 2, dtype=np.float64)
    freq = np.power(base, -2.0 * i / max(dims, 1))
    pair_of = lambda turns: dims * math.log(original / (2.0 * math.pi * turns)) / (2.0 * math.log(base))
    lo, hi = max(math.floor(pair_of(fast)), 0), min(math.ceil(pair_of(slow)), dims - 1)
    ramp = np.clip((i - lo) / max(hi - lo, 0.001), 0.0, 1.0)
    return freq / factor * ramp + freq * (1.0 - ramp), 0.1 * math.log(factor) + 1.0


class RotaryFrequencies(PositionEncoding):
    """Rotation given as its frequencies only: `freq_i = base^(-2i/dims) / factor`, i < dims/2.  The kernels
    that use it compute `position * freq_i` and its cosine and sine in float32 themselves, so no table
    exists and no largest position: `factor` > 1 is linear position scaling.  Only the first `dims`
    values of a head are rotated; a mixer's heads may be wider.  Value i turns with value i + dims/2, or, with
    `interleaved`, value 2i with value 2i + 1: (u, v) -> (u cos a - v sin a, v cos a + u sin a), a = position * freq_i
    (a mixer's kernels must know that layout; those that do not refuse it).
    With `scaling` = {factor, low, high, original} only long wavelengths are slowed down (`scaled_frequencies`); with `yarn` =
    {factor, original, fast, slow} the frequencies are `yarn_frequencies`, and cosine and sine carry the factor `magnitude`, which a
    mixer's kernels must apply (`plain_rotation` refuses it for those that do not).
    Parameters: base, dims, factor (default 1), interleaved (default False), scaling, yarn (default None).  No weights."""

    def __init__(self, spec):
        super().__init__(spec)
        self.base = float(spec.params["base"])
        self.dims = int(spec.params["dims"])
        self.factor = float(spec.params.get("factor", 1.0))
        self.interleaved = bool(spec.params.get("interleaved", False))
        if self.dims < 0 or self.dims % 2 or self.base <= 0 or self.factor <= 0:
            raise ValueError(f"a rotation of {self.dims} values with base {self.base} and factor {self.factor} is not defined")
        scaling = spec.params.get("scaling")
        self.scaling = {k: float(scaling[k]) for k in ("factor", "low", "high", "original")} if scaling else None
        if self.scaling is not None and not (self.scaling["high"] > self.scaling["low"] and self.scaling["factor"] > 0
                                             and self.scaling["original"] > 0):
            raise ValueError(f"a frequency scaling {self.scaling} is not defined")
        yarn = spec.params.get("yarn")
        self.yarn = {k: float(yarn[k]) for k in ("factor", "original", "fast", "slow")} if yarn else None
        self._yarn_freq, self.magnitude = None, 1.0
        if self.yarn is not None:
            if min(self.yarn.values()) <= 0 or self.base == 1.0 or self.scaling is not None or self.factor != 1.0:
                raise ValueError(f"a YaRN scaling {self.yarn} with base {self.base} is not defined (it excludes any other scaling)")
            self._yarn_freq, self.magnitude = yarn_frequencies(self.base, self.dims, **self.yarn)
        self._freq: Optional[torch.Tensor] = None

    def bind(self, tensors, rt) -> None:
        if self._yarn_freq is not None:
            self._freq = torch.from_numpy(self._yarn_freq.astype(np.float32)).to(rt.device)
            return
        i = np.arange(self.dims // 2, dtype=np.float64)
        freq = np.power(self.base, -2.0 * i / max(self.dims, 1)) / self.factor
        if self.scaling is not None:
            freq = scaled_frequencies(freq, **self.scaling)
        self._freq = torch.from_numpy(freq.astype(np.float32)).to(rt.device)

    def frequencies(self) -> torch.Tensor:
        return self._freq


def plain_rotation(position):
    """`position`, unless it needs a factor on cosine and sine that the caller's kernels do not apply."""
    if getattr(position, "magnitude", 1.0) != 1.0:
        raise ConfigError("this mixer rotates by plain cosines and sines: a scaling with a factor on them needs another")
    return position


register_part("position", "rotary_frequencies", RotaryFrequencies)
