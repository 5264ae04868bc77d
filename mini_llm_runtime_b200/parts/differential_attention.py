"""Differential attention over the paged cache: every head has TWO attention maps, each with queries and keys of its own, over the same
values; the head's result is their weighted difference, normed.

    q, k, v = x [Wq; Wk; Wv]^T                    one stacked product; q [H, 2, D], k [G, 2, D] (a head's two maps side by side), v [G, Dv]
    each channel of q, k, v through a causal convolution over time (no activation), q and k rotated; cache <- k, v     `mlr_conv_rotate_cache`
    a_m = softmax over the visible keys of scale * q_m . k_m, times v        (head h uses keys and values of h // (H/G))
    o = a_1 - l a_2,  o / sqrt(mean(o^2) + eps) * (1 - diff),  l = exp(lq1 . lk1) - exp(lq2 . lk2) + diff              `attention_masked`
    result = o Wo^T

A key's row in the cache holds both maps' keys, so the few-row kernel reads keys and values of a group of heads once: the maps are query
heads that are zero in the other map's half of the row.  The prompt kernel takes both maps of a head in one block over one copy of the
values and combines them before it stores.

Parameters: hidden_size, num_heads, num_kv_heads, head_dim (of one map), value_dim, scale, diff, conv (taps), eps, window (None or n),
position (name of a `rotary_frequencies` encoding of the plan, or None; its factor on cosine and sine is applied).  Weights: "q" [2 H D, W],
"k" [2 G D, W], "v" [G Dv, W], "q_conv", "k_conv", "v_conv" [rows of each, taps], "lq1", "lk1", "lq2", "lk2" [D], "o" [W, H Dv].
The last taps-1 projections of q, k, v are a state per request (float32 [taps - 1, channels])."""
from __future__ import annotations

import math
from typing import List, Optional, Tuple

import torch

from ..config.base import ConfigError
from ..config.registry import register_part
from ..ops import functions as F
from ..ops import native
from ..ops.specs import MaskedAttentionSpec, address
from ..weights.loader import WeightSpec
from .base import CacheNeed, RunContext, SequenceCore, StateNeed
from .masked_attention import emit_masked_attention

MAPS = 2


class DifferentialAttentionMixer(SequenceCore):
    def __init__(self, spec):
        super().__init__(spec)
        p = spec.params
        self.width = int(p["hidden_size"])
        self.heads, self.kv_heads = int(p["num_heads"]), int(p["num_kv_heads"])
        self.dim, self.vdim, self.taps = int(p["head_dim"]), int(p["value_dim"]), int(p["conv"])
        self.scale, self.diff, self.eps = float(p["scale"]), float(p["diff"]), float(p["eps"])
        self.window = p.get("window")
        self.position_name, self.position = p.get("position"), None
        if self.heads % self.kv_heads:
            raise ConfigError(f"{self.heads} query heads cannot share {self.kv_heads} kv heads")
        if not (1 <= self.dim <= 1024 and 1 <= self.vdim <= 1024):
            raise ConfigError(f"key size {self.dim} / value size {self.vdim} is outside what the masked attention kernel takes (1024 / 1024)")
        if not 1 <= self.taps <= 16:
            raise ConfigError(f"a convolution of {self.taps} taps is outside what the kernel takes (1 to 16)")
        if self.window is not None and self.window <= 0:
            raise ConfigError("a window must be positive")
        self.channels = MAPS * (self.heads + self.kv_heads) * self.dim + self.kv_heads * self.vdim
        self.desc: Optional[MaskedAttentionSpec] = None

    def attach_positions(self, positions) -> None:
        if self.position_name is not None:
            self.position = positions[self.position_name]
            if getattr(self.position, "interleaved", False):
                raise ConfigError("this mixer pairs value i with value i + dims / 2; an interleaved rotation is not built there")
            if self.position.dims > self.dim:
                raise ConfigError(f"{self.position.dims} rotated values do not fit a map of {self.dim}")

    def cache_need(self) -> CacheNeed:
        return CacheNeed(self.window, self.kv_heads, MAPS * self.dim, self.vdim)

    def state_need(self) -> Optional[StateNeed]:
        return StateNeed(((self.taps - 1) * self.channels,), torch.float32) if self.taps > 1 else None

    def _rows(self) -> List[Tuple[str, int]]:
        return [("q", MAPS * self.heads * self.dim), ("k", MAPS * self.kv_heads * self.dim), ("v", self.kv_heads * self.vdim)]

    def in_roles(self) -> List[Tuple[str, int]]:
        return self._rows()

    def core_width(self) -> int:
        return self.heads * self.vdim

    def extra_weight_specs(self) -> List[WeightSpec]:
        w = self.spec.weights
        return ([WeightSpec(w[f"{role}_conv"], (rows, self.taps), "vector", ("normal", 0.3)) for role, rows in self._rows()]
                + [WeightSpec(w[role], (self.dim,), "vector", ("normal", 0.1)) for role in ("lq1", "lk1", "lq2", "lk2")])

    def kernel_modules(self, dtype) -> List[str]:
        return ["attention_masked", "short_conv"] + F.product_modules(dtype)

    def bind_core(self, tensors, rt, out_scale: float) -> None:
        w = self.spec.weights
        self.taps_weight = torch.cat([rt.vector(tensors[w[f"{role}_conv"]]).float() for role, _ in self._rows()], dim=0).contiguous()
        dot = lambda a, b: float((rt.vector(tensors[w[a]]).double() * rt.vector(tensors[w[b]]).double()).sum())
        factor = math.exp(dot("lq1", "lk1")) - math.exp(dot("lq2", "lk2")) + self.diff
        self._freq = self.position.frequencies() if self.position is not None else None
        rotated = self._freq is not None and self._freq.numel() > 0
        common = dict(heads=MAPS * self.heads, kv_heads=self.kv_heads, dim=self.dim, vdim=self.vdim, window=self.window or 0, maps=MAPS,
                      scale=self.scale, out_scale=float(out_scale) * (1.0 - self.diff), map_weight=factor, map_eps=self.eps)
        # The preparation rotates; the attention kernels take rotated queries.
        self.prepare_desc = MaskedAttentionSpec(freq=self._freq.data_ptr() if rotated else None, rot_dims=self.position.dims if rotated else 0,
                                                rot_mult=self.position.magnitude if rotated else 1.0, **common)
        self.desc = MaskedAttentionSpec(**common)

    def emit_core(self, b, proj, act, run: RunContext) -> None:
        if run.cache is None or run.cache.dtype is not proj.dtype or not run.write_cache:
            raise native.KernelError("differential attention: the cache must be the layer's own, in the activations' precision")
        q = b.temp(proj.rows, MAPS * self.heads * self.dim, proj.dtype)
        few = b.le(proj.rows, b.rt.recurrence_fused_rows)
        state = run.state
        at, stride = (state.data_ptr(), state.stride(0)) if state is not None else (None, 0)
        info = b.meta("segment_info")
        b.launch("short_conv", "mlr_conv_rotate_cache", address(self.prepare_desc), proj.ptr, proj.ld, q.ptr, q.ld, proj.is_bf16, self.taps,
                 self.taps_weight.data_ptr(), at, stride, run.cache.data_ptr(), run.cache.shape[0], b.meta("positions"), info, b.meta("segment_of_row"),
                 b.table(run.group), b.table_stride(run.group), b.page_size, b.segments, proj.rows, int(few), b.status, b.stream)
        if state is not None and not few:
            b.launch("short_conv", "mlr_short_conv_state", proj.ptr, proj.ld, proj.is_bf16, self.channels, self.taps, at, stride, info, b.segments,
                     b.stream)
        emit_masked_attention(b, self.desc, q, None, act, run)


register_part("mixer", "differential_attention", DifferentialAttentionMixer)
