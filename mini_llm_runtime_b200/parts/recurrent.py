"""Mixers with a matrix state per head and request (linear attention): retention with a fixed decay
per head, gated linear attention with a decay per key channel, the gated delta rule behind short convolutions with a decay per
head or per key channel, and the state-space duality mixer.  All are the kernel `mlr_linear_recurrence` (csrc/kernels/recurrence.cu) under different descriptions.

Retention:   q, k [H, D], v [H, Dv];  q, k rotated on their first values;  k *= D^(-1/2);
             S <- decay_h S + k v^T;  o = S^T q;  o / rms(o) per head, times silu(g);  result = o Wo^T.
Delta rule:  q, k [G, D] (head h uses q/k head h // (H/G)), v [H, Dv], each through a causal convolution
             over time per channel and silu;  q, k made unit vectors, q *= D^(-1/2);
             beta = sigmoid(Wb x);  g = exp(-exp(A_log) softplus(Wa x + dt_bias));
             S <- g S;  u = beta (v - S^T k);  S <- S + k u^T;  o = S^T q;
             o / rms(o) per head times a weight [Dv], times silu(Wg x);  result = o Wo^T.

The state (float32, [H, Dv, D] per request, for the delta rule followed by the last taps-1 inputs of
the convolutions) lives in the model's state slots; a new request starts from zeros.
"""
from __future__ import annotations

from typing import Dict, List, Optional, Tuple

import torch

from ..config.base import ConfigError
from ..config.registry import register_part
from ..ops import functions as F
from ..ops.specs import GATES, RecurrenceSpec, address
from ..weights.loader import WeightSpec
from .base import RunContext, SequenceCore, StateNeed, columns_of
from .rotary import plain_rotation


def emit_recurrence(b, mixer, proj, side, act, run: RunContext) -> None:
    """The recurrence of `mixer.desc` over the step's rows: q, k, v from `proj`, the rule's inputs and the gate
    from `side`, the result into `act`.  Few rows: one kernel.  Many: prepare, scan, read-out."""
    state, info = run.state, b.meta("segment_info")
    d = mixer.desc
    if b.le(proj.rows, b.rt.recurrence_fused_rows):
        # A read-out whose norm spans heads of a token cannot happen in a block that owns one head: the kernel then
        # leaves its plain float32 outputs in a buffer and the read-out is a second launch.
        plain = b.temp(proj.rows, d.heads * d.vdim, torch.float32) if d.norm_all or d.gate_first else None
        b.launch("recurrence", "mlr_linear_recurrence", address(d), proj.ptr, proj.ld, side.ptr, side.ld, proj.is_bf16,
                 act.ptr, act.ld, state.data_ptr(), state.stride(0), info, b.segments, proj.rows, plain.ptr if plain else None,
                 b.status, b.stream)
        return
    # A decay per key channel, and a gate that comes of a product of small rank, are made for all rows beforehand: by the matrix
    # product where its operand (a few columns of the projections) starts on a 16-byte border, else by a kernel of the family.
    df = gf = None
    made = 0
    if d.channel_decay:
        halves = [(d.col_a, mixer.second_decay)] + ([(d.col_gate, mixer.second_gate)] if d.gate_rank else [])
        made = int(b.rt.is_bf16 and all(at % 8 == 0 and w.shape[1] % 8 == 0 and w.shape[0] % 8 == 0 for at, w in halves) and side.ld % 8 == 0)
        if made:
            df = b.rt.linear(b, columns_of(side, d.col_a, d.decay_rank), mixer.second_decay, out_dtype=torch.float32, activation=True)
            gf = b.rt.linear(b, columns_of(side, d.col_gate, d.gate_rank), mixer.second_gate, out_dtype=torch.float32, activation=True) if d.gate_rank else None
        else:
            df = b.temp(proj.rows, d.heads * d.dim, torch.float32)
            gf = b.temp(proj.rows, d.heads * d.vdim, torch.float32) if d.gate_rank else None
    qf = b.temp(proj.rows, d.qk_heads * d.dim, torch.float32)
    kf = b.temp(proj.rows, d.qk_heads * d.dim, torch.float32)
    gates = b.temp(proj.rows, 2 * d.heads, torch.float32)
    obuf = b.temp(proj.rows, d.heads * d.vdim, torch.float32)
    b.launch("recurrence", "mlr_linear_recurrence_split", address(d), proj.ptr, proj.ld, side.ptr, side.ld, proj.is_bf16, act.ptr,
             act.ld, state.data_ptr(), state.stride(0), info, b.segments, b.meta("positions"), proj.rows, qf.ptr, kf.ptr, gates.ptr,
             obuf.ptr, df.ptr if df else None, gf.ptr if gf else None, made, b.stream)


def emit_short_conv(b, x, taps_weight: torch.Tensor, bias: Optional[torch.Tensor], state: torch.Tensor, state_offset: int):
    """The causal convolution (and SiLU) of the channels `x` into a buffer of its own (a row's other tokens read `x` meanwhile); then
    the convolution's state, the last taps - 1 inputs of every request from float `state_offset` of its slot on, moves on."""
    at, stride, info = state.data_ptr() + 4 * state_offset, state.stride(0), b.meta("segment_info")
    channels, taps = taps_weight.shape
    shift = bias.data_ptr() if bias is not None else None
    conv = b.temp(x.rows, channels, x.dtype)
    if b.le(x.rows, b.rt.recurrence_fused_rows):
        b.launch("short_conv", "mlr_short_conv_step", x.ptr, x.ld, conv.ptr, conv.ld, x.is_bf16, channels, taps, taps_weight.data_ptr(), at, stride,
                 info, b.segments, shift, b.stream)
    else:
        b.launch("short_conv", "mlr_short_conv", x.ptr, x.ld, conv.ptr, conv.ld, x.is_bf16, channels, taps, taps_weight.data_ptr(), at, stride,
                 info, b.meta("segment_of_row"), x.rows, shift, b.stream)
        b.launch("short_conv", "mlr_short_conv_state", x.ptr, x.ld, x.is_bf16, channels, taps, at, stride, info, b.segments, b.stream)
    return conv


def _check_state_size(dim: int, vdim: int) -> None:
    if not (1 <= dim <= 256 and 1 <= vdim <= 256) or (dim > 128 and vdim > 128):
        raise ConfigError(f"a state of {dim} x {vdim} per head is more than the recurrence kernel keeps in registers "
                          f"(256 x 128 or 128 x 256)")


class RetentionMixer(SequenceCore):
    """Parameters: hidden_size, num_heads, head_dim, value_dim, decay (one per head), eps (of the norm per
    head), position (name of a `rotary_frequencies` encoding, or None), gate (None | "silu" | "sigmoid").
    Weights: "q", "k" [H D, W], "v", "g" [H Dv, W], "o" [W, H Dv]."""

    def __init__(self, spec):
        super().__init__(spec)
        p = spec.params
        self.width = int(p["hidden_size"])
        self.heads, self.dim, self.vdim = int(p["num_heads"]), int(p["head_dim"]), int(p["value_dim"])
        self.decay = [float(d) for d in p["decay"]]
        self.eps = float(p["eps"])
        self.gate = p.get("gate", "silu")
        self.position_name = p.get("position")
        self.position = None
        if len(self.decay) != self.heads:
            raise ConfigError(f"{len(self.decay)} decays for {self.heads} heads")
        _check_state_size(self.dim, self.vdim)
        self.desc: Optional[RecurrenceSpec] = None

    def attach_positions(self, positions) -> None:
        if self.position_name is not None:
            self.position = plain_rotation(positions[self.position_name])
            if self.position.dims > self.dim:
                raise ConfigError(f"{self.position.dims} rotated values do not fit a head of {self.dim}")

    def state_need(self) -> StateNeed:
        return StateNeed((self.heads * self.vdim * self.dim,), torch.float32)

    def in_roles(self) -> List[Tuple[str, int]]:
        roles = [("q", self.heads * self.dim), ("k", self.heads * self.dim), ("v", self.heads * self.vdim)]
        return roles + ([("g", self.heads * self.vdim)] if self.gate else [])

    def core_width(self) -> int:
        return self.heads * self.vdim

    def kernel_modules(self, dtype) -> List[str]:
        return ["recurrence"] + F.product_modules(dtype)

    def bind_core(self, tensors, rt, out_scale: float) -> None:
        at = self.in_columns()
        freq = self.position.frequencies() if self.position is not None else None
        self._held = (freq, torch.tensor(self.decay, dtype=torch.float32, device=rt.device))
        rotate = freq is not None and freq.numel() > 0
        self.desc = RecurrenceSpec(
            freq=freq.data_ptr() if rotate else None, decay=self._held[1].data_ptr(), heads=self.heads, qk_heads=self.heads,
            dim=self.dim, vdim=self.vdim, prep=RecurrenceSpec.PREP["rotate" if rotate else None],
            rot_dims=self.position.dims if rotate else 0, rule=RecurrenceSpec.RULE["decay"], gate_kind=GATES[self.gate],
            col_q=at["q"], col_k=at["k"], col_v=at["v"], col_gate=at.get("g", 0), q_mult=1.0, k_mult=float(self.dim) ** -0.5,
            unit_eps=0.0, eps=self.eps, out_scale=float(out_scale))

    def emit_core(self, b, proj, act, run: RunContext) -> None:
        emit_recurrence(b, self, proj, proj, act, run)


class DeltaRuleMixer(SequenceCore):
    """Parameters: hidden_size, num_heads, num_qk_heads, head_dim, value_dim, conv (taps), eps.
    Weights: "q", "k" [G D, W], "v", "g" [H Dv, W], "b", "a" [H, W], "o" [W, H Dv], "q_conv", "k_conv" [G D, taps],
    "v_conv" [H Dv, taps], "A_log", "dt_bias" [H], "norm" [Dv]."""

    def __init__(self, spec):
        super().__init__(spec)
        p = spec.params
        self.width = int(p["hidden_size"])
        self.heads, self.qk_heads = int(p["num_heads"]), int(p["num_qk_heads"])
        self.dim, self.vdim, self.taps = int(p["head_dim"]), int(p["value_dim"]), int(p["conv"])
        self.eps = float(p["eps"])
        if self.heads % self.qk_heads:
            raise ConfigError(f"{self.heads} heads cannot share {self.qk_heads} q/k heads")
        if not 1 <= self.taps <= 16:
            raise ConfigError(f"a convolution of {self.taps} taps is outside what the kernel takes (1 to 16)")
        _check_state_size(self.dim, self.vdim)
        self.channels = 2 * self.qk_heads * self.dim + self.heads * self.vdim
        self.matrix_floats = self.heads * self.vdim * self.dim
        self.desc: Optional[RecurrenceSpec] = None

    def state_need(self) -> StateNeed:
        return StateNeed((self.matrix_floats + (self.taps - 1) * self.channels,), torch.float32)

    def in_roles(self) -> List[Tuple[str, int]]:
        return [("q", self.qk_heads * self.dim), ("k", self.qk_heads * self.dim), ("v", self.heads * self.vdim),
                ("g", self.heads * self.vdim), ("b", self.heads), ("a", self.heads)]

    def core_width(self) -> int:
        return self.heads * self.vdim

    def extra_weight_specs(self) -> List[WeightSpec]:
        w = self.spec.weights
        return [WeightSpec(w["q_conv"], (self.qk_heads * self.dim, self.taps), "vector", ("normal", 0.3)),
                WeightSpec(w["k_conv"], (self.qk_heads * self.dim, self.taps), "vector", ("normal", 0.3)),
                WeightSpec(w["v_conv"], (self.heads * self.vdim, self.taps), "vector", ("normal", 0.3)),
                WeightSpec(w["A_log"], (self.heads,), "vector", ("normal", 0.5)),
                WeightSpec(w["dt_bias"], (self.heads,), "vector", ("normal", 0.5)),
                WeightSpec(w["norm"], (self.vdim,), "vector", ("one_plus_normal", 0.01))]

    def kernel_modules(self, dtype) -> List[str]:
        return ["recurrence", "short_conv"] + F.product_modules(dtype)

    def bind_core(self, tensors, rt, out_scale: float) -> None:
        w = self.spec.weights
        vec = lambda role: rt.vector(tensors[w[role]]).float().contiguous()
        self.taps_weight = torch.cat([vec("q_conv"), vec("k_conv"), vec("v_conv")], dim=0).contiguous()
        self._held = (vec("A_log"), vec("dt_bias"), vec("norm"))
        at = self.in_columns()
        self._held += self._channel_weights(tensors, rt)
        # q, k, v are the first columns of the projections' output and, convolved, all columns of a buffer of
        # their own; b, a and the gate are read from the projections' output.
        self.desc = RecurrenceSpec(
            a_log=self._held[0].data_ptr(), dt_bias=self._held[1].data_ptr(), out_weight=self._held[2].data_ptr(), heads=self.heads,
            qk_heads=self.qk_heads, dim=self.dim, vdim=self.vdim, prep=RecurrenceSpec.PREP["unit"], rot_dims=0,
            rule=RecurrenceSpec.RULE["delta"], gate_kind=GATES["silu"], col_q=at["q"], col_k=at["k"], col_v=at["v"],
            col_a=at.get("a", 0), col_b=at["b"], col_gate=at.get("g", 0), q_mult=float(self.dim) ** -0.5, k_mult=1.0, unit_eps=1e-6, eps=self.eps,
            out_scale=float(out_scale))
        self._describe(at)

    def _channel_weights(self, tensors, rt) -> tuple:
        return ()

    def _describe(self, at) -> None:
        """What a form of the rule changes in `desc`."""

    def emit_core(self, b, proj, act, run: RunContext) -> None:
        # The recurrence reads q, k, v from the convolved buffer and b, a and the gate from the projections' output.
        conv = emit_short_conv(b, columns_of(proj, 0, self.channels), self.taps_weight, None, run.state, self.matrix_floats)
        emit_recurrence(b, self, conv, proj, act, run)


register_part("mixer", "retention", RetentionMixer)
register_part("mixer", "delta_rule", DeltaRuleMixer)


class LightningMixer(SequenceCore):
    """Lightning attention: linear attention with a fixed decay per head, no positions and no scale.

        q, k = silu(Wq x), silu(Wk x) [H, D];  v = silu(Wv x) [H, Dv];  S <- decay_h S + k v^T;  o = S^T q;
        all heads of a token together over their root mean square, times a weight [H Dv], times sigmoid(Wg x);  result = o Wo^T.

    Parameters: hidden_size, num_heads, head_dim, value_dim, decay (one per head), eps.  Weights: "q", "k" [H D, W],
    "v", "g" [H Dv, W], "o" [W, H Dv], "norm" [H Dv].  The state is the retention mixer's: float32 [H, Dv, D] per request."""

    def __init__(self, spec):
        super().__init__(spec)
        p = spec.params
        self.width = int(p["hidden_size"])
        self.heads, self.dim, self.vdim = int(p["num_heads"]), int(p["head_dim"]), int(p["value_dim"])
        self.decay = [float(d) for d in p["decay"]]
        self.eps = float(p["eps"])
        if len(self.decay) != self.heads:
            raise ConfigError(f"{len(self.decay)} decays for {self.heads} heads")
        _check_state_size(self.dim, self.vdim)
        self.desc: Optional[RecurrenceSpec] = None

    def state_need(self) -> StateNeed:
        return StateNeed((self.heads * self.vdim * self.dim,), torch.float32)

    def in_roles(self) -> List[Tuple[str, int]]:
        return [("q", self.heads * self.dim), ("k", self.heads * self.dim), ("v", self.heads * self.vdim), ("g", self.heads * self.vdim)]

    def core_width(self) -> int:
        return self.heads * self.vdim

    def extra_weight_specs(self) -> List[WeightSpec]:
        return [WeightSpec(self.spec.weights["norm"], (self.heads * self.vdim,), "vector", ("one_plus_normal", 0.01))]

    def kernel_modules(self, dtype) -> List[str]:
        return ["recurrence"] + F.product_modules(dtype)

    def bind_core(self, tensors, rt, out_scale: float) -> None:
        at = self.in_columns()
        self._held = (torch.tensor(self.decay, dtype=torch.float32, device=rt.device),
                      rt.vector(tensors[self.spec.weights["norm"]]).float().contiguous())
        self.desc = RecurrenceSpec(
            decay=self._held[0].data_ptr(), out_weight=self._held[1].data_ptr(), heads=self.heads, qk_heads=self.heads, dim=self.dim,
            vdim=self.vdim, prep=RecurrenceSpec.PREP[None], rot_dims=0, rule=RecurrenceSpec.RULE["decay"], gate_kind=GATES["sigmoid"],
            col_q=at["q"], col_k=at["k"], col_v=at["v"], col_gate=at["g"], in_act=RecurrenceSpec.IN_ACT["silu"], norm_all=1,
            q_mult=1.0, k_mult=1.0, unit_eps=0.0, eps=self.eps, out_scale=float(out_scale))

    def emit_core(self, b, proj, act, run: RunContext) -> None:
        emit_recurrence(b, self, proj, proj, act, run)


register_part("mixer", "lightning", LightningMixer)


RANK_LIMIT = 512


def _check_rank(rank: int, what: str) -> int:
    if not 1 <= rank <= RANK_LIMIT:
        raise ConfigError(f"a {what} of rank {rank} is outside what the recurrence kernel takes (1 to {RANK_LIMIT})")
    return rank


def _second_half(tensors, name: str, rt) -> Tuple[torch.Tensor, torch.Tensor]:
    """The second matrix of a low-rank product: [outputs, rank] for the matrix product, [rank, outputs] as the recurrence kernels read it."""
    w = rt.matrix(tensors[name]).contiguous()
    return w, w.t().contiguous()


class GatedLinearMixer(SequenceCore):
    """Gated linear attention: a decay per head and key channel, made by a product of small rank.

        q = Wq x D^(-1/2), k = Wk x [H, D];  v = Wv x [H, Dv];  alpha = sigmoid(A2 (A1 x) + a)^(1 / tau) [H, D]
        S <- diag(alpha) S + k v^T;  o = S^T q;   o / rms(o) per head times a weight [Dv], times silu(Wg x);  result = o Wo^T.

    Parameters: hidden_size, num_heads, head_dim, value_dim, tau, decay_rank (rows of A1), eps.  Weights: "q", "k" [H D, W],
    "v", "g" [H Dv, W], "a1" [rank, W], "a2" [H D, rank], "a2_bias" [H D], "norm" [Dv], "o" [W, H Dv].  The state is the
    retention mixer's: float32 [H, Dv, D] per request."""

    def __init__(self, spec):
        super().__init__(spec)
        p = spec.params
        self.width = int(p["hidden_size"])
        self.heads, self.dim, self.vdim = int(p["num_heads"]), int(p["head_dim"]), int(p["value_dim"])
        self.tau, self.eps = float(p["tau"]), float(p["eps"])
        self.rank = _check_rank(int(p["decay_rank"]), "decay")
        if self.tau <= 0:
            raise ConfigError(f"tau = {self.tau} must be positive")
        _check_state_size(self.dim, self.vdim)
        self.desc: Optional[RecurrenceSpec] = None

    def state_need(self) -> StateNeed:
        return StateNeed((self.heads * self.vdim * self.dim,), torch.float32)

    def in_roles(self) -> List[Tuple[str, int]]:
        return [("q", self.heads * self.dim), ("k", self.heads * self.dim), ("v", self.heads * self.vdim), ("g", self.heads * self.vdim),
                ("a1", self.rank)]

    def core_width(self) -> int:
        return self.heads * self.vdim

    def extra_weight_specs(self) -> List[WeightSpec]:
        w = self.spec.weights
        return [WeightSpec(w["a2"], (self.heads * self.dim, self.rank)),
                WeightSpec(w["a2_bias"], (self.heads * self.dim,), "vector", ("normal", 0.5)),
                WeightSpec(w["norm"], (self.vdim,), "vector", ("one_plus_normal", 0.01))]

    def kernel_modules(self, dtype) -> List[str]:
        return ["recurrence"] + F.product_modules(dtype)

    def bind_core(self, tensors, rt, out_scale: float) -> None:
        w = self.spec.weights
        at = self.in_columns()
        vec = lambda role: rt.vector(tensors[w[role]]).float().contiguous()
        self.second_decay, turned = _second_half(tensors, w["a2"], rt)
        self._held = (vec("a2_bias"), vec("norm"), turned)
        self.desc = RecurrenceSpec(
            dt_bias=self._held[0].data_ptr(), out_weight=self._held[1].data_ptr(), decay_w=self._held[2].data_ptr(), heads=self.heads,
            qk_heads=self.heads, dim=self.dim, vdim=self.vdim, prep=RecurrenceSpec.PREP[None], rot_dims=0, rule=RecurrenceSpec.RULE["decay"],
            gate_kind=GATES["silu"], col_q=at["q"], col_k=at["k"], col_v=at["v"], col_a=at["a1"], col_gate=at["g"],
            channel_decay=RecurrenceSpec.CHANNEL_DECAY["sigmoid_root"], decay_rank=self.rank, q_mult=float(self.dim) ** -0.5, k_mult=1.0,
            unit_eps=0.0, eps=self.eps, out_scale=float(out_scale), inv_tau=1.0 / self.tau)

    def emit_core(self, b, proj, act, run: RunContext) -> None:
        emit_recurrence(b, self, proj, proj, act, run)


register_part("mixer", "gated_linear", GatedLinearMixer)


class ChannelDeltaMixer(DeltaRuleMixer):
    """The gated delta rule with a decay per head and key channel, and a gate that is a low-rank product through a sigmoid:

        g = exp(-exp(A_log_h) softplus(A2 (A1 x) + dt_bias)) [H, D], acting on the rows of S;
        o / rms(o) per head times a weight [Dv], times sigmoid(G2 (G1 x)).

    The rest is `delta_rule`.  Further parameters: decay_rank, gate_rank (rows of A1 and G1).  Weights: "q", "k", "v", "o", "b", the three
    convolutions, "A_log" [H] and "norm" as there, "a1" [rank, W], "a2" [H D, rank], "dt_bias" [H D], "g1" [rank, W], "g2" [H Dv, rank]."""

    def __init__(self, spec):
        super().__init__(spec)
        self.decay_rank = _check_rank(int(spec.params["decay_rank"]), "decay")
        self.gate_rank = _check_rank(int(spec.params["gate_rank"]), "gate")

    def in_roles(self) -> List[Tuple[str, int]]:
        return [("q", self.qk_heads * self.dim), ("k", self.qk_heads * self.dim), ("v", self.heads * self.vdim),
                ("a1", self.decay_rank), ("g1", self.gate_rank), ("b", self.heads)]

    def extra_weight_specs(self) -> List[WeightSpec]:
        w = self.spec.weights
        specs = [s for s in super().extra_weight_specs() if s.name != w["dt_bias"]]
        return specs + [WeightSpec(w["dt_bias"], (self.heads * self.dim,), "vector", ("normal", 0.5)),
                        WeightSpec(w["a2"], (self.heads * self.dim, self.decay_rank)),
                        WeightSpec(w["g2"], (self.heads * self.vdim, self.gate_rank))]

    def _channel_weights(self, tensors, rt) -> tuple:
        w = self.spec.weights
        self.second_decay, decay = _second_half(tensors, w["a2"], rt)
        self.second_gate, gate = _second_half(tensors, w["g2"], rt)
        self._seconds = (decay, gate)
        return self._seconds

    def _describe(self, at) -> None:
        d = self.desc
        d.channel_decay, d.decay_rank, d.gate_rank = RecurrenceSpec.CHANNEL_DECAY["softplus"], self.decay_rank, self.gate_rank
        d.decay_w, d.gate_w = (t.data_ptr() for t in self._seconds)
        d.col_a, d.col_gate, d.gate_kind = at["a1"], at["g1"], GATES["sigmoid"]


register_part("mixer", "channel_delta", ChannelDeltaMixer)


class StateSpaceMixer(SequenceCore):
    """The state-space duality mixer: a state per head with a step size and a decay per token, keys and queries that groups of heads share.

        z | v | k | q | dt = Win x                   [H Dv | H Dv | G N | G N | H]
        v, k, q through a causal convolution over time per channel, a bias and silu;   dt <- softplus(dt + dt_bias)
        S <- exp(-exp(A_log_h) dt) S + dt k v^T [N, Dv];  o = S^T q + D_h v          (head h uses k and q number h // (H/G))
        o (all heads side by side) times silu(z), each of `norm_groups` equal parts over its own root mean square, times a weight [H Dv];
        result = o Wo^T

    Parameters: hidden_size, num_heads, num_groups (G), state_dim (N), value_dim (Dv), conv (taps), norm_groups, eps.  Weights: "in"
    [2 H Dv + 2 G N + H, W], "conv" [H Dv + 2 G N, taps], "conv_bias" [H Dv + 2 G N], "dt_bias", "A_log", "D" [H], "norm" [H Dv],
    "o" [W, H Dv].  The state is float32 [H, Dv, N] per request, followed by the last taps-1 inputs of the convolution."""

    def __init__(self, spec):
        super().__init__(spec)
        p = spec.params
        self.width = int(p["hidden_size"])
        self.heads, self.groups = int(p["num_heads"]), int(p["num_groups"])
        self.dim, self.vdim, self.taps = int(p["state_dim"]), int(p["value_dim"]), int(p["conv"])
        self.norm_groups, self.eps = int(p["norm_groups"]), float(p["eps"])
        self.inner = self.heads * self.vdim
        if self.heads % self.groups:
            raise ConfigError(f"{self.heads} heads cannot share {self.groups} keys and queries")
        if self.norm_groups < 1 or self.inner % self.norm_groups:
            raise ConfigError(f"{self.inner} values cannot be normed in {self.norm_groups} equal parts")
        if not 1 <= self.taps <= 16:
            raise ConfigError(f"a convolution of {self.taps} taps is outside what the kernel takes (1 to 16)")
        _check_state_size(self.dim, self.vdim)
        self.channels = self.inner + 2 * self.groups * self.dim
        self.matrix_floats = self.heads * self.vdim * self.dim
        self.desc: Optional[RecurrenceSpec] = None

    def state_need(self) -> StateNeed:
        return StateNeed((self.matrix_floats + (self.taps - 1) * self.channels,), torch.float32)

    def in_roles(self) -> List[Tuple[str, int]]:
        return [("in", self.inner + self.channels + self.heads)]

    def core_width(self) -> int:
        return self.inner

    def extra_weight_specs(self) -> List[WeightSpec]:
        w = self.spec.weights
        vector = lambda role, n, init: WeightSpec(w[role], (n,), "vector", init)
        return [WeightSpec(w["conv"], (self.channels, self.taps), "vector", ("normal", 0.3)), vector("conv_bias", self.channels, ("normal", 0.1)),
                vector("dt_bias", self.heads, ("normal", 0.5)), vector("A_log", self.heads, ("normal", 0.5)),
                vector("D", self.heads, ("one_plus_normal", 0.1)), vector("norm", self.inner, ("one_plus_normal", 0.01))]

    def kernel_modules(self, dtype) -> List[str]:
        return ["recurrence", "short_conv"] + F.product_modules(dtype)

    def bind_core(self, tensors, rt, out_scale: float) -> None:
        w = self.spec.weights
        vec = lambda role: rt.vector(tensors[w[role]]).float().contiguous()
        self.taps_weight, self.conv_bias = vec("conv"), vec("conv_bias")
        self._held = {role: vec(role) for role in ("A_log", "dt_bias", "D", "norm")}
        at = lambda role: self._held[role].data_ptr()
        self.desc = RecurrenceSpec(
            a_log=at("A_log"), dt_bias=at("dt_bias"), skip=at("D"), out_weight=at("norm"), heads=self.heads, qk_heads=self.groups, dim=self.dim,
            vdim=self.vdim, prep=RecurrenceSpec.PREP[None], rot_dims=0, rule=RecurrenceSpec.RULE["step"], gate_kind=GATES["silu"],
            col_v=0, col_k=self.inner, col_q=self.inner + self.groups * self.dim, col_gate=0, col_a=self.inner + self.channels, gate_first=1,
            norm_parts=self.norm_groups, q_mult=1.0, k_mult=1.0, unit_eps=0.0, eps=self.eps, out_scale=float(out_scale))

    def emit_core(self, b, proj, act, run: RunContext) -> None:
        conv = emit_short_conv(b, columns_of(proj, self.inner, self.channels), self.taps_weight, self.conv_bias, run.state, self.matrix_floats)
        emit_recurrence(b, self, conv, proj, act, run)


register_part("mixer", "state_space", StateSpaceMixer)
