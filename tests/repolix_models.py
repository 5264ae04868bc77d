"""Small Repolix configurations and random weights for the tests.  The configurations differ in every size and option: width, vocabulary,
layer order, one kind of mixer only, layers with and without a feed-forward; maps of 6 to 64 values with values wider and narrower, heads that
share key/value heads (up to 36 maps on one) and heads of their own; windows from 5 to 70 and none; rotations of all, some and none of a map's values,
with YaRN ramps over some, all and none of the pairs and without scaling; differences of 0 to 0.8; state sizes of 10 to 128, keys and queries
that groups of heads share, norms whose parts cut through heads; convolutions of 1 to 7 taps; routers with and without groups, identity
experts and a shared expert, from one chosen of four to eight of twenty; an eps large enough to show where it stands."""
from __future__ import annotations

import copy
import math
from typing import Dict

import torch


def _moe(ff, limit, experts, top, identity=0, groups=None, shared=None):
    router = {"experts": experts, "top": top}
    if identity:
        router["identity"] = identity
    if groups is not None:
        router["groups"] = {"count": groups[0], "keep": groups[1]}
    mlp = {"kind": "moe", "expert": {"ff": ff, "limit": limit}, "router": router}
    if shared is not None:
        mlp["shared"] = {"ff": shared[0], "limit": shared[1]}
    return mlp


def _attention(heads, kv_heads, dim, vdim, scale, diff, conv, window=None, rot=None, mlp=None):
    mixer = {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "scale": scale, "diff": diff, "conv": conv}
    if window is not None:
        mixer["mask"] = {"size": window}
    if rot is not None:
        mixer["rot"] = {"dims": rot[0], "base": rot[1]}
        if len(rot) > 2:
            mixer["rot"]["scaling"] = dict(zip(("factor", "original", "fast", "slow"), rot[2]))
    return {"type": "attention", "mixer": mixer, "mlp": mlp}


def _state(heads, groups, state, vdim, conv, norm_groups, mlp=None):
    return {"type": "mamba2", "mixer": {"heads": heads, "groups": groups, "state": state, "vdim": vdim, "conv": conv, "norm_groups": norm_groups}, "mlp": mlp}


def _delta(heads, kv_heads, dim, vdim, conv, ranks, mlp=None):
    return {"type": "channel_delta", "mixer": {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "conv": conv,
                                               "decay_rank": ranks[0], "gate_rank": ranks[1]}, "mlp": mlp}


def _model(vocab, width, eps, scale, layers):
    return {"architecture": "Repolix", "vocab": vocab, "width": width, "norm": {"eps": eps}, "embedding": {"scale": scale}, "layers": layers}


ALL = {
    # All kinds of layers, groups with identity experts among them, a window of some tokens.
    "small_a": _model(97, 48, 1e-5, 3.0, [
        _state(4, 2, 16, 12, 3, 3, _moe(24, 1.5, 6, 3, identity=3, groups=(3, 2), shared=(40, 2.0))),
        _attention(6, 3, 16, 24, 0.3, 0.3, 4, 20, (8, 100.0, (8.0, 64, 4.0, 1.0)), _moe(32, 1.0, 5, 2, identity=1, shared=(16, 0.7))),
        _delta(6, 2, 16, 24, 4, (7, 9), _moe(16, 3.0, 8, 2, groups=(4, 1)))]),
    # Sizes that miss every fast path; one tap and seven; no window, no rotation, no groups, no shared expert; layers without a feed-forward.
    "small_b": _model(130, 36, 0.05, 0.8, [
        _attention(5, 5, 6, 10, 0.4, 0.8, 1, None, (6, 50.0), _moe(10, 2.0, 4, 1)),
        _state(3, 1, 10, 7, 5, 7), _attention(3, 1, 7, 6, 0.5, 0.0, 7, 5), _delta(4, 1, 14, 6, 1, (1, 2), _moe(12, 0.5, 3, 3, identity=2)),
        _state(3, 3, 40, 9, 1, 1, _moe(20, 1.0, 7, 2, groups=(7, 3)))]),
    # Sizes the tensor cores and the wide walk take; a prompt beyond one tile of rows; more maps on a key/value head than one tile of heads.
    "small_c": _model(200, 64, 1e-6, 1.4, [
        _attention(6, 2, 32, 64, 0.2, 0.5, 3, 70, (16, 5000.0, (4.0, 96, 8.0, 2.0)), _moe(64, 2.0, 16, 8, identity=4, groups=(5, 3), shared=(96, 1.5))),
        _state(4, 2, 64, 32, 4, 4, _moe(32, 1.0, 8, 2, identity=8, groups=(2, 2))),
        _attention(18, 1, 16, 8, 0.3, 0.2, 2, 33, (16, 300.0, (32.0, 16, 1.0, 0.1))),
        _state(2, 1, 128, 16, 2, 2), _attention(2, 2, 64, 96, 0.12, 0.6, 4, None, (64, 1e4, (40.0, 4096, 32.0, 1.0)))]),
    "only_attention": _model(61, 32, 1e-5, 1.5, [_attention(2, 1, 16, 16, 0.3, 0.4, 2, 9, (16, 20.0)), _attention(4, 4, 8, 24, 0.4, 0.7, 3, None, None, _moe(16, 1.0, 4, 2, identity=2))]),
    "only_state": _model(61, 32, 1e-5, 3.5, [_state(4, 4, 32, 8, 3, 2, _moe(24, 1.0, 4, 2, shared=(8, 1.0))), _state(1, 1, 12, 20, 6, 5)]),
}


def get(name: str) -> dict:
    return copy.deepcopy(ALL[name])


def random_weights(config: dict, seed: int) -> Dict[str, torch.Tensor]:
    """bfloat16 tensors by their checkpoint names; decays between quick and nearly none, corrections that push most choices below zero."""
    g = torch.Generator().manual_seed(seed)
    W = config["width"]
    out: Dict[str, torch.Tensor] = {}

    def matrix(name, rows, cols, gain=1.0):
        out[name] = (torch.randn(rows, cols, generator=g) * gain / math.sqrt(cols)).bfloat16()

    def vector(name, n, mean=0.0, std=1.0):
        out[name] = (mean + std * torch.randn(n, generator=g)).bfloat16()

    matrix("embed", config["vocab"], W, math.sqrt(W) / config["embedding"]["scale"])
    for i, layer in enumerate(config["layers"]):
        p = f"l{i}."
        m = layer["mixer"]
        H, Dv = m["heads"], m["vdim"]
        vector(p + "norm1", W, 1.0, 0.2)
        vector(p + "ls1", W, 0.8, 0.3)
        if layer["type"] == "attention":
            D, G = m["dim"], m["kv_heads"]
            for role, n in (("q", 2 * H * D), ("k", 2 * G * D), ("v", G * Dv)):
                matrix(p + "mix." + role, n, W)
                out[p + f"mix.{role}.conv"] = (0.5 * torch.randn(n, m["conv"], generator=g)).bfloat16()
            for role in ("lq1", "lk1", "lq2", "lk2"):
                vector(p + "mix." + role, D, 0.0, 0.5 / math.sqrt(D) * 2.0)
            matrix(p + "mix.o", W, H * Dv)
        elif layer["type"] == "mamba2":
            inner, N, G = H * Dv, m["state"], m["groups"]
            channels = inner + 2 * G * N
            matrix(p + "mix.in", inner + channels + H, W)
            out[p + "mix.conv"] = (0.5 * torch.randn(channels, m["conv"], generator=g)).bfloat16()
            vector(p + "mix.conv.b", channels, 0.0, 0.3)
            vector(p + "mix.dt_bias", H, -1.0, 1.5)
            vector(p + "mix.A_log", H, -0.5, 1.0)
            vector(p + "mix.D", H, 0.5, 0.5)
            vector(p + "mix.norm", inner, 1.0, 0.2)
            matrix(p + "mix.o", W, inner)
        else:
            D, G = m["dim"], m["kv_heads"]
            for role, n in (("q", G * D), ("k", G * D), ("v", H * Dv)):
                matrix(p + "mix." + role, n, W)
                out[p + f"mix.{role}.conv"] = (0.5 * torch.randn(n, m["conv"], generator=g)).bfloat16()
            matrix(p + "mix.b", H, W, 1.5)
            vector(p + "mix.A_log", H, -1.0, 1.0)
            vector(p + "mix.dt_bias", H * D, -2.0, 1.5)
            vector(p + "mix.norm", Dv, 1.0, 0.2)
            matrix(p + "mix.a1", m["decay_rank"], W)
            matrix(p + "mix.a2", H * D, m["decay_rank"])
            matrix(p + "mix.g1", m["gate_rank"], W)
            matrix(p + "mix.g2", H * Dv, m["gate_rank"], 2.0)
            matrix(p + "mix.o", W, H * Dv)
        if layer["mlp"] is not None:
            e = layer["mlp"]
            vector(p + "norm2", W, 1.0, 0.2)
            vector(p + "ls2", W, 0.8, 0.3)
            everyone = e["router"]["experts"] + e["router"].get("identity", 0)
            matrix(p + "mlp.router", everyone, W, 2.0)
            vector(p + "mlp.correction", everyone, -0.5, 0.2)
            names = [(f"e{j}.", e["expert"]["ff"]) for j in range(e["router"]["experts"])] + ([("shared.", e["shared"]["ff"])] if e.get("shared") else [])
            for name, ff in names:
                for role, rows, cols in (("gate", ff, W), ("up", ff, W), ("down", W, ff)):
                    matrix(p + "mlp." + name + role, rows, cols, 1.5)
    vector("final.norm", W, 1.0, 0.2)
    matrix("head", config["vocab"], W)
    return out
