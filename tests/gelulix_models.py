"""Small Gelulix configurations and random weights for the tests.  The configurations differ in every size and option: width,
vocabulary, layer order, one kind of mixer only, layers with and without a feed-forward; state heads of 10 to 128 key and 6 to 72 value
channels; q/k heads that several heads share and heads of their own; convolutions of 1, 2, 4 and 7 taps; decay and gate ranks from 1 up
that differ from one another; latents and rotated parts of sizes that do and do not suit the tensor cores, values wider and narrower than
keys; YaRN frequencies whose ramp covers some, all and none of the pairs, and no scaling; factors on the stream of 1, above and below;
tau of 1 and more; an eps large enough to show where it stands."""
from __future__ import annotations

import copy
import math
from typing import Dict

import torch


def _gla(heads, dim, vdim, tau, rank, ff=None):
    return {"type": "gla", "mixer": {"heads": heads, "dim": dim, "vdim": vdim, "tau": tau, "decay_rank": rank}, "mlp": _dense(ff)}


def _delta(heads, kv_heads, dim, vdim, conv, ranks, ff=None):
    return {"type": "channel_delta", "mixer": {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "conv": conv,
                                               "decay_rank": ranks[0], "gate_rank": ranks[1]}, "mlp": _dense(ff)}


def _latent(heads, dim, rot_dim, vdim, rank, scale, base, scaling=None, ff=None):
    rot = {"base": base, "dims": rot_dim}
    if scaling is not None:
        rot["scaling"] = dict(zip(("factor", "original", "fast", "slow"), scaling))
    return {"type": "latent_attention", "mixer": {"heads": heads, "dim": dim, "rot_dim": rot_dim, "vdim": vdim, "kv_rank": rank, "scale": scale,
                                                  "rot": rot}, "mlp": _dense(ff)}


def _dense(ff):
    return {"kind": "dense", "ff": ff} if ff is not None else None


def _model(vocab, width, eps, alpha, layers):
    return {"architecture": "Gelulix", "vocab": vocab, "width": width, "norm": {"eps": eps}, "postln_alpha": alpha, "layers": layers}


ALL = {
    # Shared q/k heads, a feed-forward behind every kind of mixer, a ramp over some of the pairs.
    "small_a": _model(97, 48, 1e-5, 2.0, [
        _delta(6, 2, 16, 24, 4, (7, 9), ff=40), _latent(3, 12, 8, 20, 24, 0.3, 100.0, (8.0, 64, 4.0, 1.0), ff=56),
        _gla(3, 24, 16, 4.0, 5, ff=24), _gla(2, 32, 8, 1.0, 12)]),
    # Sizes that miss every fast path; one tap and seven; no scaling; a factor below one; an eps that shows.
    "small_b": _model(130, 36, 0.05, 0.9, [
        _latent(5, 10, 6, 6, 14, 0.4, 50.0), _gla(3, 10, 6, 16.0, 3), _delta(5, 5, 6, 10, 1, (2, 11), ff=28),
        _delta(4, 1, 14, 6, 7, (1, 1)), _gla(1, 40, 72, 8.0, 9, ff=12)]),
    # Sizes the tensor cores and the wide walk take; a prompt beyond one tile of rows.
    "small_c": _model(200, 64, 1e-6, 1.4, [
        _gla(2, 64, 32, 12.0, 16, ff=64), _delta(2, 1, 128, 16, 2, (16, 8)), _latent(4, 32, 32, 64, 96, 0.15, 5000.0, (4.0, 96, 8.0, 2.0), ff=96),
        _delta(4, 2, 32, 64, 4, (8, 24)), _latent(2, 64, 64, 16, 64, 0.1, 300.0, (32.0, 16, 1.0, 0.1))]),
    "only_gla": _model(61, 32, 1e-5, 1.5, [_gla(2, 16, 12, 6.0, 4), _gla(4, 96, 8, 2.0, 8, ff=16)]),
    "only_delta": _model(61, 32, 1e-5, 3.5, [_delta(4, 2, 12, 16, 3, (4, 6), ff=24), _delta(1, 1, 16, 40, 4, (8, 8))]),
    "only_latent": _model(61, 32, 1e-5, 1.2, [_latent(2, 16, 8, 16, 24, 0.3, 20.0, (3.0, 32, 2.0, 0.5)), _latent(4, 8, 16, 24, 272, 0.2, 1000.0, ff=16)]),
}


def get(name: str) -> dict:
    return copy.deepcopy(ALL[name])


def random_weights(config: dict, seed: int) -> Dict[str, torch.Tensor]:
    """bfloat16 tensors by their checkpoint names; decays between quick and nearly none, sinks that take a visible share."""
    g = torch.Generator().manual_seed(seed)
    W = config["width"]
    out: Dict[str, torch.Tensor] = {}

    def matrix(name, rows, cols, gain=1.0):
        out[name] = (torch.randn(rows, cols, generator=g) * gain / math.sqrt(cols)).bfloat16()

    def vector(name, n, mean=0.0, std=1.0):
        out[name] = (mean + std * torch.randn(n, generator=g)).bfloat16()

    matrix("embed", config["vocab"], W, math.sqrt(W))
    for i, layer in enumerate(config["layers"]):
        p = f"l{i}."
        m = layer["mixer"]
        H, D, Dv = m["heads"], m["dim"], m["vdim"]
        vector(p + "norm1", W, 1.0, 0.2)
        if layer["type"] == "gla":
            for role, n in (("q", H * D), ("k", H * D), ("v", H * Dv), ("g", H * Dv)):
                matrix(p + "mix." + role, n, W)
            matrix(p + "mix.a1", m["decay_rank"], W)
            matrix(p + "mix.a2", H * D, m["decay_rank"])
            vector(p + "mix.a2.b", H * D, 2.0, 2.0)
            vector(p + "mix.norm", Dv, 1.0, 0.2)
            matrix(p + "mix.o", W, H * Dv)
        elif layer["type"] == "channel_delta":
            G = m["kv_heads"]
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
        else:
            R, P = m["kv_rank"], m["rot_dim"]
            matrix(p + "mix.q", H * (D + P), W)
            matrix(p + "mix.dkv", R + P, W)
            vector(p + "mix.dkv.norm", R, 1.0, 0.2)
            matrix(p + "mix.uk", H * D, R)
            matrix(p + "mix.uv", H * Dv, R, 2.0)
            vector(p + "mix.sink", H, 1.0, 1.0)
            matrix(p + "mix.o", W, H * Dv)
        if layer["mlp"] is not None:
            ff = layer["mlp"]["ff"]
            vector(p + "norm2", W, 1.0, 0.2)
            for role, rows, cols in (("gate", ff, W), ("up", ff, W), ("down", W, ff)):
                matrix(p + "mlp." + role, rows, cols)
                vector(p + f"mlp.{role}.b", rows, 0.0, 0.3)
    vector("final.norm", W, 1.0, 0.2)
    matrix("head", config["vocab"], W)
    return out
