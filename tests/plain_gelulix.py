"""A plain, slow implementation of the Gelulix decoder for the tests: whole sequences, float64, no cache, no batching, one
function per mechanism, nothing shared with the package.

    x = table[token]
    layer:  x = norm1(a x + mixer(x));  with a feed-forward also  x = norm2(a x + feed_forward(x))
    logits = head . final_norm(x)

`weights` maps checkpoint names to float64 tensors; `config` is the dictionary of config.json.
"""
from __future__ import annotations

import math
from typing import Dict, List, Optional

import torch


def rms_norm(x, weight, eps):
    y = x / torch.sqrt((x * x).mean(dim=-1, keepdim=True) + eps)
    return y if weight is None else y * weight


def silu(z):
    return z * torch.sigmoid(z)


def residual_norm(x, delta, a, weight, eps):
    """The sum of the scaled stream and a sub-layer's result, normed."""
    return rms_norm(a * x + delta, weight, eps)


def channel_decay_recurrence(q, k, v, decay):
    """q, k, decay [T, H, D], v [T, H, Dv]: S <- diag(decay) S + k v^T, o = S^T q, token by token."""
    T, H, D = q.shape
    S = torch.zeros(H, D, v.shape[-1], dtype=q.dtype)
    out = []
    for t in range(T):
        S = decay[t][:, :, None] * S + k[t][:, :, None] * v[t][:, None, :]
        out.append(torch.einsum("hdv,hd->hv", S, q[t]))
    return torch.stack(out) if out else torch.zeros(0, H, v.shape[-1], dtype=q.dtype)


def gated_linear_decay(x, a1, a2, bias, tau):
    """sigmoid(a2 a1 x + bias)^(1 / tau)."""
    return torch.sigmoid((x @ a1.T) @ a2.T + bias) ** (1.0 / tau)


def gated_linear_attention(m: dict, w: Dict[str, torch.Tensor], p: str, x, eps):
    T, H, D, Dv = x.shape[0], m["heads"], m["dim"], m["vdim"]
    q = (x @ w[p + "q"].T * D ** -0.5).view(T, H, D)
    k = (x @ w[p + "k"].T).view(T, H, D)
    v = (x @ w[p + "v"].T).view(T, H, Dv)
    decay = gated_linear_decay(x, w[p + "a1"], w[p + "a2"], w[p + "a2.b"], m["tau"]).view(T, H, D)
    o = rms_norm(channel_decay_recurrence(q, k, v, decay), w[p + "norm"], eps)
    return (o.reshape(T, H * Dv) * silu(x @ w[p + "g"].T)) @ w[p + "o"].T


def causal_convolution(x, taps):
    """x [T, C], taps [C, n]: y[t, c] = sum_i taps[c, i] x[t - (n - 1) + i, c], zeros before the start, then silu."""
    T, n = x.shape[0], taps.shape[1]
    y = torch.zeros_like(x)
    for i in range(n):
        back = n - 1 - i
        if back < T:
            y[back:] += x[:T - back] * taps[:, i]
    return silu(y)


def unit(x):
    return x / torch.sqrt((x * x).sum(dim=-1, keepdim=True) + 1e-6)


def delta_recurrence(q, k, v, g, beta):
    """q, k, g [T, H, D], v [T, H, Dv], beta [T, H]: decay the rows of S, write the corrected value, read."""
    T, H, D = q.shape
    S = torch.zeros(H, D, v.shape[-1], dtype=q.dtype)
    out = []
    for t in range(T):
        S = g[t][:, :, None] * S
        u = beta[t][:, None] * (v[t] - torch.einsum("hdv,hd->hv", S, k[t]))
        S = S + k[t][:, :, None] * u[:, None, :]
        out.append(torch.einsum("hdv,hd->hv", S, q[t]))
    return torch.stack(out) if out else torch.zeros(0, H, v.shape[-1], dtype=q.dtype)


def channel_delta_decay(x, a_log, a1, a2, dt_bias, heads, dim):
    z = torch.nn.functional.softplus((x @ a1.T) @ a2.T + dt_bias, threshold=1e9).view(-1, heads, dim)
    return torch.exp(-torch.exp(a_log)[None, :, None] * z)


def channel_delta(m: dict, w: Dict[str, torch.Tensor], p: str, x, eps):
    T, H, G, D, Dv = x.shape[0], m["heads"], m["kv_heads"], m["dim"], m["vdim"]
    conv = {r: causal_convolution(x @ w[p + r].T, w[p + r + ".conv"]) for r in ("q", "k", "v")}
    q = (unit(conv["q"].view(T, G, D)) * D ** -0.5).repeat_interleave(H // G, dim=1)
    k = unit(conv["k"].view(T, G, D)).repeat_interleave(H // G, dim=1)
    v = conv["v"].view(T, H, Dv)
    beta = torch.sigmoid(x @ w[p + "b"].T)
    g = channel_delta_decay(x, w[p + "A_log"], w[p + "a1"], w[p + "a2"], w[p + "dt_bias"], H, D)
    o = rms_norm(delta_recurrence(q, k, v, g, beta), w[p + "norm"], eps)
    return (o.reshape(T, H * Dv) * torch.sigmoid((x @ w[p + "g1"].T) @ w[p + "g2"].T)) @ w[p + "o"].T


def yarn(dims: int, base: float, scaling: Optional[dict]):
    """(frequencies [dims / 2], factor on cosine and sine)."""
    plain = [base ** (-2.0 * i / dims) for i in range(dims // 2)]
    if scaling is None:
        return plain, 1.0
    turns_at = lambda turns: dims * math.log(scaling["original"] / (2.0 * math.pi * turns)) / (2.0 * math.log(base))
    lo = max(math.floor(turns_at(scaling["fast"])), 0)
    hi = min(math.ceil(turns_at(scaling["slow"])), dims - 1)
    freqs = []
    for i, f in enumerate(plain):
        ramp = min(max((i - lo) / max(hi - lo, 0.001), 0.0), 1.0)
        freqs.append(f / scaling["factor"] * ramp + f * (1.0 - ramp))
    return freqs, 0.1 * math.log(scaling["factor"]) + 1.0


def rotate_pairs(x, positions, freqs, mult):
    """x [T, heads, n]: value 2i and value 2i + 1 turn by position * freqs[i]; cosine and sine times `mult`."""
    out = x.clone()
    for i, f in enumerate(freqs):
        angle = positions.double() * f
        c, s = (torch.cos(angle) * mult)[:, None], (torch.sin(angle) * mult)[:, None]
        u, v = x[..., 2 * i], x[..., 2 * i + 1]
        out[..., 2 * i] = u * c - v * s
        out[..., 2 * i + 1] = v * c + u * s
    return out


def causal_attention(q, k, v, scale, sink):
    """q, k [T, H, D], v [T, H, Dv], sink [H]: softmax over j <= i, with exp(sink_h) more in the denominator."""
    T = q.shape[0]
    scores = torch.einsum("ihd,jhd->hij", q, k) * scale
    seen = torch.arange(T)[:, None] >= torch.arange(T)[None, :]
    scores = scores.masked_fill(~seen[None], -math.inf)
    top = torch.maximum(scores.max(dim=-1).values, sink[:, None])
    e = torch.exp(scores - top[..., None])
    weights = e / (e.sum(dim=-1) + torch.exp(sink[:, None] - top))[..., None]
    return torch.einsum("hij,jhd->ihd", weights, v)


def latent_attention(m: dict, w: Dict[str, torch.Tensor], p: str, x, eps):
    T, H, D, P, Dv, R = x.shape[0], m["heads"], m["dim"], m["rot_dim"], m["vdim"], m["kv_rank"]
    positions = torch.arange(T)
    q = (x @ w[p + "q"].T).view(T, H, D + P)
    down = x @ w[p + "dkv"].T
    latent = rms_norm(down[:, :R], w[p + "dkv.norm"], eps)
    freqs, mult = yarn(m["rot"]["dims"], m["rot"]["base"], m["rot"].get("scaling"))
    q = torch.cat([q[..., :D], rotate_pairs(q[..., D:], positions, freqs, mult)], dim=-1)
    key_part = rotate_pairs(down[:, R:].view(T, 1, P), positions, freqs, mult)
    k = torch.cat([(latent @ w[p + "uk"].T).view(T, H, D), key_part.expand(T, H, P)], dim=-1)
    v = (latent @ w[p + "uv"].T).view(T, H, Dv)
    out = causal_attention(q, k, v, m["scale"], w[p + "sink"])
    return out.reshape(T, H * Dv) @ w[p + "o"].T


def gated_feed_forward(w: Dict[str, torch.Tensor], p: str, x):
    gate, up = x @ w[p + "gate"].T + w[p + "gate.b"], x @ w[p + "up"].T + w[p + "up.b"]
    return (silu(gate) * up) @ w[p + "down"].T + w[p + "down.b"]


MIXERS = {"gla": gated_linear_attention, "channel_delta": channel_delta, "latent_attention": latent_attention}


def forward(config: dict, weights: Dict[str, torch.Tensor], tokens: List[int], layers_out: Optional[list] = None):
    """float64 logits [T, vocab]; `layers_out` collects the stream after every layer."""
    w = {name: t.double() for name, t in weights.items()}
    eps, a = config["norm"]["eps"], config["postln_alpha"]
    x = w["embed"][torch.tensor(tokens, dtype=torch.long)]
    for i, layer in enumerate(config["layers"]):
        p = f"l{i}."
        x = residual_norm(x, MIXERS[layer["type"]](layer["mixer"], w, p + "mix.", x, eps), a, w[p + "norm1"], eps)
        if layer.get("mlp") is not None:
            x = residual_norm(x, gated_feed_forward(w, p + "mlp.", x), a, w[p + "norm2"], eps)
        if layers_out is not None:
            layers_out.append(x)
    return rms_norm(x, w["final.norm"], eps) @ w["head"].T
