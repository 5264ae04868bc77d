"""A plain, slow implementation of the Repolix decoder for the tests: whole sequences, float64, no cache, no batching, one
function per mechanism, nothing shared with the package.

    x = table[token] * scale
    layer:  x += s1 * mixer(norm1(x));  with a feed-forward also  x += s2 * feed_forward(norm2(x))     (s1, s2 vectors)
    logits = head . final_norm(x)

`weights` maps checkpoint names to tensors; `config` is the dictionary of config.json.
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


def softplus(z):
    return torch.clamp(z, min=0) + torch.log1p(torch.exp(-torch.abs(z)))


def causal_convolution(x, taps, bias=None):
    """x [T, C], taps [C, n]: y[t, c] = sum_i taps[c, i] x[t - (n - 1) + i, c] (+ bias[c]), zeros before the start."""
    T, n = x.shape[0], taps.shape[1]
    y = torch.zeros_like(x)
    for i in range(n):
        back = n - 1 - i
        if back < T:
            y[back:] += x[:T - back] * taps[:, i]
    return y if bias is None else y + bias


# ----------------------------------------------------------------------------- attention
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


def rotate_halves(x, positions, freqs, mult):
    """x [T, heads, n]: value i and value i + len(freqs) turn by position * freqs[i], cosine and sine times `mult`; the rest stays."""
    out, half = x.clone(), len(freqs)
    for i, f in enumerate(freqs):
        angle = positions.double() * f
        c, s = (torch.cos(angle) * mult)[:, None], (torch.sin(angle) * mult)[:, None]
        u, v = x[..., i], x[..., i + half]
        out[..., i] = u * c - v * s
        out[..., i + half] = v * c + u * s
    return out


def windowed_attention(q, k, v, scale, window):
    """q [T, H, D], k [T, H, D], v [T, H, Dv]: softmax over the keys j <= i with i - j < window (None: all of them)."""
    T = q.shape[0]
    scores = torch.einsum("ihd,jhd->hij", q, k) * scale
    back = torch.arange(T)[:, None] - torch.arange(T)[None, :]
    seen = (back >= 0) & ((back < window) if window is not None else torch.ones_like(back, dtype=torch.bool))
    weights = torch.softmax(scores.masked_fill(~seen[None], -math.inf), dim=-1)
    return torch.einsum("hij,jhd->ihd", weights, v)


def difference_factor(w: Dict[str, torch.Tensor], p: str, diff: float):
    return torch.exp((w[p + "lq1"] * w[p + "lk1"]).sum()) - torch.exp((w[p + "lq2"] * w[p + "lk2"]).sum()) + diff


def difference(a1, a2, factor, diff, eps):
    """Two maps' outputs [T, H, Dv] to one."""
    return rms_norm(a1 - factor * a2, None, eps) * (1.0 - diff)


def differential_attention(m: dict, w: Dict[str, torch.Tensor], p: str, x, eps):
    T, H, D, Dv = x.shape[0], m["heads"], m["dim"], m["vdim"]
    G = m.get("kv_heads", H)
    conv = {r: causal_convolution(x @ w[p + r].T, w[p + r + ".conv"]) for r in ("q", "k", "v")}
    q, k, v = conv["q"].view(T, H, 2, D), conv["k"].view(T, G, 2, D), conv["v"].view(T, G, Dv)
    v = v.repeat_interleave(H // G, dim=1)
    positions = torch.arange(T)
    rot = m.get("rot")
    freqs, mult = yarn(rot["dims"], rot["base"], rot.get("scaling")) if rot else ([], 1.0)
    maps = []
    for i in range(2):
        qi = rotate_halves(q[:, :, i], positions, freqs, mult)
        ki = rotate_halves(k[:, :, i], positions, freqs, mult).repeat_interleave(H // G, dim=1)
        maps.append(windowed_attention(qi, ki, v, m["scale"], m["mask"]["size"] if m.get("mask") else None))
    o = difference(maps[0], maps[1], difference_factor(w, p, m["diff"]), m["diff"], eps)
    return o.reshape(T, H * Dv) @ w[p + "o"].T


# ----------------------------------------------------------------------------- state-space mixer
def state_space_recurrence(v, k, q, decay, step):
    """v [T, H, Dv], k, q [T, H, N], decay, step [T, H]: S <- decay S + step k v^T, y = S^T q, token by token."""
    T, H, Dv = v.shape
    S = torch.zeros(H, k.shape[-1], Dv, dtype=v.dtype)
    out = []
    for t in range(T):
        S = decay[t][:, None, None] * S + step[t][:, None, None] * k[t][:, :, None] * v[t][:, None, :]
        out.append(torch.einsum("hnv,hn->hv", S, q[t]))
    return torch.stack(out)


def state_space(m: dict, w: Dict[str, torch.Tensor], p: str, x, eps):
    T, H, Dv, N, G = x.shape[0], m["heads"], m["vdim"], m["state"], m["groups"]
    inner = H * Dv
    z, mixed, dt = torch.split(x @ w[p + "in"].T, [inner, inner + 2 * G * N, H], dim=-1)
    mixed = silu(causal_convolution(mixed, w[p + "conv"], w[p + "conv.b"]))
    v, k, q = torch.split(mixed, [inner, G * N, G * N], dim=-1)
    v = v.view(T, H, Dv)
    k, q = (u.view(T, G, N).repeat_interleave(H // G, dim=1) for u in (k, q))
    step = softplus(dt + w[p + "dt_bias"])
    y = state_space_recurrence(v, k, q, torch.exp(-torch.exp(w[p + "A_log"]) * step), step) + w[p + "D"][:, None] * v
    parts = m["norm_groups"]
    y = (y.reshape(T, inner) * silu(z)).view(T, parts, inner // parts)
    return (rms_norm(y, None, eps).reshape(T, inner) * w[p + "norm"]) @ w[p + "o"].T


# ----------------------------------------------------------------------------- delta rule
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
    return torch.stack(out)


def channel_delta(m: dict, w: Dict[str, torch.Tensor], p: str, x, eps):
    T, H, D, Dv = x.shape[0], m["heads"], m["dim"], m["vdim"]
    G = m.get("kv_heads", H)
    conv = {r: silu(causal_convolution(x @ w[p + r].T, w[p + r + ".conv"])) for r in ("q", "k", "v")}
    q = (unit(conv["q"].view(T, G, D)) * D ** -0.5).repeat_interleave(H // G, dim=1)
    k = unit(conv["k"].view(T, G, D)).repeat_interleave(H // G, dim=1)
    beta = torch.sigmoid(x @ w[p + "b"].T)
    z = softplus((x @ w[p + "a1"].T) @ w[p + "a2"].T + w[p + "dt_bias"]).view(T, H, D)
    g = torch.exp(-torch.exp(w[p + "A_log"])[None, :, None] * z)
    o = rms_norm(delta_recurrence(q, k, conv["v"].view(T, H, Dv), g, beta), w[p + "norm"], eps)
    return (o.reshape(T, H * Dv) * torch.sigmoid((x @ w[p + "g1"].T) @ w[p + "g2"].T)) @ w[p + "o"].T


# ----------------------------------------------------------------------------- routed experts
def expert(w: Dict[str, torch.Tensor], p: str, x, limit):
    g, u = x @ w[p + "gate"].T, x @ w[p + "up"].T
    if limit is not None:
        g, u = torch.clamp(g, max=limit), torch.clamp(u, -limit, limit)
    return (g * torch.sigmoid(1.702 * g) * (u + 1.0)) @ w[p + "down"].T


def choose(scores, correction, top, groups, keep):
    """The indices that one token uses: scores [E], grouped by neighbours, a group as good as its best choice."""
    choice = scores + correction
    per = len(choice) // groups
    best = [max(choice[g * per:(g + 1) * per].tolist()) for g in range(groups)]
    kept = sorted(range(groups), key=lambda g: (-best[g], g))[:keep]
    allowed = [e for g in kept for e in range(g * per, (g + 1) * per)]
    return sorted(allowed, key=lambda e: (-float(choice[e]), e))[:top]


def routed_experts(m: dict, w: Dict[str, torch.Tensor], p: str, x):
    r = m["router"]
    groups = r.get("groups") or {"count": 1, "keep": 1}
    scores = torch.softmax(x @ w[p + "router"].T, dim=-1)
    out = torch.zeros_like(x)
    for t in range(x.shape[0]):
        for e in choose(scores[t], w[p + "correction"], r["top"], groups["count"], groups["keep"]):
            y = expert(w, f"{p}e{e}.", x[t], m["expert"].get("limit")) if e < r["experts"] else x[t]
            out[t] += scores[t, e] * y
    if m.get("shared"):
        out = out + expert(w, p + "shared.", x, m["shared"].get("limit"))
    return out


MIXERS = {"attention": differential_attention, "mamba2": state_space, "channel_delta": channel_delta}


def forward(config: dict, weights: Dict[str, torch.Tensor], tokens: List[int], layers_out: Optional[list] = None):
    """float64 logits [T, vocab]; `layers_out` collects the stream after every layer."""
    w = {name: t.double() for name, t in weights.items()}
    eps = config["norm"]["eps"]
    x = w["embed"][torch.tensor(tokens, dtype=torch.long)] * config["embedding"]["scale"]
    for i, layer in enumerate(config["layers"]):
        p = f"l{i}."
        x = x + w[p + "ls1"] * MIXERS[layer["type"]](layer["mixer"], w, p + "mix.", rms_norm(x, w[p + "norm1"], eps), eps)
        if layer.get("mlp") is not None:
            x = x + w[p + "ls2"] * routed_experts(layer["mlp"], w, p + "mlp.", rms_norm(x, w[p + "norm2"], eps))
        if layers_out is not None:
            layers_out.append(x)
    return rms_norm(x, w["final.norm"], eps) @ w["head"].T
