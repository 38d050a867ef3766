"""Plain, slow restatement of the Zalazen design on CPU tensors, one function per mechanism.

Written from the design's equations only; shares no code with the product path.  Every function works on one whole
sequence in the dtype of its inputs (float64 or float32), without a cache or a carried state.
Notation: ``T`` tokens, ``D`` model width, ``H`` query heads, ``G`` key/value heads, ``dk`` query/key and ``dv`` value
entries per head.

``weights`` maps tensor names (``l<i>.mix.o`` ...) to tensors; ``config`` is the parsed ``config.json``.  Every layer adds
a windowed attention and a gated feed-forward, each behind a norm of its own, to the residual sum.
"""

from __future__ import annotations

import math

import torch


# ---- small pieces ---------------------------------------------------------------------------
def rms_unit(x: torch.Tensor, eps: float) -> torch.Tensor:
    """x / sqrt(mean(x^2) + eps) over the last axis."""
    return x / torch.sqrt(x.pow(2).mean(dim=-1, keepdim=True) + eps)


def silu(z):
    return z * torch.sigmoid(z)


# ---- embedding --------------------------------------------------------------------------------
def bigram_row(before, token: int, *, mul_prev: int, mul_cur: int, buckets: int) -> int:
    """Row of the pair table for ``token`` after ``before`` (None: the sequence starts with ``token``)."""
    return buckets if before is None else (before * mul_prev + token * mul_cur) % buckets


def embed(ids, weights, config) -> torch.Tensor:
    spec = config["embedding"]
    rows = []
    for t, token in enumerate(ids):
        x = weights["embed"][token] * spec["scale"]
        if spec.get("bigram"):
            x = x + weights["bigram"][bigram_row(ids[t - 1] if t else None, token, **spec["bigram"])]
        rows.append(x)
    return torch.stack(rows)


# ---- positions --------------------------------------------------------------------------------
def frequencies(rot: dict):
    """-> (one frequency per rotated pair, the factor on cos and sin)."""
    dims, base, scaling = rot["dims"], rot["base"], rot.get("scaling")
    plain = [base ** (-2.0 * i / dims) for i in range(dims // 2)]
    if not scaling:
        return plain, 1.0
    at = lambda turns: dims * math.log(scaling["original"] / (2 * math.pi * turns)) / (2 * math.log(base))
    lo, hi = max(math.floor(at(scaling["fast"])), 0), min(math.ceil(at(scaling["slow"])), dims - 1)
    out = []
    for i, f in enumerate(plain):
        ramp = min(max((i - lo) / max(hi - lo, 0.001), 0.0), 1.0)
        out.append(f / scaling["factor"] * ramp + f * (1.0 - ramp))
    return out, 0.1 * math.log(scaling["factor"]) + 1.0


def rotate(x: torch.Tensor, rot: dict) -> torch.Tensor:
    """x [T, heads, d]: entries i and i + dims/2 of every head turn by position times frequency i; entries from dims up pass."""
    half = rot["dims"] // 2
    freqs, gain = frequencies(rot)
    out = x.clone()
    for t in range(x.shape[0]):
        for i in range(half):
            c, s = math.cos(t * freqs[i]) * gain, math.sin(t * freqs[i]) * gain
            u, v = x[t, :, i], x[t, :, i + half]
            out[t, :, i] = u * c - v * s
            out[t, :, i + half] = v * c + u * s
    return out


# ---- attention --------------------------------------------------------------------------------
def visible(i: int, j: int, size: int, keep_first: int) -> bool:
    """May position i read position j: the last ``size`` positions up to its own, and the sequence's first ``keep_first``."""
    return j <= i and (i - j < size or j < keep_first)


def sink_window_attention(q, k, v, sink, *, scale: float, size: int, keep_first: int) -> torch.Tensor:
    """q [T, H, dk], k [T, G, dk], v [T, G, dv], sink [H]: softmax over the visible keys, exp(sink) added to its denominator."""
    T, H, _ = q.shape
    group = H // k.shape[1]
    see = torch.tensor([[visible(i, j, size, keep_first) for j in range(T)] for i in range(T)])
    out = torch.zeros((T, H, v.shape[2]), dtype=q.dtype)
    for h in range(H):
        s = (q[:, h] @ k[:, h // group].t()) * scale
        s = s.masked_fill(~see, -math.inf)
        m = torch.maximum(s.max(dim=1, keepdim=True).values, sink[h])
        e = torch.exp(s - m)
        out[:, h] = (e / (e.sum(dim=1, keepdim=True) + torch.exp(sink[h] - m))) @ v[:, h // group]
    return out


def keys_values(h, weights, prefix, spec, *, eps):
    """What a layer with projections of its own caches: normed, rotated keys [T, G, dk] and values [T, G, dv]."""
    T, G = h.shape[0], spec["kv_heads"]
    k = rms_unit(h @ weights[prefix + "k"].t(), eps) * weights[prefix + "k.norm"]       # the whole projection is one row
    return rotate(k.view(T, G, spec["dim"]), spec["rot"]), (h @ weights[prefix + "v"].t()).view(T, G, spec["vdim"])


def attention_mixer(h, weights, prefix, spec, kv, *, eps) -> torch.Tensor:
    T, H = h.shape[0], spec["heads"]
    q = rms_unit(h @ weights[prefix + "q"].t(), eps) * weights[prefix + "q.norm"]
    q = rotate(q.view(T, H, spec["dim"]), spec["rot"])
    o = sink_window_attention(q, kv[0], kv[1], weights[prefix + "sink"], scale=spec["scale"], size=spec["mask"]["size"],
                              keep_first=spec["mask"]["keep_first"])
    o = o * torch.sigmoid(h @ weights[prefix + "g"].t())[:, :, None]
    return o.reshape(T, H * spec["vdim"]) @ weights[prefix + "o"].t()


# ---- feed-forward -------------------------------------------------------------------------------
def gated_ff(h, weights, prefix) -> torch.Tensor:
    return (silu(h @ weights[prefix + "gate"].t()) * (h @ weights[prefix + "up"].t())) @ weights[prefix + "down"].t()


# ---- the stack ------------------------------------------------------------------------------------
def layer_forward(x, weights, config, i: int, cached: dict) -> torch.Tensor:
    """``cached``: keys and values of the layers before, by layer number; this layer's join them if it has its own."""
    spec, eps, p = config["layers"][i], config["norm"]["eps"], f"l{i}."
    if spec["type"] != "attention":
        raise ValueError(spec["type"])
    m = spec["mixer"]
    h1 = rms_unit(x, eps) * weights[p + "norm1"]
    source = m.get("kv_from")
    if source is None:
        cached[i] = keys_values(h1, weights, p + "mix.", m, eps=eps)
        source = i
    y = attention_mixer(h1, weights, p + "mix.", m, cached[source], eps=eps)
    if spec.get("mlp"):
        if spec["mlp"]["kind"] != "dense":
            raise ValueError(spec["mlp"]["kind"])
        y = y + gated_ff(rms_unit(x, eps) * weights[p + "norm2"], weights, p + "mlp.")
    return x + y


def forward(ids, weights, config, dtype=torch.float64, tap: list | None = None) -> torch.Tensor:
    """ids: list of token ids -> logits [T, vocab]; ``tap`` receives the residual sum after every layer."""
    weights = {n: (t.to(dtype) if t.is_floating_point() else t) for n, t in weights.items()}
    x, cached = embed(list(ids), weights, config), {}
    for i in range(len(config["layers"])):
        x = layer_forward(x, weights, config, i, cached)
        if tap is not None:
            tap.append(x)
    return (rms_unit(x, config["norm"]["eps"]) * weights["final.norm"]) @ weights["head"].t()


def greedy(ids, weights, config, new_tokens: int, dtype=torch.float64) -> list:
    ids, out = list(ids), []
    for _ in range(new_tokens):
        nxt = int(forward(ids, weights, config, dtype)[-1].argmax())
        out.append(nxt)
        ids.append(nxt)
    return out
