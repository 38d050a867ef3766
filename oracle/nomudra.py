"""Plain, slow restatement of the Nomudra design on CPU tensors, one function per mechanism.

Written from the design's equations only; shares no code with the product path.  Every function works on one whole
sequence in the dtype of its inputs (float64 or float32), without a cache or a carried state.
Notation: ``T`` tokens, ``D`` model width, ``H`` heads, ``G`` key/value heads, ``dk`` query/key and ``dv`` value entries
per head, ``E`` experts with weights, ``N`` router outputs.

``weights`` maps tensor names (``l<i>.mix.o`` ...) to tensors; ``config`` is the parsed ``config.json``.  Every sublayer
has a bounded elementwise norm in front of it and another one behind it, ahead of the residual sum.
"""

from __future__ import annotations

import math

import torch


# ---- small pieces ---------------------------------------------------------------------------
def tanh_norm(x: torch.Tensor, weights, name: str) -> torch.Tensor:
    """Every entry by itself: w tanh(alpha x) + b, alpha one number."""
    return torch.tanh(x * weights[name + ".alpha"].reshape(())) * weights[name] + weights[name + ".b"]


def rms_unit(x: torch.Tensor, eps: float) -> torch.Tensor:
    """x / sqrt(mean(x^2) + eps) over the last axis."""
    return x / torch.sqrt(x.pow(2).mean(dim=-1, keepdim=True) + eps)


def log_sigmoid(z: torch.Tensor) -> torch.Tensor:
    return -(torch.log1p(torch.exp(-z.abs())) + torch.clamp(-z, min=0))


def soft_bound(z: torch.Tensor, cap: float) -> torch.Tensor:
    return cap * torch.tanh(z / cap)


# ---- chunked attention whose values are its keys ----------------------------------------------
def visible(i: int, j: int, size: int) -> bool:
    """May position i read position j: not later, and in the same block of ``size`` positions counted from 0."""
    return j <= i and i // size == j // size


def rotate(x: torch.Tensor, dims: int, base: float) -> torch.Tensor:
    """x [T, heads, d]: entries i and i + dims/2 of every head turn by position times base^(-2i/dims); the rest pass."""
    half, out = dims // 2, x.clone()
    for t in range(x.shape[0]):
        for i in range(half):
            angle = t * base ** (-2.0 * i / dims)
            c, s = math.cos(angle), math.sin(angle)
            u, v = x[t, :, i], x[t, :, i + half]
            out[t, :, i] = u * c - v * s
            out[t, :, i + half] = v * c + u * s
    return out


def chunk_attention(q, k, v, *, scale: float, size: int) -> torch.Tensor:
    """q [T, H, dk], k [T, G, dk], v [T, G, dv] -> [T, H, dv]: softmax over the visible keys."""
    T, H, _ = q.shape
    group = H // k.shape[1]
    see = torch.tensor([[visible(i, j, size) for j in range(T)] for i in range(T)])
    out = torch.zeros((T, H, v.shape[2]), dtype=q.dtype)
    for h in range(H):
        s = (q[:, h] @ k[:, h // group].t()) * scale
        out[:, h] = torch.softmax(s.masked_fill(~see, -math.inf), dim=1) @ v[:, h // group]
    return out


def attention_mixer(h, weights, p, spec) -> torch.Tensor:
    T, H, G, d = h.shape[0], spec["heads"], spec["kv_heads"], spec["dim"]
    q = (h @ weights[p + "q"].t() + weights[p + "q.b"]).view(T, H, d)
    k = (h @ weights[p + "k"].t() + weights[p + "k.b"]).view(T, G, d)
    v = k                                                              # ahead of the rotation
    if spec.get("rot"):
        q, k = (rotate(x, spec["rot"]["dims"], spec["rot"]["base"]) for x in (q, k))
    o = chunk_attention(q, k, v, scale=spec["scale"], size=spec["mask"]["size"]).reshape(T, H * d)
    o = o * torch.sigmoid(h @ weights[p + "g"].t())                    # one gate per entry of every head
    return o @ weights[p + "o"].t() + weights[p + "o.b"]


# ---- matrix memory ------------------------------------------------------------------------------
def matrix_memory(q, k, v, log_in, log_forget) -> torch.Tensor:
    """q, k [T, H, dk], v [T, H, dv], log gates [T, H] -> [T, H, dv].  The memory S [dk, dv] and the normaliser n [dk] are kept
    divided by e^m, m the running maximum of the log weights, which starts at 0."""
    T, H, dk = q.shape
    out = torch.zeros((T, H, v.shape[2]), dtype=q.dtype)
    for h in range(H):
        S, n = torch.zeros((dk, v.shape[2]), dtype=q.dtype), torch.zeros(dk, dtype=q.dtype)
        m = torch.zeros((), dtype=q.dtype)
        for t in range(T):
            f, i = log_forget[t, h], log_in[t, h]
            top = torch.maximum(f + m, i)
            keep, write = torch.exp(f + m - top), torch.exp(i - top)
            S = keep * S + write * torch.outer(k[t, h], v[t, h])
            n = keep * n + write * k[t, h]
            m = top
            size = torch.maximum((n @ q[t, h]).abs(), torch.exp(-m))
            out[t, h] = (q[t, h] @ S) / (size + 1e-6)
    return out


def matrix_memory_mixer(h, weights, p, spec, eps: float) -> torch.Tensor:
    T, H, dk, dv, cap = h.shape[0], spec["heads"], spec["dim"], spec["vdim"], spec["gate_cap"]
    proj = lambda name: h @ weights[p + name].t()
    q, k, v = proj("q").view(T, H, dk) / math.sqrt(dk), proj("k").view(T, H, dk), proj("v").view(T, H, dv)
    log_in = soft_bound(proj("i") + weights[p + "i.b"], cap)
    log_forget = log_sigmoid(soft_bound(proj("f") + weights[p + "f.b"], cap))
    o = rms_unit(matrix_memory(q, k, v, log_in, log_forget), eps).reshape(T, H * dv) * weights[p + "norm"]
    return (o * torch.sigmoid(proj("g"))) @ weights[p + "o"].t()


# ---- feed-forward -------------------------------------------------------------------------------
def clamped_swish_ff(x, gate, up, down, limit: float) -> torch.Tensor:
    g = torch.clamp(x @ gate.t(), max=limit)
    u = torch.clamp(x @ up.t(), -limit, limit)
    return (g * torch.sigmoid(1.702 * g) * (u + 1.0)) @ down.t()


def choose(scores: torch.Tensor, correction: torch.Tensor, top: int, groups=None) -> list:
    """One token's router scores [N] -> the chosen outputs, best first.  ``groups`` = {"count", "keep"}: equal runs of
    neighbours; only those whose best corrected score is among the ``keep`` best of the groups may be chosen from."""
    by = (scores + correction).tolist()
    allowed = set(range(len(by)))
    if groups:
        size = len(by) // groups["count"]
        best = {j: max(by[j * size : (j + 1) * size]) for j in range(groups["count"])}
        kept = sorted(best, key=lambda j: -best[j])[: groups["keep"]]
        allowed = {e for j in kept for e in range(j * size, (j + 1) * size)}
    return sorted(allowed, key=lambda e: -by[e])[:top]


def expert_mixture(h, weights, p, spec) -> torch.Tensor:
    r, E = spec["router"], spec["router"]["experts"]
    scores = torch.softmax(h @ weights[p + "router"].t(), dim=-1)
    y = torch.zeros_like(h)
    for t in range(h.shape[0]):
        chosen = choose(scores[t], weights[p + "correction"], r["top"], r.get("groups"))
        total = sum(scores[t, e] for e in chosen) + 1e-20
        for e in chosen:
            x = h[t : t + 1]
            if e < E:                                                   # the outputs past E hand their input on
                x = clamped_swish_ff(x, *(weights[f"{p}e{e}.{n}"] for n in ("gate", "up", "down")), spec["expert"]["limit"])
            y[t] = y[t] + scores[t, e] / total * x[0]
    if spec.get("shared"):
        s = clamped_swish_ff(h, *(weights[f"{p}shared.{n}"] for n in ("gate", "up", "down")), spec["shared"]["limit"])
        y = y + torch.sigmoid(h @ weights[p + "shared.sg"].t()) * s
    return y


# ---- the stack ------------------------------------------------------------------------------------
def layer_forward(x, weights, config, i: int) -> torch.Tensor:
    spec, p = config["layers"][i], f"l{i}."
    h = tanh_norm(x, weights, p + "norm1")
    if spec["type"] == "attention":
        y = attention_mixer(h, weights, p + "mix.", spec["mixer"])
    elif spec["type"] == "mlstm":
        y = matrix_memory_mixer(h, weights, p + "mix.", spec["mixer"], config["norm"]["eps"])
    else:
        raise ValueError(spec["type"])
    x = x + tanh_norm(y, weights, p + "norm1b")
    if spec.get("mlp"):
        if spec["mlp"]["kind"] != "moe":
            raise ValueError(spec["mlp"]["kind"])
        y = expert_mixture(tanh_norm(x, weights, p + "norm2"), weights, p + "mlp.", spec["mlp"])
        x = x + tanh_norm(y, weights, p + "norm2b")
    return x


def forward(ids, weights, config, dtype=torch.float64, tap: list | None = None) -> torch.Tensor:
    """ids: list of token ids -> logits [T, vocab]; ``tap`` receives the residual sum after every layer."""
    weights = {n: (t.to(dtype) if t.is_floating_point() else t) for n, t in weights.items()}
    x = tanh_norm(weights["embed"][torch.tensor(list(ids))], weights, "embed.norm")
    for i in range(len(config["layers"])):
        x = layer_forward(x, weights, config, i)
        if tap is not None:
            tap.append(x)
    return tanh_norm(x, weights, "final.norm") @ weights["head"].t()


def greedy(ids, weights, config, new_tokens: int, dtype=torch.float64) -> list:
    ids, out = list(ids), []
    for _ in range(new_tokens):
        nxt = int(forward(ids, weights, config, dtype)[-1].argmax())
        out.append(nxt)
        ids.append(nxt)
    return out
