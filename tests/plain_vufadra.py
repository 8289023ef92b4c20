"""Vufadra restated from its equations: whole sequences, no cache, no kernels, one function per mechanism.

Everything runs in the dtype of the tensors it is given (float64 in the tests).  ``config`` is the parsed
``config.json``; ``w`` maps tensor names to tensors.
"""

from __future__ import annotations

import math

import torch


def rms_norm(x, weight, eps):
    y = x / torch.sqrt((x * x).mean(-1, keepdim=True) + eps)
    return y if weight is None else y * weight


def dynamic_tanh(x, w, name):
    return torch.tanh(w[name + ".alpha"] * x) * w[name] + w[name + ".b"]


def sigmoid(z):
    return 1.0 / (1.0 + torch.exp(-z))


def silu(z):
    return z * sigmoid(z)


def gelu_tanh(z):
    return 0.5 * z * (1.0 + torch.tanh(math.sqrt(2.0 / math.pi) * (z + 0.044715 * z**3)))


def softplus(z):
    return torch.log1p(torch.exp(-z.abs())) + torch.clamp(z, min=0.0)


def previous(h):
    """Every token's predecessor, zeros in front of the first."""
    return torch.cat((torch.zeros_like(h[:1]), h[:-1]))


def mix_previous(h, share):
    return h + (previous(h) - h) * share


def embedding(tokens, config, w):
    tokens = torch.as_tensor(tokens)
    x = w["embed"][tokens]
    pairs = (config.get("embedding") or {}).get("bigram")
    if pairs:
        row = torch.full_like(tokens, pairs["buckets"])
        row[1:] = (tokens[:-1] * pairs["mul_prev"] + tokens[1:] * pairs["mul_cur"]) % pairs["buckets"]
        x = x + w["bigram"][row]
    return x


# -------------------------------------------------------------------------------- delta rule


def removal_recurrence(r, k, v, decay, rate):
    """Per head ``S <- diag(decay) S - (rate * u) (u^T S) + k v^T`` with ``u`` the unit key and both terms of the old state;
    ``o = S^T r`` of the new one.  All inputs ``[T, H, D]``; returns the outputs and the last state."""
    tokens, heads, dim = r.shape
    u = k / torch.sqrt((k * k).sum(-1, keepdim=True) + 1e-6)
    state = torch.zeros(heads, dim, v.shape[2], dtype=r.dtype)
    out = []
    for t in range(tokens):
        read = torch.einsum("hd,hde->he", u[t], state)
        state = decay[t].unsqueeze(2) * state - (rate[t] * u[t]).unsqueeze(2) * read.unsqueeze(1) + k[t].unsqueeze(2) * v[t].unsqueeze(1)
        out.append(torch.einsum("hd,hde->he", r[t], state))
    return torch.stack(out), state


def general_delta(h, w, p, m, eps):
    tokens, shape = h.shape[0], (h.shape[0], m["heads"], m["dim"])
    r, k, v = ((h @ w[p + name].T).view(shape) for name in ("r", "k", "v"))
    logits = torch.tanh(h @ w[p + "w1"].T) @ w[p + "w2"].T + w[p + "w0"]
    decay = torch.exp(-math.exp(-0.5) * sigmoid(logits)).view(shape)
    rate = sigmoid(h @ w[p + "a"].T + w[p + "a.b"]).view(shape)
    o, _ = removal_recurrence(r, k, v, decay, rate)
    o = rms_norm(o, None, eps).reshape(tokens, -1) * w[p + "norm"] * sigmoid(h @ w[p + "g"].T)
    return o @ w[p + "o"].T


# --------------------------------------------------------------------------------- attention


def frequencies(rot):
    """Frequencies of the rotation and the factor of its cosines and sines."""
    dims, base = rot["dims"], rot["base"]
    freq = [base ** (-2.0 * i / dims) for i in range(dims // 2)]
    scaling = rot.get("scaling")
    if not scaling:
        return freq, 1.0
    turn = lambda t: dims * math.log(scaling["original"] / (2.0 * math.pi * t)) / (2.0 * math.log(base))  # noqa: E731
    lo = max(math.floor(turn(scaling["fast"])), 0)
    hi = min(math.ceil(turn(scaling["slow"])), dims - 1)
    out = []
    for i, f in enumerate(freq):
        ramp = min(max((i - lo) / max(hi - lo, 0.001), 0.0), 1.0)
        out.append(f / scaling["factor"] * ramp + f * (1.0 - ramp))
    return out, 0.1 * math.log(scaling["factor"]) + 1.0


def rotate(x, positions, rot):
    """The first ``dims`` elements of the last axis of ``x [T, H, d]`` in pairs ``(i, i + dims / 2)``."""
    half = rot["dims"] // 2
    freq, factor = frequencies(rot)
    angle = positions.to(x.dtype).view(-1, 1, 1) * torch.tensor(freq, dtype=x.dtype)
    cos, sin = torch.cos(angle) * factor, torch.sin(angle) * factor
    u, v = x[..., :half], x[..., half : 2 * half]
    return torch.cat((u * cos - v * sin, v * cos + u * sin, x[..., 2 * half :]), dim=-1)


def chunk_mask(tokens, size):
    i, j = torch.arange(tokens).view(-1, 1), torch.arange(tokens).view(1, -1)
    return (j <= i) & (i // size == j // size)


def sigmoid_attention(q, k, v, scale, bias, seen):
    """Weights ``sigmoid(score + bias_h)`` of the visible keys, not normalised."""
    tokens, heads, _ = q.shape
    groups = k.shape[1]
    out = torch.zeros(tokens, heads, v.shape[2], dtype=q.dtype)
    for h in range(heads):
        g = h // (heads // groups)
        out[:, h] = (sigmoid(q[:, h] @ k[:, g].T * scale + bias[h]) * seen) @ v[:, g]
    return out


def attention(h, w, p, m, eps):
    tokens = h.shape[0]
    positions = torch.arange(tokens)
    q = rms_norm((h @ w[p + "q"].T).view(tokens, m["heads"], m["dim"]), w[p + "q.norm"], eps)
    k = rms_norm((h @ w[p + "k"].T).view(tokens, m["kv_heads"], m["dim"]), w[p + "k.norm"], eps)
    v = (h @ w[p + "v"].T).view(tokens, m["kv_heads"], m["vdim"])
    q, k = rotate(q, positions, m["rot"]), rotate(k, positions, m["rot"])
    seen = chunk_mask(tokens, m["mask"]["size"] if m.get("mask") else tokens).to(h.dtype)
    return sigmoid_attention(q, k, v, m["scale"], w[p + "pb"], seen).reshape(tokens, -1) @ w[p + "o"].T


# ------------------------------------------------------------------------------- time mixing


def bonus_recurrence(r, k, v, decay, bonus):
    """Per head ``o = (S + diag(bonus) k v^T)^T r`` of the old state, then ``S <- diag(decay) S + k v^T``."""
    tokens, heads, dim = r.shape
    state = torch.zeros(heads, dim, v.shape[2], dtype=r.dtype)
    out = []
    for t in range(tokens):
        kv = k[t].unsqueeze(2) * v[t].unsqueeze(1)
        out.append(torch.einsum("hd,hde->he", r[t], state + bonus.unsqueeze(2) * kv))
        state = decay[t].unsqueeze(2) * state + kv
    return torch.stack(out), state


def time_mixing(h, w, p, m, eps):
    tokens, shape = h.shape[0], (h.shape[0], m["heads"], m["dim"])
    mixed = {s: mix_previous(h, w[p + "mu." + s]) for s in "rkvgw"}
    r, k, v = ((mixed[s] @ w[p + s].T).view(shape) for s in "rkv")
    gate = silu(mixed["g"] @ w[p + "g"].T)
    decay = torch.exp(-torch.exp(torch.tanh(mixed["w"] @ w[p + "w1"].T) @ w[p + "w2"].T + w[p + "w0"])).view(shape)
    o, _ = bonus_recurrence(r, k, v, decay, w[p + "u"])
    return (rms_norm(o, None, eps).reshape(tokens, -1) * w[p + "norm"] * gate) @ w[p + "o"].T


def parallel(h, w, p, m, eps):
    left = rms_norm(attention(h, w, p + "left.", m["left"], eps), w[p + "left.out"], eps)
    right = rms_norm(time_mixing(h, w, p + "right.", m["right"], eps), w[p + "right.out"], eps)
    return 0.5 * (left + right)


# -------------------------------------------------------------------- gated linear recurrence


def causal_conv(x, taps, bias):
    """``y_t = bias + sum_j taps[:, j] x_(t - K + 1 + j)`` per channel, zeros in front of the sequence.  ``x [T, C]``."""
    count = taps.shape[1]
    padded = torch.cat((torch.zeros(count - 1, x.shape[1], dtype=x.dtype), x))
    return sum(taps[:, j] * padded[j : j + x.shape[0]] for j in range(count)) + bias


def channel_recurrence(log_a, driven):
    a, state, out = torch.exp(log_a), torch.zeros(driven.shape[1], dtype=driven.dtype), []
    for t in range(driven.shape[0]):
        state = a[t] * state + torch.sqrt(-torch.expm1(2.0 * log_a[t])) * driven[t]
        out.append(state)
    return torch.stack(out)


def rglru(h, w, p, m, eps):
    tokens, blocks, width = h.shape[0], m["blocks"], m["width"] // m["blocks"]
    y = gelu_tanh(h @ w[p + "y"].T + w[p + "y.b"])
    u = causal_conv(h @ w[p + "x"].T + w[p + "x.b"], w[p + "conv"], w[p + "conv.b"])
    parts = u.view(tokens, blocks, width)
    gate = lambda name: sigmoid(torch.einsum("tbi,boi->tbo", parts, w[p + name]) + w[p + name + ".b"]).reshape(tokens, -1)  # noqa: E731
    s = channel_recurrence(-8.0 * gate("ra") * softplus(w[p + "lam"]), gate("ri") * u)
    return (s * y) @ w[p + "o"].T


# ------------------------------------------------------------------------------------- model

MIXERS = {"general_delta": general_delta, "parallel": parallel, "rglru": rglru}


def feed_forward(h, w, p):
    return (silu(h @ w[p + "gate"].T) * (h @ w[p + "up"].T)) @ w[p + "down"].T


def layer(x, config, w, index):
    entry, p = config["layers"][index], f"l{index}."
    h = mix_previous(dynamic_tanh(x, w, p + "norm1"), w[p + "shift"])
    y = MIXERS[entry["type"]](h, w, p + "mix.", entry["mixer"], config["norm"]["eps"])
    if entry.get("mlp") is not None:
        y = y + feed_forward(dynamic_tanh(x, w, p + "norm2"), w, p + "mlp.")
    return x + y


def passes(config):
    """The order in which layers run: (layer, number of the pass it opens or None)."""
    count, loop = len(config["layers"]), config.get("loop")
    if not loop:
        return [(i, None) for i in range(count)]
    start, stop, times = loop["start"], loop["stop"], loop["times"]
    inner = [(i, t if i == start else None) for t in range(times) for i in range(start, stop)]
    return [(i, None) for i in range(start)] + inner + [(i, None) for i in range(stop, count)]


def forward(config, w, tokens, return_layers=False):
    """Logits ``[T, vocab]`` (and the stream behind every layer run)."""
    first = x = embedding(tokens, config, w)
    layers = []
    for index, opens in passes(config):
        if opens is not None:
            x = torch.cat((x, first), dim=-1) @ w["loop.in"].T + w["loop.step"][opens]
        x = layer(x, config, w, index)
        layers.append(x)
    logits = dynamic_tanh(x, w, "final.norm") @ w["head"].T
    return (logits, layers) if return_layers else logits
