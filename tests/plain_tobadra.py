"""Tobadra restated from its equations: whole sequences, no cache, no kernels, one function per mechanism.

Everything runs in the dtype of the tensors it is given (float64 in the tests).  ``config`` is the parsed
``config.json``; ``w`` maps tensor names to tensors.
"""

from __future__ import annotations

import math

import torch


def rms_norm(x, weight, eps):
    y = x / torch.sqrt((x * x).mean(-1, keepdim=True) + eps)
    return y if weight is None else y * weight


def sigmoid(z):
    return 1.0 / (1.0 + torch.exp(-z))


def silu(z):
    return z * sigmoid(z)


def gelu_tanh(z):
    return 0.5 * z * (1.0 + torch.tanh(math.sqrt(2.0 / math.pi) * (z + 0.044715 * z**3)))


def gelu_erf(z):
    return 0.5 * z * (1.0 + torch.erf(z / math.sqrt(2.0)))


def causal_conv(x, taps):
    """``y_t = sum_j taps[:, j] x_(t - K + 1 + j)`` per channel, zeros in front of the sequence.  ``x [T, C]``."""
    count = taps.shape[1]
    padded = torch.cat((torch.zeros(count - 1, x.shape[1], dtype=x.dtype), x))
    return sum(taps[:, j] * padded[j : j + x.shape[0]] for j in range(count))


def rotate(x, positions, base, dims, back=False):
    """The first ``dims`` elements of the last axis of ``x [T, H, d]``: (u, v) = elements (i, i + dims / 2) become
    (u cos a - v sin a, v cos a + u sin a) with a = p * base^(-2 i / dims) (-a with ``back``)."""
    half = dims // 2
    freq = torch.tensor([base ** (-2.0 * i / dims) for i in range(half)], dtype=x.dtype)
    angle = positions.to(x.dtype).view(-1, 1, 1) * freq * (-1.0 if back else 1.0)
    u, v = x[..., :half], x[..., half:dims]
    return torch.cat((u * torch.cos(angle) - v * torch.sin(angle), v * torch.cos(angle) + u * torch.sin(angle), x[..., dims:]), dim=-1)


def window_mask(tokens, size):
    i, j = torch.arange(tokens).view(-1, 1), torch.arange(tokens).view(1, -1)
    return (i - j >= 0) & (i - j < size)


def attention_heads(q, k, v, scale, base, size, positions=None):
    """Windowed softmax attention with values that are cached rotated by their own position and turned back by the
    query's: ``q [T, H, d]`` and ``k [T, G, d]`` are already rotated, ``v [T, G, dv]`` is not."""
    tokens, heads, _ = q.shape
    groups, vdim = k.shape[1], v.shape[2]
    positions = torch.arange(tokens) if positions is None else positions
    turned = rotate(v, positions, base, vdim)
    out = torch.zeros(tokens, heads, vdim, dtype=q.dtype)
    seen = window_mask(tokens, size)
    for h in range(heads):
        g = h // (heads // groups)
        scores = (q[:, h] @ k[:, g].T * scale).masked_fill(~seen, -math.inf)
        out[:, h] = torch.softmax(scores, dim=-1) @ turned[:, g]
    return rotate(out, positions, base, vdim, back=True)


def attention(h, w, p, m, eps):
    tokens = h.shape[0]
    positions = torch.arange(tokens)
    linear = lambda name: h @ w[p + name].T + w[p + name + ".b"]  # noqa: E731
    q = linear("q").view(tokens, m["heads"], m["dim"])
    k = linear("k").view(tokens, m["kv_heads"], m["dim"])
    v = linear("v").view(tokens, m["kv_heads"], m["vdim"])
    base, dims = m["rot"]["base"], m["rot"]["dims"]
    q, k = rotate(q, positions, base, dims), rotate(k, positions, base, dims)
    o = attention_heads(q, k, v, m["scale"], base, m["mask"]["size"])
    return o.reshape(tokens, -1) @ w[p + "o"].T + w[p + "o.b"]


def lightning_recurrence(q, k, v, decay):
    """``S_t = decay_h S_(t-1) + k_t v_t^T``, ``o_t = S_t^T q_t``; returns the outputs and the last state."""
    tokens, heads, dim = q.shape
    state = torch.zeros(heads, dim, v.shape[2], dtype=q.dtype)
    a = torch.tensor(decay, dtype=q.dtype).view(-1, 1, 1)
    out = []
    for t in range(tokens):
        state = a * state + k[t].unsqueeze(2) * v[t].unsqueeze(1)
        out.append(torch.einsum("hd,hde->he", q[t], state))
    return torch.stack(out), state


def lightning(h, w, p, m, eps):
    tokens, heads = h.shape[0], m["heads"]
    q = silu(h @ w[p + "q"].T).view(tokens, heads, m["dim"])
    k = silu(h @ w[p + "k"].T).view(tokens, heads, m["dim"])
    v = silu(h @ w[p + "v"].T).view(tokens, heads, m["vdim"])
    o, _ = lightning_recurrence(q, k, v, m["decay"])
    o = rms_norm(o.reshape(tokens, -1), w[p + "norm"], eps)  # all heads together
    return (o * sigmoid(h @ w[p + "g"].T)) @ w[p + "o"].T


def delta_recurrence(q, k, v, beta, g):
    """Per head and token: ``S <- g * S`` (rows), ``u = beta (v - S^T k)``, ``S <- S + k u^T``, ``o = S^T q``.  All
    inputs ``[T, H, ...]``; returns the outputs and the last state."""
    tokens, heads, dim = q.shape
    state = torch.zeros(heads, dim, v.shape[2], dtype=q.dtype)
    out = []
    for t in range(tokens):
        state = g[t].unsqueeze(2) * state
        u = beta[t].unsqueeze(1) * (v[t] - torch.einsum("hd,hde->he", k[t], state))
        state = state + k[t].unsqueeze(2) * u.unsqueeze(1)
        out.append(torch.einsum("hd,hde->he", q[t], state))
    return torch.stack(out), state


def delta_inputs(h, w, p, m):
    """q, k (unit, per q/k head spread over the heads), v, beta and the decays of every token."""
    tokens, heads, groups = h.shape[0], m["heads"], m["kv_heads"]
    convolved = lambda name: silu(causal_conv(h @ w[p + name].T, w[p + name + ".conv"]))  # noqa: E731
    q = convolved("q").view(tokens, groups, m["dim"])
    k = convolved("k").view(tokens, groups, m["dim"])
    v = convolved("v").view(tokens, heads, m["vdim"])
    unit = lambda x: x / torch.sqrt((x * x).sum(-1, keepdim=True) + 1e-6)  # noqa: E731
    q, k = unit(q) * m["dim"] ** -0.5, unit(k)
    q, k = q.repeat_interleave(heads // groups, dim=1), k.repeat_interleave(heads // groups, dim=1)
    beta = sigmoid(h @ w[p + "b"].T)
    z = (h @ w[p + "a1"].T) @ w[p + "a2"].T + w[p + "dt_bias"]
    softplus = torch.log1p(torch.exp(-z.abs())) + torch.clamp(z, min=0.0)
    g = torch.exp(-torch.exp(w[p + "A_log"]).view(1, heads, 1) * softplus.view(tokens, heads, m["dim"]))
    return q, k, v, beta, g


def channel_delta(h, w, p, m, eps):
    tokens = h.shape[0]
    o, _ = delta_recurrence(*delta_inputs(h, w, p, m))
    o = rms_norm(o, w[p + "norm"], eps)  # per head, one weight for all heads
    gate = sigmoid((h @ w[p + "g1"].T) @ w[p + "g2"].T)
    return (o.reshape(tokens, -1) * gate) @ w[p + "o"].T


def route(h, w, p, router, follow=None, close=0.0):
    """Chosen units ``[T, top]`` and their weights.  Softmax over all units (those that pass the input through
    included), choice by score + correction among the units of the best groups (a group is worth its largest choice
    score), weights by the score alone times the scale.

    ``follow [T, top]``: another implementation's choice, taken for a token whose own decision was won by less than
    ``close`` in choice score, whether between units or between groups; elsewhere it must agree."""
    scores = torch.softmax(h @ w[p + "router"].T, dim=-1)
    choice = scores + w[p + "correction"]
    tokens, units = choice.shape
    top, groups = router["top"], router.get("groups")
    if groups:
        per = units // groups["count"]
        worth = choice.view(tokens, groups["count"], per).amax(-1)
        order = worth.sort(dim=-1, descending=True)
        kept = torch.zeros_like(worth, dtype=torch.bool).scatter_(1, order.indices[:, : groups["keep"]], True)
        eligible = kept.repeat_interleave(per, dim=1)
    else:
        eligible, order = torch.ones_like(choice, dtype=torch.bool), None
    allowed = choice.masked_fill(~eligible, -math.inf)
    chosen = allowed.sort(dim=-1, descending=True).indices[:, :top]
    if follow is not None:
        ranked = allowed.sort(dim=-1, descending=True).values
        for t in range(tokens):
            if set(chosen[t].tolist()) == set(follow[t].tolist()):
                continue
            margin = float(ranked[t, top - 1] - ranked[t, top]) if top < units else math.inf
            if order is not None and groups["keep"] < groups["count"]:
                margin = min(margin, float(order.values[t, groups["keep"] - 1] - order.values[t, groups["keep"]]))
            assert margin <= close, f"token {t}: a choice won by {margin:.3g} went the other way"
            chosen[t] = follow[t]
    return chosen, scores.gather(1, chosen) * router.get("scale", 1.0)


def feed_forward(h, w, p, mlp, follow=None, close=0.0):
    if mlp["kind"] == "dense":
        return gelu_tanh(h @ w[p + "up"].T) @ w[p + "down"].T
    unit = lambda x, e: gelu_erf(x @ w[p + e + ".up"].T) @ w[p + e + ".down"].T  # noqa: E731
    router = mlp["router"]
    chosen, weights = route(h, w, p, router, follow, close)
    out = torch.zeros_like(h)
    for e in range(router["experts"] + router.get("identity", 0)):
        rows, place = (chosen == e).nonzero(as_tuple=True)
        if len(rows):
            y = unit(h[rows], f"e{e}") if e < router["experts"] else h[rows]
            out.index_add_(0, rows, weights[rows, place].unsqueeze(1) * y)
    if mlp.get("shared"):
        out = out + sigmoid(h @ w[p + "shared.sg"].T) * unit(h, "shared")
    return out


MIXERS = {"attention": attention, "lightning": lightning, "channel_delta": channel_delta}


def owner(config, index):
    """The layer whose tensors layer ``index`` uses."""
    return config["layers"][index].get("weights_of", index)


def layer(x, config, w, index, follow=None, close=0.0):
    entry, eps = config["layers"][index], config["norm"]["eps"]
    p = f"l{owner(config, index)}."
    h = rms_norm(x, w[p + "norm1"], eps)
    gate = sigmoid(h @ w[p + "rg1"].T + w[p + "rg1.b"])
    y = MIXERS[entry["type"]](h + causal_conv(h, w[p + "canon1"]), w, p + "mix.", entry["mixer"], eps)
    x = x + rms_norm(gate * y, w[p + "norm1b"], eps)
    if entry.get("mlp") is not None:
        h = rms_norm(x, w[p + "norm2"], eps)
        gate = sigmoid(h @ w[p + "rg2"].T + w[p + "rg2.b"])
        x = x + rms_norm(gate * feed_forward(h, w, p + "mlp.", entry["mlp"], follow, close), w[p + "norm2b"], eps)
    return x


def forward(config, w, tokens, return_layers=False, follow=None, close=0.0):
    """Logits ``[T, vocab]``.  ``follow``: layer -> the routing to follow on close calls (see :func:`route`)."""
    eps = config["norm"]["eps"]
    x = rms_norm(w["embed"][torch.as_tensor(tokens)], w["embed.norm"], eps)
    layers = []
    for index in range(len(config["layers"])):
        x = layer(x, config, w, index, None if follow is None else follow.get(index), close)
        layers.append(x)
    logits = rms_norm(x, w["final.norm"], eps) @ w["embed"].T * config.get("logit_scale", 1.0)
    return (logits, layers) if return_layers else logits
