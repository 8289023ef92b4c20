"""Time mixing as a mixer part: a matrix state per head with a decay per key channel, read before the current token enters it.

Every projection reads a mix of its own of the input ``h`` and the previous token's, ``h + (h' - h) * mu_s`` (zeros in front of the
sequence)::

    r, k, v = W_r m_r, W_k m_k, W_v m_v        gate = silu(W_g m_g)        w = exp(-exp(W_w2 tanh(W_w1 m_w) + w0))
    o = (S + diag(bonus) k v^T)^T r            S <- diag(w) S + k v^T

Each head's ``o`` is divided by its root mean square, multiplied by a weight ``[heads * dim]`` and by the gate, and the
concatenated heads are projected by ``W_o``.  A request's state is one float32 row in its slot: the matrix states ``[heads, dim
(values), dim (keys)]``, then the last ``h``.  The five mixes are one kernel; recurrence and decays are computed in 32-bit from
the 32-bit sums of the projections.
"""

from __future__ import annotations

from typing import Mapping

import torch

from mini_engine_b200.csrc import ops
from mini_engine_b200.parts.base import LayerCache, Mixer, StateSpec, StepContext, register
from mini_engine_b200.parts.delta_rule import low_rank_second, walk_states
from mini_engine_b200.parts.linear import Linear
from mini_engine_b200.weights.loader import WeightSpec

MIXES = ("r", "k", "v", "g", "w")


@register("mixer", "time_mixing")
class TimeMixing(Mixer):
    capturable = True
    programmatic_launch = False  # it shares the walk of the delta rule, whose steps run in plain stream order

    def __init__(
        self, prefix: str, hidden_size: int, *, num_heads: int, head_dim: int, decay_rank: int, norm_eps: float,
        names: Mapping[str, str] | None = None,
    ):  # fmt: skip
        if min(num_heads, head_dim, decay_rank) < 1:
            raise ValueError("time_mixing: sizes must be positive")
        if head_dim > ops.DELTA_MAX_DIM:
            raise ValueError(f"time_mixing takes up to {ops.DELTA_MAX_DIM} key channels per head, got {head_dim}")
        self.hidden, self.heads, self.dim, self.rank, self.eps = hidden_size, num_heads, head_dim, decay_rank, float(norm_eps)
        defaults = {"r": "r_proj.weight", "k": "k_proj.weight", "v": "v_proj.weight", "g": "g_proj.weight", "w1": "decay_down.weight",
                    "w2": "decay_up.weight", "w0": "decay_up.bias", "u": "bonus", "norm": "norm.weight", "o": "o_proj.weight",
                    **{f"mu_{s}": f"mix.{s}" for s in MIXES}}  # fmt: skip
        self.names = {key: prefix + (names or {}).get(key, value) for key, value in defaults.items()}
        self.matrix = num_heads * head_dim * head_dim  # floats of a request's matrix states
        self.products: dict[str, Linear] = {}
        self.second: Linear | None = None
        self.out: Linear | None = None
        self.mu: torch.Tensor | None = None
        self.norm_weight = self.w0 = self.bonus = None

    def state(self) -> StateSpec:
        return StateSpec((self.matrix + self.hidden,), torch.float32)

    def weight_specs(self) -> list[WeightSpec]:
        n, inner = self.names, self.heads * self.dim
        small = dict(role="vector", init="small_normal")
        return [
            *[WeightSpec(n[f"mu_{s}"], (self.hidden,), **small) for s in MIXES],
            *[WeightSpec(n[key], (inner, self.hidden)) for key in ("r", "k", "v", "g")],
            WeightSpec(n["w1"], (self.rank, self.hidden)),
            WeightSpec(n["w2"], (inner, self.rank)),
            WeightSpec(n["w0"], (inner,), **small),
            WeightSpec(n["u"], (self.heads, self.dim), **small),
            WeightSpec(n["norm"], (inner,), role="vector", init="ones_normal"),
            WeightSpec(n["o"], (self.hidden, inner)),
        ]

    def load(self, tensors: Mapping[str, torch.Tensor]) -> None:
        n = self.names
        self.mu = torch.stack([tensors[n[f"mu_{s}"]] for s in MIXES]).contiguous()
        self.products = {key: Linear(tensors[n[key]]) for key in ("r", "k", "v", "g", "w1")}
        self.second, self.halves = low_rank_second(tensors[n["w2"]])
        self.out = Linear(tensors[n["o"]])
        self.norm_weight, self.w0, self.bonus = tensors[n["norm"]], tensors[n["w0"]], tensors[n["u"]]

    def forward(self, h: torch.Tensor, ctx: StepContext, cache: LayerCache) -> torch.Tensor:
        tokens, heads, dim = h.shape[0], self.heads, self.dim
        flat = ctx.buffer("timemix.mixed", (tokens, len(MIXES) * self.hidden), h.dtype)
        mixed = flat.view(len(MIXES), tokens, self.hidden)
        ops.token_mix(h=h, mu=self.mu, ctx=ctx, state=cache.state, out=mixed, state_column=self.matrix)
        sums = {key: self.products[key].forward(mixed[i], ctx, f"timemix.{key}") for i, key in enumerate(("r", "k", "v", "g", "w1"))}
        low = ctx.buffer("timemix.low", (tokens, self.halves * self.rank), h.dtype)
        ops.split_halves(sums["w1"], 0, self.rank, low, activate=True)
        logits = self.second.forward(low, ctx, "timemix.second")
        raw = walk_states(
            "bonus", ctx, cache.state, heads, dim, dim, q=(sums["r"], 0), k=(sums["k"], 0), v=(sums["v"], 0), logits=(logits, 0),
            decay_bias=self.w0, channel=self.bonus,
        )  # fmt: skip
        gated = ctx.buffer("timemix.out", (tokens, heads * dim), ctx.dtype)
        ops.gla_finish(
            o=raw, proj=sums["g"], gate_column=0, weight=self.norm_weight, eps=self.eps, out=gated, heads=heads, vdim=dim, gate="silu"
        )
        return self.out.forward(gated, ctx, "timemix.o")
