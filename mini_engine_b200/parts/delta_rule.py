"""The gated delta rule with a decay per key channel as a mixer part: a matrix state per head that is corrected, not
only added to.

From the layer's input ``h``: ``q, k`` (``qk_heads`` heads of ``dim``), ``v`` (``heads`` heads of ``vdim``) pass a short causal
convolution per channel (``taps`` columns, the last one the current token's, zeros in front of the sequence) and silu; q
and k become unit vectors per head, ``x / sqrt(sum x^2 + unit_eps)``, and q is multiplied by ``query_scale``.  Head ``h``
uses q/k head ``h // (heads / qk_heads)``.  With ``beta = sigmoid(W_b h)`` (one per head) and ``g = exp(-exp(A_h) *
softplus(W_a2 (W_a1 h) + dt_bias))`` (one per head and key channel)::

    S <- diag(g) S        u = beta (v - S^T k)        S <- S + k u^T        o = S^T q

Each head's ``o`` is divided by its root mean square over ``vdim``, multiplied by a weight ``[vdim]`` shared by the heads
and by ``sigmoid(W_g2 (W_g1 h))``, and the concatenated heads are projected by ``W_o``.

A request's state is one float32 row in its slot of the cache manager: the matrix states, head by head with the key
channels of a value column side by side (``[heads, vdim, dim]``), then the convolution's last ``taps - 1`` inputs.  Decays,
unit norms, gates of the recurrence and the recurrence are computed in 32-bit from the 32-bit sums of the projections.

Products: all projections of ``h`` run as one product on the row-concatenated weight (q, k, v, both low-rank first
factors, beta); the two second factors run as one product on a block-diagonal weight.  In bfloat16 the low-rank sums
enter it as two bfloat16 halves each (the sum rounded, and what rounding left), side by side on the reduction axis against
the same weight twice, so that the decay is formed from the 32-bit sums up to 2^-16.
"""

from __future__ import annotations

from typing import Mapping

import torch

from mini_engine_b200.csrc import ops
from mini_engine_b200.parts.base import LayerCache, Mixer, StateSpec, StepContext, register
from mini_engine_b200.parts.linear import Linear
from mini_engine_b200.weights.loader import WeightSpec


@register("mixer", "gated_delta_rule")
class GatedDeltaRule(Mixer):
    capturable = True
    # A walk over the tokens is one long kernel per layer, like the scan of the gated linear attention, with which
    # prompt steps launched as programmatic dependents were seen to stall; this mixer's steps run in plain stream order too.
    programmatic_launch = False

    def __init__(
        self,
        prefix: str,
        hidden_size: int,
        *,
        num_heads: int,
        qk_heads: int,
        head_dim: int,
        value_dim: int,
        taps: int,
        decay_rank: int,
        gate_rank: int,
        norm_eps: float,
        unit_eps: float = 1e-6,
        query_scale: float | None = None,
        names: Mapping[str, str] | None = None,
    ):
        if min(num_heads, qk_heads, head_dim, value_dim, taps, decay_rank, gate_rank) < 1 or num_heads % qk_heads:
            raise ValueError("gated_delta_rule: sizes must be positive and num_heads a multiple of qk_heads")
        if head_dim > ops.DELTA_MAX_DIM or taps > ops.MAX_CONV_TAPS:
            raise ValueError(f"gated_delta_rule takes up to {ops.DELTA_MAX_DIM} key channels per head and {ops.MAX_CONV_TAPS} taps, got {head_dim} and {taps}")
        self.hidden, self.heads, self.qk_heads, self.dim, self.vdim = hidden_size, num_heads, qk_heads, head_dim, value_dim
        self.taps, self.ranks = taps, (decay_rank, gate_rank)
        self.eps, self.unit_eps = float(norm_eps), float(unit_eps)
        self.q_scale = float(query_scale) if query_scale is not None else head_dim**-0.5
        defaults = {"q": "q_proj.weight", "k": "k_proj.weight", "v": "v_proj.weight", "q_conv": "q_conv.weight",
                    "k_conv": "k_conv.weight", "v_conv": "v_conv.weight", "beta": "b_proj.weight", "a_log": "A_log",
                    "a1": "decay_down.weight", "a2": "decay_up.weight", "dt_bias": "dt_bias", "norm": "norm.weight",
                    "g1": "gate_down.weight", "g2": "gate_up.weight", "o": "o_proj.weight"}  # fmt: skip
        self.names = {key: prefix + (names or {}).get(key, value) for key, value in defaults.items()}
        # Columns of the fused input projection, in this order.
        widths = {"q": qk_heads * head_dim, "k": qk_heads * head_dim, "v": num_heads * value_dim, "a1": decay_rank,
                  "g1": gate_rank, "beta": num_heads}  # fmt: skip
        self.columns, column = {}, 0
        for key, width in widths.items():
            self.columns[key] = column
            column += width
        self.channels = self.columns["a1"]  # of the convolution: q, k and v
        self.matrix = num_heads * head_dim * value_dim  # floats of a request's matrix states
        self.proj: Linear | None = None
        self.second: Linear | None = None  # both second factors, block-diagonal
        self.out: Linear | None = None
        self.conv: torch.Tensor | None = None
        self.norm_weight = self.a_log = self.dt_bias = None

    def state(self) -> StateSpec:
        return StateSpec((self.matrix + (self.taps - 1) * self.channels,), torch.float32)

    def weight_specs(self) -> list[WeightSpec]:
        n, keys, inner, outer = self.names, self.qk_heads * self.dim, self.heads * self.dim, self.heads * self.vdim
        small = dict(role="vector", init="small_normal")
        return [
            WeightSpec(n["q"], (keys, self.hidden)),
            WeightSpec(n["q_conv"], (keys, self.taps), **small),
            WeightSpec(n["k"], (keys, self.hidden)),
            WeightSpec(n["k_conv"], (keys, self.taps), **small),
            WeightSpec(n["v"], (outer, self.hidden)),
            WeightSpec(n["v_conv"], (outer, self.taps), **small),
            WeightSpec(n["beta"], (self.heads, self.hidden)),
            WeightSpec(n["a_log"], (self.heads,), **small),
            WeightSpec(n["a1"], (self.ranks[0], self.hidden)),
            WeightSpec(n["a2"], (inner, self.ranks[0])),
            WeightSpec(n["dt_bias"], (inner,), **small),
            WeightSpec(n["norm"], (self.vdim,), role="vector", init="ones_normal"),
            WeightSpec(n["g1"], (self.ranks[1], self.hidden)),
            WeightSpec(n["g2"], (outer, self.ranks[1])),
            WeightSpec(n["o"], (self.hidden, outer)),
        ]

    def load(self, tensors: Mapping[str, torch.Tensor]) -> None:
        n, (decay_rank, gate_rank) = self.names, self.ranks
        rows = [tensors[n[key]] for key in ("q", "k", "v", "a1", "g1", "beta")]
        count = sum(r.shape[0] for r in rows)
        if count % 4:  # rows of zeros: the sums of a token then start on 16 bytes
            rows.append(torch.zeros(4 - count % 4, self.hidden, dtype=rows[0].dtype, device=rows[0].device))
        self.proj = Linear(torch.cat(rows, dim=0).contiguous())
        a2, g2 = tensors[n["a2"]], tensors[n["g2"]]
        self.halves = 2 if a2.dtype == torch.bfloat16 else 1
        inner, outer = a2.shape[0], g2.shape[0]
        second = torch.zeros(inner + outer, self.halves * (decay_rank + gate_rank), dtype=a2.dtype, device=a2.device)
        for half in range(self.halves):
            first = half * (decay_rank + gate_rank)
            second[:inner, first : first + decay_rank] = a2
            second[inner:, first + decay_rank : first + decay_rank + gate_rank] = g2
        self.second = Linear(second)
        self.out = Linear(tensors[n["o"]])
        self.conv = torch.cat([tensors[n[key]] for key in ("q_conv", "k_conv", "v_conv")], dim=0).t().contiguous()  # [taps, channels]
        self.norm_weight, self.a_log, self.dt_bias = tensors[n["norm"]], tensors[n["a_log"]], tensors[n["dt_bias"]]

    def forward(self, h: torch.Tensor, ctx: StepContext, cache: LayerCache) -> torch.Tensor:
        tokens, heads, dim, vdim = h.shape[0], self.heads, self.dim, self.vdim
        proj = self.proj.forward(h, ctx, "delta.proj")
        low = ctx.buffer("delta.low", (tokens, self.halves * sum(self.ranks)), h.dtype)
        ops.split_halves(proj, self.columns["a1"], sum(self.ranks), low)
        second = self.second.forward(low, ctx, "delta.second")  # [decay logits | gate logits]
        qk = ctx.buffer("delta.qk", (tokens, self.qk_heads * 2 * dim), torch.float32)
        gv = ctx.buffer("delta.gv", (tokens, heads * (dim + vdim)), torch.float32)
        scalars = ctx.buffer("delta.scalars", (tokens, heads * 2), torch.float32)
        sizes = dict(heads=heads, qk_heads=self.qk_heads, dim=dim, vdim=vdim)
        ops.delta_prepare(
            proj=proj, columns=self.columns, second=second, conv=self.conv, a_log=self.a_log, dt_bias=self.dt_bias, ctx=ctx,
            state=cache.state, matrix=self.matrix, qk=qk, gv=gv, scalars=scalars, q_scale=self.q_scale, unit_eps=self.unit_eps,
            **sizes,
        )  # fmt: skip
        raw = ctx.buffer("delta.raw", (tokens, heads * vdim), torch.float32)
        ops.delta_scan(qk=qk, gv=gv, scalars=scalars, ctx=ctx, state=cache.state, out=raw, **sizes)
        gated = ctx.buffer("delta.out", (tokens, heads * vdim), ctx.dtype)
        ops.gla_finish(
            o=raw, proj=second, gate_column=heads * dim, weight=self.norm_weight, eps=self.eps, out=gated, heads=heads,
            vdim=vdim, gate="sigmoid",
        )  # fmt: skip
        return self.out.forward(gated, ctx, "delta.o")


@register("mixer", "generalized_delta_rule")
class GeneralizedDeltaRule(Mixer):
    """The delta rule with a removal rate per key channel: what the unit key ``u = k / sqrt(sum k^2 + unit_eps)`` reads of the old
    state is removed channel by channel, and the key is added as it is.  From the layer's input ``h`` (``heads`` heads of ``dim``)::

        r, k, v = W_r h, W_k h, W_v h        a = sigmoid(W_a h + b_a)
        w = exp(-decay_scale * sigmoid(W_w2 tanh(W_w1 h) + w0))          (per head and key channel, like a)
        S <- diag(w) S - (a * u) (u^T S) + k v^T        o = S^T r

    Each head's ``o`` is divided by its root mean square, multiplied by a weight ``[heads * dim]`` and by ``sigmoid(W_g h)``, and
    the concatenated heads are projected by ``W_o``.  A request's state is ``[heads, dim (values), dim (keys)]`` float32.  All
    projections of ``h`` run as one product; the tanh of the low-rank sums enters the product with ``W_w2`` as two bfloat16
    halves, as in :class:`GatedDeltaRule`."""

    capturable = True
    programmatic_launch = False  # the walk of the gated rule

    def __init__(
        self, prefix: str, hidden_size: int, *, num_heads: int, head_dim: int, decay_rank: int, norm_eps: float, decay_scale: float,
        unit_eps: float = 1e-6, names: Mapping[str, str] | None = None,
    ):  # fmt: skip
        if min(num_heads, head_dim, decay_rank) < 1 or not decay_scale > 0:
            raise ValueError("generalized_delta_rule: sizes and decay_scale must be positive")
        if head_dim > ops.DELTA_MAX_DIM:
            raise ValueError(f"generalized_delta_rule takes up to {ops.DELTA_MAX_DIM} key channels per head, got {head_dim}")
        self.hidden, self.heads, self.dim, self.rank = hidden_size, num_heads, head_dim, decay_rank
        self.eps, self.unit_eps, self.decay_scale = float(norm_eps), float(unit_eps), float(decay_scale)
        defaults = {"r": "r_proj.weight", "k": "k_proj.weight", "v": "v_proj.weight", "g": "g_proj.weight", "a": "a_proj.weight",
                    "a_bias": "a_proj.bias", "w1": "decay_down.weight", "w2": "decay_up.weight", "w0": "decay_up.bias",
                    "norm": "norm.weight", "o": "o_proj.weight"}  # fmt: skip
        self.names = {key: prefix + (names or {}).get(key, value) for key, value in defaults.items()}
        inner = num_heads * head_dim
        self.columns = {key: i * inner for i, key in enumerate(("r", "k", "v", "a", "g", "w1"))}  # of the fused input projection
        self.proj: Linear | None = None
        self.second: Linear | None = None
        self.out: Linear | None = None
        self.norm_weight = self.a_bias = self.w0 = None

    def state(self) -> StateSpec:
        return StateSpec((self.heads * self.dim * self.dim,), torch.float32)

    def weight_specs(self) -> list[WeightSpec]:
        n, inner = self.names, self.heads * self.dim
        small = dict(role="vector", init="small_normal")
        return [
            *[WeightSpec(n[key], (inner, self.hidden)) for key in ("r", "k", "v", "g", "a")],
            WeightSpec(n["a_bias"], (inner,), **small),
            WeightSpec(n["w1"], (self.rank, self.hidden)),
            WeightSpec(n["w2"], (inner, self.rank)),
            WeightSpec(n["w0"], (inner,), **small),
            WeightSpec(n["norm"], (inner,), role="vector", init="ones_normal"),
            WeightSpec(n["o"], (self.hidden, inner)),
        ]

    def load(self, tensors: Mapping[str, torch.Tensor]) -> None:
        n = self.names
        rows = [tensors[n[key]] for key in ("r", "k", "v", "a", "g", "w1")]
        count = sum(r.shape[0] for r in rows)
        if count % 4:  # rows of zeros: the sums of a token then start on 16 bytes
            rows.append(torch.zeros(4 - count % 4, self.hidden, dtype=rows[0].dtype, device=rows[0].device))
        self.proj = Linear(torch.cat(rows, dim=0).contiguous())
        self.second, self.halves = low_rank_second(tensors[n["w2"]])
        self.out = Linear(tensors[n["o"]])
        self.norm_weight, self.a_bias, self.w0 = tensors[n["norm"]], tensors[n["a_bias"]], tensors[n["w0"]]

    def forward(self, h: torch.Tensor, ctx: StepContext, cache: LayerCache) -> torch.Tensor:
        tokens, heads, dim, at = h.shape[0], self.heads, self.dim, self.columns
        proj = self.proj.forward(h, ctx, "removal.proj")
        low = ctx.buffer("removal.low", (tokens, self.halves * self.rank), h.dtype)
        ops.split_halves(proj, at["w1"], self.rank, low, activate=True)
        logits = self.second.forward(low, ctx, "removal.second")
        raw = walk_states(
            "removal", ctx, cache.state, heads, dim, dim, q=(proj, at["r"]), k=(proj, at["k"]), v=(proj, at["v"]), rate=(proj, at["a"]),
            logits=(logits, 0), decay_bias=self.w0, channel=self.a_bias, decay_scale=self.decay_scale, unit_eps=self.unit_eps,
        )  # fmt: skip
        gated = ctx.buffer("removal.out", (tokens, heads * dim), ctx.dtype)
        ops.gla_finish(
            o=raw, proj=proj, gate_column=at["g"], weight=self.norm_weight, eps=self.eps, out=gated, heads=heads, vdim=dim, gate="sigmoid"
        )
        return self.out.forward(gated, ctx, "removal.o")


def low_rank_second(weight: torch.Tensor) -> tuple[Linear, int]:
    """The product with the second factor of a low-rank projection, and how many halves its input is cut into: in bfloat16 the
    32-bit sums enter as two bfloat16 halves each, against the same weight twice."""
    halves = 2 if weight.dtype == torch.bfloat16 else 1
    return Linear(torch.cat([weight] * halves, dim=1).contiguous()), halves


# An entry of at least this many tokens runs in chunks; decoded tokens and short portions walk and keep the bits of a
# token-by-token run.
CHUNKED_MIN_TOKENS = 33


def walk_states(rule: str, ctx: StepContext, state: torch.Tensor, heads: int, dim: int, vdim: int, **inputs) -> torch.Tensor:
    """Prepare and walk a recurrence of :data:`ops.STATE_RULES`; returns the heads' outputs ``[T, heads * vdim]`` float32."""
    tokens = ctx.num_tokens
    row, numbers = ops.state_rule_floats(rule, dim, vdim)
    rows = ctx.buffer(f"{rule}.rows", (tokens, heads * row), torch.float32)
    scalars = ctx.buffer(f"{rule}.scalars", (tokens, heads * numbers), torch.float32)
    sizes = dict(heads=heads, dim=dim, vdim=vdim)
    ops.state_prepare(rule=rule, rows=rows, scalars=scalars, **{"rate": None, "unit_eps": 0.0, "decay_scale": 1.0, **inputs}, **sizes)
    raw = ctx.buffer(f"{rule}.raw", (tokens, heads * vdim), torch.float32)
    chunk_min, records = 0, None
    # a step's longest entry is known on the host
    if ctx.max_query_len >= CHUNKED_MIN_TOKENS and ops.state_chunks_support(dim, vdim, state.shape[1]):
        chunk_min = CHUNKED_MIN_TOKENS
        chunks = tokens // ops.STATE_CHUNK + ctx.num_entries
        records = ctx.workspace.growing(f"{rule}.records", (chunks, heads * ops.state_record_floats(rule, dim)), torch.float32)
    ops.state_walk(rule=rule, rows=rows, scalars=scalars, ctx=ctx, state=state, out=raw, chunk_min=chunk_min, records=records, **sizes)
    return raw
