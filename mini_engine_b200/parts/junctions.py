"""Steps on the residual stream in front of an entry of the execution order.

``reinjection`` opens a pass of a loop over layers: the stream and the embedding's output, side by side, go through a product,
and a learned vector of the pass is added, ``x <- W [x; x0] + step[turn]``.  The embedding's output is laid into its columns of
the product's input once per step; a pass rounds the stream (with what is pending) into the others.  The product's partial
sums and the vector then take the stream's place inside the next norm.
"""

from __future__ import annotations

from typing import Mapping

import torch

from mini_engine_b200.csrc import ops
from mini_engine_b200.parts.base import Junction, Residual, StepContext, register
from mini_engine_b200.parts.linear import Linear
from mini_engine_b200.weights.loader import WeightSpec


@register("junction", "reinjection")
class Reinjection(Junction):
    capturable = True

    def __init__(self, prefix: str, hidden_size: int, *, weight: str, step: str | None, turns: int):
        """``weight``: the product's tensor ``[hidden, 2 * hidden]``, the stream's columns first; ``step``: the vectors of the
        passes ``[turns, hidden]``, or ``None``."""
        if turns < 1:
            raise ValueError("reinjection: a loop has at least one pass")
        self.hidden, self.turns = hidden_size, int(turns)
        self.weight_name, self.step_name = prefix + weight, None if step is None else prefix + step
        self.product: Linear | None = None
        self.steps: torch.Tensor | None = None

    def weight_specs(self) -> list[WeightSpec]:
        specs = [WeightSpec(self.weight_name, (self.hidden, 2 * self.hidden))]
        if self.step_name is not None:
            specs.append(WeightSpec(self.step_name, (self.turns, self.hidden), role="vector", init="small_normal"))
        return specs

    def load(self, tensors: Mapping[str, torch.Tensor]) -> None:
        self.product = Linear(tensors[self.weight_name])
        self.steps = None if self.step_name is None else tensors[self.step_name]

    def _joined(self, ctx: StepContext) -> torch.Tensor:
        return ctx.buffer(f"junction.{self.weight_name}", (ctx.num_tokens, 2 * self.hidden), ctx.dtype)

    def begin(self, state: Residual, ctx: StepContext) -> None:
        ops.sum_rows(x=state.x, first=None, second=None, bias=None, out=self._joined(ctx), column=self.hidden)

    def forward(self, state: Residual, ctx: StepContext, turn: int) -> None:
        if not 0 <= turn < self.turns:
            raise ValueError(f"reinjection: pass {turn} of {self.turns}")
        if state.pending_scale is not None or state.pending_norm is not None or state.streams is not None:
            raise ValueError("reinjection adds plain outputs to one stream")
        joined = self._joined(ctx)
        ops.sum_rows(
            x=None if state.replaced else state.x, first=state.pending, second=state.pending_more, bias=state.pending_bias, out=joined
        )
        whole = self.product.forward(joined, ctx, f"junction.{self.weight_name}.out")
        state.replace(whole, None if self.steps is None else self.steps[turn])
