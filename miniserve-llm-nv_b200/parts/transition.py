"""Transition parts: what happens to the residual stream between two layers (``LayerRun.enters`` names the runs before which a
transition acts, and which of its times in the step it is).

``reinjection``: the stream is mixed with the embedding output and receives a vector of its own each time, ``x <- W [x ; x_0] +
s_t``: ``x_0`` is the stream as the embedding left it, ``W`` of shape ``[width, 2 width]`` reads the stream first, ``s_t`` is row t of
a table with as many rows as the transition acts times in a step.  It stands before every pass of a run of layers that is
repeated with the same weights, so that a pass can tell which one it is and sees the tokens again.

How it runs: both operands lie side by side in one matrix of the compute type (``x_0`` is put there once per step; the stream
with the layer outputs that are still to be added, by one kernel each time), one product writes the new stream in float32, and
the vector is handed on (:class:`~.base.StreamVector`) to the norm that reads the stream next, which adds it in float32.
"""

from __future__ import annotations

from typing import Optional

import torch

from .. import kernels
from .base import ParamSpec, Part, StreamVector, register_transition
from .context import StepContext


@register_transition("reinjection")
class Reinjection(Part):
    def __init__(self, *, hidden_size: int, times: int, in_name: str, step_name: str) -> None:
        if hidden_size < 1 or times < 1:
            raise ValueError(f"reinjection: width {hidden_size} and {times} passes must be positive")
        self.hidden_size, self.times = int(hidden_size), int(times)
        self.in_name, self.step_name = in_name, step_name
        self.in_weight: Optional[torch.Tensor] = None
        self.steps: Optional[torch.Tensor] = None

    def param_specs(self) -> list[ParamSpec]:
        return [ParamSpec(self.in_name, (self.hidden_size, 2 * self.hidden_size)),
                ParamSpec(self.step_name, (self.times, self.hidden_size), "vector")]

    def load(self, tensors: dict[str, torch.Tensor]) -> None:
        self.in_weight = tensors[self.in_name]
        self.steps = tensors[self.step_name].float().contiguous()

    def _pair(self, residual: torch.Tensor, ctx: StepContext) -> torch.Tensor:
        return ctx.buffer(f"reinjection.{self.in_name}", (residual.shape[0], 2 * self.hidden_size), ctx.dtype)

    def remember(self, residual: torch.Tensor, ctx: StepContext) -> None:
        kernels.stream_to_columns(residual, None, self._pair(residual, ctx), self.hidden_size)

    def enter(self, residual: torch.Tensor, pending, ctx: StepContext, number: int) -> StreamVector:
        first, second = pending if isinstance(pending, tuple) else (pending, None)
        if isinstance(first, StreamVector):          # (two transitions before one layer)
            kernels.add_bias(residual, first.vector)
            first = None
        if first is not None and not isinstance(first, torch.Tensor):
            raise TypeError(f"reinjection: a stream with {type(first).__name__} still to be added is not implemented")
        pair = self._pair(residual, ctx)
        kernels.stream_to_columns(residual, first, pair, 0, second)
        kernels.linear(pair, self.in_weight, residual)
        return StreamVector(self.steps[number])
