"""What is done to the whole residual stream between two layers.

``RecallOrigin``: ``x <- W [x; x_0] + step[n]`` with ``x_0`` the embedded tokens as they entered the stream and ``n``
the number the schedule gives it (a loop of layers that share their weights begins each of its passes with it).
The stream is 32-bit; the product reads it (and ``x_0``) in the activation type and leaves a 32-bit stream, and
``step[n]`` (one row for all tokens) is left to the norm behind it to add.

``AddStep``: ``x <- x + step[n]``.  The row is left to the norm behind it too, together with what the layer in front has
left there.
"""
from __future__ import annotations

import torch

from .. import kernels as K
from .base import STREAM_STEPS, PendingNorm, StreamStep, Summed, WeightSlot
from .norm import add_pending


class RecallOrigin(StreamStep):
    graph_safe = True

    def __init__(self, *, hidden_size: int, times: int, in_tensor: str, step_tensor: str, dtype: torch.dtype,
                 device: torch.device) -> None:
        if times < 1:
            raise ValueError(f"a loop runs at least once, got {times}")
        self.hidden_size, self.times = int(hidden_size), int(times)
        self.in_tensor, self.step_tensor, self.dtype = in_tensor, step_tensor, dtype
        self.weight = torch.empty(self.hidden_size, 2 * self.hidden_size, dtype=dtype, device=device)
        self.steps = torch.empty(self.times, self.hidden_size, dtype=dtype, device=device)

    def weight_slots(self) -> list[WeightSlot]:
        return [WeightSlot(self.in_tensor, self.weight), WeightSlot(self.step_tensor, self.steps)]

    def forward(self, h, residual, origin, number, ctx):
        if residual is None:                       # ahead of every layer: the stream is the embedded tokens
            residual, h = origin, Summed(None)
        elif residual.dtype != torch.float32:      # a block in front kept its stream in the activation type
            residual = K.stream_add(residual)
        if isinstance(h, PendingNorm):             # an output that wants its own norm first
            residual, h = add_pending(residual, h)[0], Summed(None)
        pending = None if isinstance(h, Summed) else h
        both = K.stream_add_rows(residual, pending, out_dtype=self.dtype, origin=origin, keep=False)[2]
        return self.steps[number:number + 1], K.linear(both, self.weight, out_dtype=torch.float32)


class AddStep(StreamStep):
    graph_safe = True
    reads_origin = False

    def __init__(self, *, hidden_size: int, times: int, step_tensor: str, dtype: torch.dtype, device: torch.device) -> None:
        if times < 1:
            raise ValueError(f"a loop runs at least once, got {times}")
        self.hidden_size, self.times, self.step_tensor = int(hidden_size), int(times), step_tensor
        self.steps = torch.empty(self.times, self.hidden_size, dtype=dtype, device=device)

    def weight_slots(self) -> list[WeightSlot]:
        return [WeightSlot(self.step_tensor, self.steps)]

    def forward(self, h, residual, origin, number, ctx):
        row = self.steps[number:number + 1]
        if isinstance(h, PendingNorm) and h.step is None:
            return PendingNorm(h.rows, h.weight, h.eps, step=row), residual
        if residual is None:                       # ahead of every layer: the stream is the embedded tokens
            residual = h if h.dtype == torch.float32 else K.stream_add(h)
        else:
            if residual.dtype != torch.float32:    # a block in front kept its stream in the activation type
                residual = K.stream_add(residual)
            if not isinstance(h, Summed):
                residual = add_pending(residual, h)[0]
        return row, residual


STREAM_STEPS.register("recall_origin", RecallOrigin)
STREAM_STEPS.register("add_step", AddStep)

__all__ = ["AddStep", "RecallOrigin"]
