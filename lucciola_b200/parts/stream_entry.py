"""What stands in front of every pass of a looped run of layers: the residual stream mixed with the embedding's output by
one linear map, plus a vector of the pass,

    x <- W [x ; x0] + step[t]          W [width, 2 width] (x first), step [passes, width], x0 the embedding's output

W x0 is the same in every pass and is formed once a step.  In the bfloat16 engine the stream enters its half of the
product in two bfloat16 parts, x = hi + lo (16 significant bits), as two rows of one product that reads the weights once;
the 32-bit sums of both, W x0 and the pass's vector are added by the norm that reads the stream next (Pending).  x0 is a row
of the table and needs no second part."""
from __future__ import annotations

from typing import Callable, Optional

import torch

from .. import ops
from .base import ParamSpec, Part, Pending, Runtime
from .norm import pending_terms


class StreamEntry(Part):
    recordable = True

    def __init__(self, rt: Runtime, map_name: str, step_name: str, width: int, passes: int):
        self.rt, self.map_name, self.step_name, self.width, self.passes = rt, map_name, step_name, width, passes
        self.w_stream: torch.Tensor | None = None          # [width, width]
        self.w_embedding: torch.Tensor | None = None       # [width, width]
        self.steps: torch.Tensor | None = None             # [passes, width] float32

    def param_specs(self) -> list[ParamSpec]:
        return [ParamSpec(self.map_name, (self.width, 2 * self.width)), ParamSpec(self.step_name, (self.passes, self.width))]

    def bind(self, get: Callable[[str], torch.Tensor]) -> None:
        w = get(self.map_name)
        self.w_stream, self.w_embedding = w[:, :self.width].contiguous(), w[:, self.width:].contiguous()
        self.steps = get(self.step_name).to(torch.float32).contiguous()

    def _product(self, x: torch.Tensor, w: torch.Tensor) -> torch.Tensor:
        y = self.rt.empty((x.shape[0], self.width), torch.float32)
        ops.linear(y, x, w, self.rt.stream, fast=self.rt.fast_kernels)
        return y

    def embedding_half(self, x0: torch.Tensor) -> torch.Tensor:
        """W x0, float32 [T, width], from the embedding's output in the activation type."""
        return self._product(x0, self.w_embedding)

    def forward(self, residual: torch.Tensor, pending: Optional[Pending], from_embedding: torch.Tensor, t: int) -> tuple[torch.Tensor, Pending]:
        """The stream as pass t starts with it: (a float32 matrix, what is still to be added to it)."""
        terms = pending_terms(pending) if pending is not None else {}
        T = residual.shape[0]
        if self.rt.act_dtype == torch.float32:
            if pending is not None:
                ops.stream_norm(residual, self.rt.stream, **terms)
            return self._product(residual, self.w_stream), Pending(plain=(from_embedding,), vector=self.steps[t])
        parts = self.rt.empty((2 * T, self.width))
        ops.stream_norm(residual, self.rt.stream, parts=(parts[:T], parts[T:]), **terms)
        y = self._product(parts, self.w_stream)
        return y[:T], Pending(plain=(y[T:], from_embedding), vector=self.steps[t])
