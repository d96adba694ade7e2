"""Dense feed-forward without a gate: y = act(x W_up^T) W_down^T, added to the residual; act by the spec's `activation`
("gelu": the exact form with erf).  The activation is the first product's epilogue."""
from __future__ import annotations

from typing import Dict, Mapping

import torch

from ..csrc import bindings as B
from ..weights.loader import TensorSpec
from .base import FeedForward, Runtime, StepContext, register_part
from .linear import Linear


class MLP(FeedForward):
    graph_safe = True

    def __init__(self, spec, rt: Runtime):
        self.rt = rt
        self.hidden_size = int(spec["hidden_size"])
        self.intermediate_size = int(spec["intermediate_size"])
        self.epilogue = B.epilogue(spec.get("activation", "gelu"))
        self.names = tuple(spec.get("tensor_names", ("up", "down")))
        self.up = self.down = None

    def tensor_specs(self) -> Dict[str, TensorSpec]:
        h, i = self.hidden_size, self.intermediate_size
        up, down = self.names
        return {up: TensorSpec((i, h)), down: TensorSpec((h, i))}

    def load(self, tensors: Mapping[str, torch.Tensor]) -> None:
        up, down = self.names
        self.up, self.down = Linear(tensors[up], self.rt), Linear(tensors[down], self.rt)

    def weight_bytes(self) -> int:
        return self.up.nbytes() + self.down.nbytes()

    def forward(self, xn, residual, ctx: StepContext) -> None:
        T = ctx.n_tokens
        act = self.rt.workspace.take("ffn.act", (T, self.intermediate_size), self.rt.dtype)
        self.up.apply(xn, act, T, ctx.stream, epilogue=self.epilogue)
        self.down.apply(act, residual, T, ctx.stream, add_residual=True, ctx=ctx)


register_part("ffn", "mlp", MLP)
