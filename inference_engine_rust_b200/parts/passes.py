"""What happens right before the passes of a run of layers that is executed several times."""
from __future__ import annotations

from typing import Dict, Mapping

import torch

from ..csrc import bindings as B
from ..weights.loader import TensorSpec
from .base import PassStart, Runtime, StepContext, register_part


class StepVectors(PassStart):
    """Pass t starts with x <- x + step[t] (tensor "step" [times, hidden]), and every pass but the first with x <- x + e in
    front of that, e being the embedded rows as they stood before the first block.  One kernel per pass, which also does the
    first block's norm where its arrangement offers that (`begin_rows`)."""
    graph_safe = True

    def __init__(self, spec, hidden_size: int, rt: Runtime):
        self.rt, self.hidden_size, self.times = rt, hidden_size, int(spec["times"])
        self.step = None

    def tensor_specs(self) -> Dict[str, TensorSpec]:
        return {"step": TensorSpec((self.times, self.hidden_size))}

    def load(self, tensors: Mapping[str, torch.Tensor]) -> None:
        self.step = tensors["step"].to(torch.float32).contiguous()

    def weight_bytes(self) -> int:
        return self.step.numel() * self.step.element_size()

    def _kept(self, x):
        return self.rt.workspace.take("passes.embedded", x.shape, torch.float32) if self.times > 1 else None

    def embedded(self, x, ctx: StepContext, begins_here: bool) -> None:
        # a pass that starts on these very rows keeps them itself
        if self.times > 1 and not begins_here:
            B.rows_begin(x, ctx.n_tokens, ctx.stream, keep=self._kept(x))

    def begin(self, t: int, x, ctx: StepContext, block, first: bool) -> None:
        kw = dict(step=self.step[t], e=self._kept(x) if t > 0 else None, keep=self._kept(x) if first else None)
        ctx.rows_ahead = None
        take = getattr(block, "begin_rows", None)
        if take is not None:
            take(x, ctx, **kw)
        else:
            B.rows_begin(x, ctx.n_tokens, ctx.stream, **kw)


register_part("pass", "step_vectors", StepVectors)
