"""Step inputs: parts that run once per step on the embedded rows, before the first block."""
from __future__ import annotations

from typing import Dict, Mapping

import torch

from ..cache import StateRequest
from ..csrc import bindings as B
from ..weights.loader import TensorSpec
from .base import Runtime, StepContext, StepInput, part_class, register_part


class EmbedNorm(StepInput):
    """A norm on the embedded rows, in place (spec: "norm" = the norm's own spec).  Its tensors: "norm"
    (the norm's weight) and "norm.<local>" for the norm's other tensors (a bias "norm.b")."""
    graph_safe = True

    def __init__(self, spec, hidden_size: int, vocab_size: int, rt: Runtime):
        ns = spec["norm"]
        self.norm = part_class("norm", ns.kind)(ns, hidden_size, rt)

    def _names(self) -> Dict[str, str]:
        return {local: "norm" if local == "weight" else "norm." + local for local in self.norm.tensor_specs()}

    def tensor_specs(self) -> Dict[str, TensorSpec]:
        specs = self.norm.tensor_specs()
        return {name: specs[local] for local, name in self._names().items()}

    def load(self, tensors: Mapping[str, torch.Tensor]) -> None:
        self.norm.load({local: tensors[name] for local, name in self._names().items()})

    def weight_bytes(self) -> int:
        return sum(t.numel() * t.element_size() for t in (self.norm.weight, getattr(self.norm, "bias", None)) if t is not None)

    def prepare(self, tokens, x, ctx: StepContext) -> None:
        self.norm.forward(x, x, ctx, rows=ctx.n_tokens)


class PairEmbedding(StepInput):
    """Adds to every embedded row a row of a second table, chosen by a hash of the token and the one in front of it:
    row (previous * mul_prev + token * mul_cur) mod buckets, or the table's last row (number `buckets`) for a sequence's
    first token.  Its tensor: `tensor_name` [buckets + 1, hidden].  State per sequence: the last token.  The kernel gathers
    both rows and writes the sum in one pass."""
    graph_safe = True
    embeds = True

    def __init__(self, spec, hidden_size: int, vocab_size: int, rt: Runtime):
        self.rt, self.hidden_size = rt, hidden_size
        self.buckets, self.mul_prev, self.mul_cur = int(spec["buckets"]), int(spec["mul_prev"]), int(spec["mul_cur"])
        self.name = spec.get("tensor_name", "pairs")
        self.table = None

    def tensor_specs(self) -> Dict[str, TensorSpec]:
        return {self.name: TensorSpec((self.buckets + 1, self.hidden_size))}

    def load(self, tensors: Mapping[str, torch.Tensor]) -> None:
        self.table = tensors[self.name].contiguous()

    def cache_request(self) -> StateRequest:
        return StateRequest((1,), torch.int32)

    def embed(self, table, tokens, x, scale: float, ctx: StepContext) -> None:
        B.embed_pairs(table, self.table, tokens, x, scale, self.buckets, self.mul_prev, self.mul_cur, ctx.input_view.state,
                      ctx.batch, self.rt.err, ctx.stream)


register_part("input", "embed_norm", EmbedNorm)
register_part("input", "pair_embedding", PairEmbedding)
