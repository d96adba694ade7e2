"""A model assembled from a `ModelSpec`: embedding table, one block per layer, final norm,
output head; and its forward pass over the tokens of one step.

Reference: the layer loop and the last-row logits of src/engine/runtime.rs:14-33,76-116,
embedding of src/engine/embed.rs:104-138.  Differences on purpose: the loop follows the
spec's schedule (a list of layer executions), and logits are produced for any wanted rows.
"""
from __future__ import annotations

from typing import Dict, List, Mapping, Optional

import torch

from ..cache import CacheRequest
from ..config.specs import ModelSpec
from ..csrc import bindings as B
from ..parts.base import Runtime, StepContext, first_norm_request_of, part_class
from ..weights.loader import (RandomSource, TensorSpec, WeightError, check_source, fetch_many)


class Model:
    def __init__(self, spec: ModelSpec, rt: Runtime):
        spec.validate()
        self.spec = spec
        self.rt = rt
        self.blocks = []
        self._layer_parts = []       # (norm1, mixer, norm2, ffn) per layer
        self._cut_askers = None
        h = spec.hidden_size
        self._extra_norms = []       # {role: norm} per layer (arrangements with more than two norms)
        for ls in spec.layers:
            norm_cls = part_class("norm", ls.norm.kind)
            norm1 = norm_cls(ls.norm, h, rt)
            # an arrangement whose feed-forward reads the first norm names no second one (`ffn_norm_name` empty)
            norm2 = norm_cls(ls.norm, h, rt) if ls.ffn is not None and ls.ffn_norm_name else None
            mixer = part_class("mixer", ls.mixer.kind)(ls.mixer, rt)
            ffn = part_class("ffn", ls.ffn.kind)(ls.ffn, rt) if ls.ffn is not None else None
            extra = {role: part_class("norm", ns.kind)(ns, h, rt) for role, (ns, _) in ls.extra_norms.items()}
            kw = {"extra_norms": extra} if extra else {}
            block = part_class("block", ls.block.kind)(ls, norm1, mixer, norm2, ffn, rt, **kw)
            self._layer_parts.append((norm1, mixer, norm2, ffn))
            self._extra_norms.append(extra)
            self.blocks.append(block)
        self.final_norm = part_class("norm", spec.final_norm.kind)(spec.final_norm, h, rt)
        self.embedding: Optional[torch.Tensor] = None
        self.lm_head = part_class("head", spec.head.kind)(spec.head, h, spec.vocab_size, rt)
        self.inputs = [(part_class("input", ps.kind)(ps, h, spec.vocab_size, rt), prefix) for ps, prefix in spec.inputs]
        self.passes, self._passes_prefix = None, ""
        if spec.passes is not None:
            ps, self._passes_prefix = spec.passes
            self.passes = part_class("pass", ps.kind)(ps, h, rt)
        self.loaded = False
        # called after every scheduled layer with (its position, the residual rows or streams, the step's
        # context): for looking at the residual between layers; runs inside the step, so it must launch on
        # the step's stream and turns captured graphs off for as long as it is set
        self.after_block = None
        self.ignored_tensors: List[str] = []
        self.notes: List[str] = []       # what loading decided on its own (tied head, ignored tensors)

    # ---- weights ------------------------------------------------------------------------
    @staticmethod
    def _norm_names(norm, weight_name: str) -> Dict[str, str]:
        """Tensor name of each of a norm's tensors: its "weight" under the name the spec gives, any
        other (a bias "b", say) under that name + "." + its local name."""
        return {local: weight_name if local == "weight" else f"{weight_name}.{local}" for local in norm.tensor_specs()}

    @staticmethod
    def _block_specs(block) -> Dict[str, TensorSpec]:
        """Tensors of a block arrangement's own (most have none, and need not say so)."""
        specs = getattr(block, "tensor_specs", None)
        return specs() if specs is not None else {}

    def _norm_specs(self, norm, weight_name: str) -> Dict[str, TensorSpec]:
        specs = norm.tensor_specs()
        return {name: specs[local] for local, name in self._norm_names(norm, weight_name).items()}

    def expected_tensors(self) -> Dict[str, TensorSpec]:
        """Every tensor name the model reads from a folder, with its shape."""
        spec = self.spec
        out: Dict[str, TensorSpec] = {
            spec.embedding_name: TensorSpec((spec.vocab_size, spec.hidden_size)),
        }
        out.update(self._norm_specs(self.final_norm, spec.final_norm_name))
        if spec.lm_head_name is not None:
            out[spec.lm_head_name] = self.lm_head.tensor_specs()["weight"]
        for part, prefix in self.inputs:
            for local, ts in part.tensor_specs().items():
                out[prefix + local] = ts
        if self.passes is not None:
            for local, ts in self.passes.tensor_specs().items():
                out[self._passes_prefix + local] = ts
        for ls, (norm1, mixer, norm2, ffn), extra, block in zip(spec.layers, self._layer_parts, self._extra_norms,
                                                                self.blocks):
            out.update(self._norm_specs(norm1, ls.mixer_norm_name))
            for local, ts in mixer.tensor_specs().items():
                out[ls.mixer_prefix + local] = ts
            if ffn is not None:
                if norm2 is not None:
                    out.update(self._norm_specs(norm2, ls.ffn_norm_name))
                for local, ts in ffn.tensor_specs().items():
                    out[ls.ffn_prefix + local] = ts
            for role, norm in extra.items():
                out.update(self._norm_specs(norm, ls.extra_norms[role][1]))
            for local, ts in self._block_specs(block).items():    # an arrangement with tensors of its own
                out[ls.block_prefix + local] = ts
        return out

    def load(self, source, where: str = "weights", strict: bool = True) -> None:
        """Check `source` against the expected tensors (one error for everything that is
        wrong), then hand each part its tensors.

        A source without the output head's tensor ties the head to the embedding table, as
        the reference does whenever `output.weight` is absent
        (src/model_weights/names.rs:300-310), whatever the configuration's flag says.
        `strict=False` accepts tensors the model does not know (a checkpoint that carries
        extras) and lists them in `self.ignored_tensors`."""
        expected = self.expected_tensors()
        rt, spec = self.rt, self.spec
        head_name = spec.lm_head_name
        if head_name is not None and head_name not in set(source.names()):
            expected.pop(head_name)
            head_name = None
            self.notes.append(f"{where}: no {spec.lm_head_name!r}; the output head is tied to "
                              f"{spec.embedding_name!r}")
        self.ignored_tensors = check_source(expected, source, where, strict=strict)
        if self.ignored_tensors:
            self.notes.append(f"{where}: {len(self.ignored_tensors)} tensor(s) the model does not use were "
                              f"ignored: " + ", ".join(self.ignored_tensors[:8])
                              + (" ..." if len(self.ignored_tensors) > 8 else ""))

        # every tensor to the device first (files: one pass of the native reader per file), then
        # each part takes its own; a part that fuses matrices lets go of the separate ones
        tensors = fetch_many(source, list(expected), rt.dtype, rt.device)

        def get(name):
            return tensors.pop(name)

        def load_norm(norm, weight_name):
            norm.load({local: get(name) for local, name in self._norm_names(norm, weight_name).items()})

        self.embedding = get(spec.embedding_name)
        load_norm(self.final_norm, spec.final_norm_name)
        self.lm_head.load({"weight": self.embedding if head_name is None else get(head_name)})
        tied = getattr(self.lm_head, "weight", None)
        if head_name is None and tied is not None and tied.dtype == self.embedding.dtype \
                and tied.shape == self.embedding.shape:
            self.embedding = tied                          # tied: one copy
        for part, prefix in self.inputs:
            part.load({local: get(prefix + local) for local in part.tensor_specs()})
        if self.passes is not None:
            self.passes.load({local: get(self._passes_prefix + local) for local in self.passes.tensor_specs()})
        for ls, (norm1, mixer, norm2, ffn), extra, block in zip(spec.layers, self._layer_parts, self._extra_norms,
                                                                self.blocks):
            load_norm(norm1, ls.mixer_norm_name)
            mixer.load({local: get(ls.mixer_prefix + local) for local in mixer.tensor_specs()})
            if ffn is not None:
                if norm2 is not None:
                    load_norm(norm2, ls.ffn_norm_name)
                ffn.load({local: get(ls.ffn_prefix + local) for local in ffn.tensor_specs()})
            for role, norm in extra.items():
                load_norm(norm, ls.extra_norms[role][1])
            if self._block_specs(block):
                block.load({local: get(ls.block_prefix + local) for local in self._block_specs(block)})
        self.loaded = True

    def load_random(self, seed: int, std: float = 0.02, on_device: bool = False) -> None:
        """Seeded random weights without a folder (`on_device` draws them on the GPU, for
        models too large to make on the host in reasonable time)."""
        src = RandomSource(self.expected_tensors(), seed, std, dtype=self.rt.dtype,
                           device=self.rt.device if on_device else "cpu")
        self.load(src, where="random weights")

    # ---- cache ----------------------------------------------------------------------------
    def cache_requests(self) -> Dict[int, CacheRequest]:
        """What each cache-writing schedule entry asks of the cache, keyed by its position, and what the step inputs ask
        (keys below 0)."""
        out = {}
        for pos, e in enumerate(self.spec.schedule):
            if e.writes_cache:
                out[pos] = self._layer_parts[e.layer][1].cache_request()
        for i, (part, _) in enumerate(self.inputs):
            request = getattr(part, "cache_request", lambda: None)()
            if request is not None:
                out[self._input_key(i)] = request
        return out

    @staticmethod
    def _input_key(i: int) -> int:
        """Under which key the cache keeps what the i-th step input asked for (the schedule's entries count from 0)."""
        return -1 - i

    def graph_safe(self) -> bool:
        """True when every part declares `graph_safe`: its forward reads the step's sequences
        from device memory only, so a captured launch sequence stays right for later steps."""
        parts = [self.final_norm, self.lm_head] + [part for part, _ in self.inputs]
        if self.passes is not None:
            parts.append(self.passes)
        for e in self.spec.schedule:
            parts.extend(p for p in self._layer_parts[e.layer] if p is not None)
            parts.extend(self._extra_norms[e.layer].values())
            parts.append(self.blocks[e.layer])
        return self.after_block is None and all(getattr(p, "graph_safe", False) for p in parts)

    def weight_bytes_per_step(self) -> int:
        """Bytes of weights a one-token step reads: every matrix each scheduled layer uses,
        the norm scales, the output head (the embedding rows it gathers are negligible)."""
        others = [part for part, _ in self.inputs] + [self.passes]
        total = self.lm_head.nbytes() + sum(part.weight_bytes() for part in others if hasattr(part, "weight_bytes"))
        for e in self.spec.schedule:
            norm1, mixer, norm2, ffn = self._layer_parts[e.layer]
            for part in (mixer, ffn):
                if part is not None and hasattr(part, "weight_bytes"):
                    total += part.weight_bytes()
            for n in (norm1, norm2, *self._extra_norms[e.layer].values()):
                if getattr(n, "weight", None) is not None:
                    total += n.weight.numel() * n.weight.element_size()
        return total

    # ---- forward --------------------------------------------------------------------------
    def cut_by_length(self, pos0, cache) -> bool:
        """Does any mixer want this one-token step (positions of the live sequences) cut by length?
        Each is asked with the view of the cache that its layer reads."""
        if self._cut_askers is None:
            # every mixer that has the (optional) method, one per `cut_by_length_key()` where mixers
            # say that their answers are the same (layers of equal shape): asked every step
            seen, self._cut_askers = set(), []
            for pos, e in enumerate(self.spec.schedule):
                mixer = self._layer_parts[e.layer][1]
                ask = getattr(mixer, "cut_by_length", None)
                if ask is None:
                    continue
                key = getattr(mixer, "cut_by_length_key", lambda m=mixer: id(m))()
                if key not in seen:
                    seen.add(key)
                    self._cut_askers.append((ask, self.spec.cache_entry(pos)))
        return any(ask(pos0, cache.layer_view(entry)) for ask, entry in self._cut_askers)

    def forward(self, ctx: StepContext, tokens: torch.Tensor, cache, logit_rows: Optional[torch.Tensor],
                n_logit_rows: int, logits_out: Optional[torch.Tensor] = None) -> Optional[torch.Tensor]:
        """Run the step's tokens through the scheduled layers.

        tokens      int32 [n_tokens] on the device
        logit_rows  int32 [n_logit_rows] on the device: packed-token rows whose logits are wanted
        Returns float32 [n_logit_rows, vocab] (None when no row is wanted)."""
        rt, spec, ws = self.rt, self.spec, self.rt.workspace
        T, H = ctx.n_tokens, spec.hidden_size
        x = ws.take("model.residual", (T, H), torch.float32)
        sched = spec.schedule
        # the first block's first norm may ask the embedding kernel for its element-wise half
        # (not when step inputs or the start of a pass may still change the embedded rows)
        begins = bool(sched) and sched[0].pass_start is not None
        request = first_norm_request_of(self.blocks[sched[0].layer], ctx) if sched and not self.inputs and not begins else None
        ahead = finish = None
        if request is not None:
            from ..parts.norm import honour
            ahead, finish = honour(request, x, ctx, "embed", 1)
        embeds = bool(self.inputs) and getattr(self.inputs[0][0], "embeds", False)
        if not embeds:
            B.embed_gather(self.embedding, tokens, x, spec.embedding_scale, rt.err, ctx.stream, ahead=ahead)
        ctx.rows_ahead = finish() if finish is not None else None
        for i, (part, _) in enumerate(self.inputs):
            ctx.input_view = cache.layer_view(self._input_key(i))
            if i == 0 and embeds:
                part.embed(self.embedding, tokens, x, spec.embedding_scale, ctx)
            else:
                part.prepare(tokens, x, ctx)
        ctx.input_view = None
        if self.passes is not None:
            self.passes.embedded(x, ctx, begins)
        S = spec.residual_streams
        rows = x
        if S is not None:
            # the residual as S streams per token, all equal to the embedded row at the start
            rows = ws.take("model.streams", (T, S, H), torch.float32)
            B.streams_expand(x, rows, T, S, H, ctx.stream)
        for pos, e in enumerate(sched):
            view = cache.layer_view(spec.cache_entry(pos))
            if e.pass_start is not None:
                self.passes.begin(e.pass_start, rows, ctx, self.blocks[e.layer], pos == 0)
            # no block prepares rows for a layer in front of which the start of a pass changes them
            last = pos + 1 == len(sched) or sched[pos + 1].pass_start is not None
            ctx.next_block = None if last else self.blocks[sched[pos + 1].layer]
            self.blocks[e.layer].forward(rows, ctx, view, e.writes_cache)
            if self.after_block is not None:
                self.after_block(pos, rows, ctx)
        ctx.rows_ahead = None
        if n_logit_rows == 0:
            return None
        hn = ws.take("model.head_in", (n_logit_rows, H), rt.dtype)
        if S is not None:                        # the final norm of the sum of the streams
            self.final_norm.forward_streams(rows, S, hn, ctx, rows_idx=logit_rows, rows=n_logit_rows)
        else:
            self.final_norm.forward(x, hn, ctx, rows_idx=logit_rows, rows=n_logit_rows)
        if logits_out is None:
            logits_out = torch.empty((n_logit_rows, spec.vocab_size), dtype=torch.float32, device=rt.device)
        self.lm_head.forward(hn, logits_out, n_logit_rows, ctx)
        return logits_out
