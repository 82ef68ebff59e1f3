"""A model put together from its description: the embedding, the blocks in the order of the
run list, the final norm and the output matrix.  Nothing here knows an architecture: the
description (air_b200.parts.spec.ModelSpec) is data that the architecture's entry in the
registry produced from config.json.
"""
from __future__ import annotations

from typing import Dict, List

import torch

from ..csrc import ops
from ..parts import registry
from ..parts.base import Norm, Runtime, row_terms
from ..parts.linear import Linear
from ..parts.spec import ModelSpec, PartSpec
from ..weights.loader import TensorSpec


class Model:
    def __init__(self, spec: ModelSpec):
        spec.validate()
        self.spec = spec
        self.blocks = [registry.BLOCKS.get(b.kind)(b) for b in spec.layers]
        self.final_norm = registry.NORMS.get(spec.final_norm.kind)(spec.final_norm, spec.final_norm_prefix)
        emb = spec.embedding or PartSpec("tokens", {"vocab": spec.vocab_size, "hidden": spec.hidden_size,
                                                    "multiplier": spec.embedding_multiplier})
        self.embedder = registry.EMBEDDINGS.get(emb.kind)(emb, spec.embedding_name)
        # runs that take the embedding's output into the stream again need a second copy of it
        self.embedding_copies = 2 if any(run.add_embedding or run.mix_embedding for run in spec.order) else 1

    # ------------------------------------------------------------------ tensors
    def tensor_specs(self) -> List[TensorSpec]:
        s = self.spec
        specs = list(self.embedder.tensor_specs())
        specs += [TensorSpec(name, (rows, s.hidden_size), wide=True) for name, rows in s.stream_tables]
        specs += [TensorSpec(name, (s.hidden_size, 2 * s.hidden_size)) for name in s.stream_mixes]
        for b in self.blocks:
            specs += b.tensor_specs()
        specs += self.final_norm.tensor_specs()
        if s.output_name is not None:
            specs.append(TensorSpec(s.output_name, (s.vocab_size, s.hidden_size)))
        if s.output_bias_name is not None:
            specs.append(TensorSpec(s.output_bias_name, (s.vocab_size,), init="zeros", wide=True))
        seen = set()
        for t in specs:
            if t.name in seen:
                raise ValueError(f"two parts claim the tensor '{t.name}'")
            seen.add(t.name)
        return specs

    def load(self, tensors: Dict[str, torch.Tensor], rt: Runtime) -> None:
        self.rt = rt
        self.embedder.load(tensors, rt)
        self.embedding = self.embedder.table
        self.stream_tables = {name: tensors[name].to(torch.float32).contiguous() for name, _ in self.spec.stream_tables}
        self.stream_mixes = {name: Linear(tensors[name], rt.status) for name in self.spec.stream_mixes}
        for b in self.blocks:
            b.load(tensors, rt)
        self.final_norm.load(tensors, rt)
        out = self.embedding if self.spec.output_name is None else tensors[self.spec.output_name]
        self.output = Linear(out, rt.status)
        bias = None if self.spec.output_bias_name is None else tensors[self.spec.output_bias_name]
        self.output_bias = None if bias is None else bias.to(torch.float32)
        self._planners = None
        # for tests and for finding a fault layer by layer: a list that receives, after every run, a copy of the
        # stream as it stands behind that run (what is still pending added to it)
        self.tap = None

    def planners(self):
        """The parts that plan on the host, one for every plan key (Part.plan_key)."""
        if self._planners is None:
            found = {}
            for b in self.blocks:
                for part in b.parts():
                    key = part.plan_key()
                    if key is not None and key not in found:
                        found[key] = part
            self._planners = tuple(found.values())
        return self._planners

    @property
    def graph_safe(self) -> bool:
        """Whether a decode step may be captured in a CUDA graph: no part reads the batch on the host."""
        return all(b.graph_safe for b in self.blocks) and getattr(self.final_norm, "graph_safe", False) \
            and getattr(self.embedder, "graph_safe", False)

    def cache_needs(self):
        """Per run of the order list: the needs of the layer's mixer, or for a run that reads another run's cache what
        it keeps all the same (usually nothing); behind the runs, what the embedding keeps per request."""
        return [self.blocks[run.layer].cache_needs() if run.cache_from is None
                else tuple(getattr(self.blocks[run.layer], "borrowing_needs", tuple)())
                for run in self.spec.order] + [tuple(self.embedder.cache_needs())]

    def weight_bytes(self) -> int:
        """Bytes of the tensors that one step reads (every weight once)."""
        seen, total = set(), 0

        def add(t):
            nonlocal total
            if isinstance(t, torch.Tensor) and t.data_ptr() not in seen:
                seen.add(t.data_ptr())
                total += t.numel() * t.element_size()

        for run in {r.layer for r in self.spec.order}:
            b = self.blocks[run]
            for part in b.parts():
                for v in vars(part).values():
                    if isinstance(v, Linear):
                        add(v.weight)
                    else:
                        add(v)
        for mix in self.stream_mixes.values():
            add(mix.weight)
        add(self.output.weight)
        add(self.final_norm.weight)
        return total

    # ------------------------------------------------------------------ computing
    def _mixed(self, h, pending, x0, mix):
        """(stream, pending) of W [x | x0]: one kernel completes x and writes the rows [x | x0] in the compute dtype; the
        product's partial sums (few rows) are the new stream and what is still to be added to it."""
        T, E = h.shape
        terms = row_terms(pending)
        if terms is None:
            h, terms = Norm.add_delta(h, pending), []
        rows = torch.empty((T, 2 * E), dtype=self.rt.dtype, device=h.device)
        ops.stream_norm(h, 1, None, None, 0.0, rows, term=terms[0][0] if terms else None, more=terms[1:], again=x0)
        y = mix.f32_sums(rows)
        if y.dim() == 2:
            return y, None
        return y[0], y[1:] if y.shape[0] > 1 else None

    def forward(self, ctx, cache) -> torch.Tensor:
        """Runs the batch's tokens through every run of the order list, writing the caches,
        and returns float32 logits [wanted rows, vocab]."""
        rt = self.rt
        ctx.shared.clear()
        h, *again = self.embedder.forward(ctx, cache.views(len(self.spec.order)), self.embedding_copies)
        pending = None
        for i, run in enumerate(self.spec.order):
            owner = i if run.cache_from is None else run.cache_from
            if run.mix_embedding is not None:
                h, pending = self._mixed(h, pending, again[0], self.stream_mixes[run.mix_embedding])
            if run.add_embedding or run.add_row is not None:
                # what the run adds to the stream ahead of its layer: the stream is completed first
                h = Norm.add_delta(h, pending)
                pending = None
                row = None if run.add_row is None else self.stream_tables[run.add_row[0]][run.add_row[1]]
                ops.stream_add(h, again[0] if run.add_embedding else None, row)
            kept = cache.views(i) if run.cache_from is not None else ()
            h, pending = self.blocks[run.layer].forward(h, pending, ctx, cache.views(owner),
                                                        owns_cache=run.cache_from is None,
                                                        **({"kept": kept} if kept else {}))
            if self.tap is not None:
                x = Norm.add_delta(h.clone(), pending)
                self.tap.append(x if x.dim() == 2 else x.sum(0))      # (several streams: their sum)
        R = ctx.logit_rows.shape[0]
        if R == 0:
            return torch.empty((0, self.spec.vocab_size), dtype=torch.float32, device=rt.device)
        y = self.final_norm.forward(h, pending, rows=ctx.logit_rows)
        logits = self.output.full(y) if self.output.small(y) else self.output(y, torch.float32)
        s = self.spec
        if self.output_bias is not None or s.logit_scale != 1.0 or s.logit_softcap > 0.0:
            ops.logits_post(logits, self.output_bias, s.logit_scale, s.logit_softcap)
        return logits
