"""The generic decoder: embedding, the scheduled runs of layers, final norm, head.

The reference's `QwenModel` hard-wires one layer class N times
(somi_inference/models/qwen2.py:342-386) and its adapter adds the head
(somi_inference/models/qwen2_adapter.py:60-62,95,146).  This decoder is built
from a `ModelSpec`: every layer names its own parts, and the order of execution
is the spec's schedule, which may run a layer twice or let a run read another
run's cache.  It knows no architecture.
"""

from __future__ import annotations

import torch

from ..config.spec import LayerSpec, ModelSpec
from .base import BuildContext, CacheNeeds, StateNeeds, StreamStart, TensorDecl, with_extra_rows
from .registry import (ARRANGEMENTS, EMBEDDINGS, FEED_FORWARDS, HEADS, LAYER_EXTRAS, MIXERS,
                       NORMS, STREAM_PARTS)


def declared_tensors(spec: ModelSpec) -> dict[str, TensorDecl]:
    """Every tensor the weight file must hold, by name."""
    out: dict[str, TensorDecl] = {}

    def add(decls) -> None:
        for d in decls:
            if d.name in out and out[d.name].shape != d.shape:
                raise ValueError(f"tensor {d.name!r} is declared twice with different shapes")
            out.setdefault(d.name, d)

    add(EMBEDDINGS.declare(spec.embedding))
    for layer in spec.layers:
        if layer.mixer is not None:
            add(MIXERS.declare(layer.mixer))
        if layer.feed_forward is not None:
            add(FEED_FORWARDS.declare(layer.feed_forward))
        for norm in layer.norms.values():
            add(NORMS.declare(norm))
        for extra in layer.extras.values():
            add(LAYER_EXTRAS.declare(extra))
    for part in spec.stream_parts.values():
        add(STREAM_PARTS.declare(part))
    add(NORMS.declare(spec.final_norm))
    add(HEADS.declare(spec.head))
    return out


class Decoder:
    def __init__(self, spec: ModelSpec, tensors: dict[str, torch.Tensor], ctx: BuildContext) -> None:
        spec.validate()
        self.spec = spec
        self.ctx = ctx
        decls = declared_tensors(spec)
        lacking = [n for n, d in decls.items() if n not in tensors and not (d.optional or d.ignored)]
        if lacking:
            raise KeyError(f"tensors missing for the model: {', '.join(sorted(lacking))}")
        placed = {name: ctx.place(tensors[name], matrix=d.matrix) for name, d in decls.items()
                  if name in tensors and not d.ignored}
        self.embedding = EMBEDDINGS.build(spec.embedding, placed, ctx)
        self.layers = [self._build_layer(layer, placed) for layer in spec.layers]
        self.stream_parts = {name: STREAM_PARTS.build(part, placed, ctx)
                             for name, part in spec.stream_parts.items()}
        self.final_norm = NORMS.build(spec.final_norm, placed, ctx)
        self.head = HEADS.build(spec.head, placed, ctx)
        self.schedule = spec.schedule
        # a step can be captured in a CUDA graph only if no part plans on the host per step
        self.graph_safe = all(getattr(p, "graph_safe", False)
                              for b in self.layers for p in (b.mixer, b.feed_forward)
                              if p is not None)

    def _build_layer(self, layer: LayerSpec, placed):
        mixer = None if layer.mixer is None else MIXERS.build(layer.mixer, placed, self.ctx)
        ff = (None if layer.feed_forward is None
              else FEED_FORWARDS.build(layer.feed_forward, placed, self.ctx))
        norms = {name: NORMS.build(spec, placed, self.ctx) for name, spec in layer.norms.items()}
        if not layer.extras:
            return ARRANGEMENTS.get(layer.arrangement)(mixer, ff, norms)
        extras = {name: LAYER_EXTRAS.build(spec, placed, self.ctx)
                  for name, spec in layer.extras.items()}
        return ARRANGEMENTS.get(layer.arrangement)(mixer, ff, norms, extras)

    def cache_needs(self) -> tuple[list[CacheNeeds | None], list[int | None]]:
        """Per run of the schedule: what its mixer needs (None: no mixer, or nothing) together
        with the state that the layer's arrangement keeps for its extras, and whose cache the
        run reads."""
        needs: list[CacheNeeds | None] = []
        for run in self.schedule:
            block = self.layers[run.layer]
            n = None if block.mixer is None else block.mixer.cache_needs()
            extra = block.state_needs() if hasattr(block, "state_needs") else None
            if extra is not None and extra.tensors:
                paged = None if n is None else n.paged
                own = {} if n is None or n.state is None else dict(n.state.tensors)
                clash = set(own) & set(extra.tensors)
                if clash:
                    raise ValueError(f"state names used twice in one layer: {sorted(clash)}")
                n = CacheNeeds(paged=paged, state=StateNeeds({**own, **extra.tensors}))
            needs.append(n)
        owners = [run.cache_of for run in self.schedule]
        return needs, owners

    def forward(self, batch, cache) -> torch.Tensor:
        """Run the step's tokens; return float32 logits [len(batch.logit_rows), vocab]."""
        residual = self.embedding.forward(batch)
        pending = None
        # a schedule that adds the embedding's output again keeps a copy of it: the stream itself
        # is written by the norms from the first run on
        start = (residual.clone() if any(run.add_embedding or run.remix is not None
                                         for run in self.schedule) else None)
        results = None
        if any(run.average is not None for run in self.schedule):
            # an average over depth reads the embedding's output and every run's result: the first
            # norm starts the stream in rows of its own, and the results are recorded beside it
            start, residual = residual, torch.empty_like(residual)
            pending = StreamStart(start)
            results = torch.empty((len(self.schedule), *start.shape), dtype=torch.float32,
                                  device=start.device)
        for i, run in enumerate(self.schedule):
            if run.add_embedding:
                pending = with_extra_rows(pending, start)
            if run.remix is not None:
                # the stream with everything added that is due, re-mixed with the embedding's
                # output: a new stream, nothing pending
                residual = self.stream_parts[run.remix].forward(residual, pending, start)
                pending = None
            pending = self.layers[run.layer].forward(residual, pending, batch, cache.view(i),
                                                     run.cache_of is None)
            if run.average is not None:
                pending = self.stream_parts[run.average].behind(pending, start, results, i)
        if batch.logit_rows.shape[0] == 0:
            return torch.empty((0, self.spec.vocab_size), dtype=torch.float32,
                               device=residual.device)
        h = self.final_norm.forward(residual, pending, rows=batch.logit_rows)
        return self.head.forward(h)
