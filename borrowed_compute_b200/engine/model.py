"""A decoder assembled from a ModelSpec: embedding, blocks in scheduled order, final norm,
head.  Nothing here knows an architecture; the sequence of work is the reference's
(crates/bc-infer/src/lib.rs:50-54: embed, forward, logits)."""

from __future__ import annotations

from typing import Any, Dict, List, Mapping, Optional, Tuple

import torch

from ..architectures import resolve
from ..parts import base as P
from ..parts.streams import StreamBundle
from ..parts.base import (BLOCKS, EMBEDDINGS, HEADS, JUNCTIONS, NORMS, POSITION_ENCODINGS, CacheNeed, ModelSpec, PartSpec, Runtime, StateNeed,
                          StepContext, TensorSpec)


def _build(registry: P.Registry, spec: PartSpec):
    return registry.get(spec.kind)(**dict(spec.params))


class DecoderModel:
    def __init__(self, spec: ModelSpec):
        self.spec = spec
        for i, run in enumerate(spec.schedule):
            if not 0 <= run.layer < len(spec.layers):
                raise ValueError(f"schedule entry {i} names layer {run.layer}, the model has {len(spec.layers)}")
            if run.memory_of is not None and not (0 <= run.memory_of < i and spec.schedule[run.memory_of].memory_of is None):
                raise ValueError(f"schedule entry {i} reads the memory of entry {run.memory_of}, which is not an earlier owner")
        self.embedding = _build(EMBEDDINGS, spec.embedding)
        self.embedding_norm = None if spec.embedding_norm is None else _build(NORMS, spec.embedding_norm)
        self.position = None if spec.position is None else _build(POSITION_ENCODINGS, spec.position)
        self.blocks = [BLOCKS.get(layer.block).build(layer, spec.hidden_size) for layer in spec.layers]
        for layer, block in zip(spec.layers, self.blocks):
            if block.STREAMS != (spec.streams > 0):
                raise ValueError(f"block '{layer.block}' runs on {'a bundle of streams' if block.STREAMS else 'one residual stream'}, the model has {spec.streams or 'one plain stream'}")
        if spec.streams and (spec.junctions or spec.position is not None):
            raise ValueError("a bundle of streams takes no junctions and no position encoding on the embeddings")
        self.junctions = [_build(JUNCTIONS, j) for j in spec.junctions]
        for i, run in enumerate(spec.schedule):
            if run.enter is not None and not 0 <= run.enter[0] < len(self.junctions):
                raise ValueError(f"schedule entry {i} enters junction {run.enter[0]}, the model has {len(self.junctions)}")
        # Positions that the embedding adds in its own kernel; where a norm stands between the two, or a junction reads the embedding
        # again, they stay apart.
        self.position_joined = self.position is not None and self.embedding_norm is None and not spec.junctions and self.embedding.join(self.position)
        # Runs whose block may leave the stream in the activation type for the next one.
        self.hand_over = [i + 1 < len(spec.schedule) and spec.schedule[i + 1].enter is None and self.blocks[run.layer].enters_plain
                          and self.blocks[spec.schedule[i + 1].layer].enters_plain for i, run in enumerate(spec.schedule)]
        self.final_norm = _build(NORMS, spec.final_norm)
        self.head = _build(HEADS, spec.head)
        self.rt: Optional[Runtime] = None
        # For looking inside a step: called as after_run(schedule entry, residual) when a run has added to the stream
        # (an eager step only; a captured step replays without it); where the stream is a bundle, residual is the sum of its copies.
        self.after_run = None

    def named_parts(self):
        """(tensor-name prefix, part) of every part of the model; each block lists its own."""
        yield self.spec.embedding.prefix, self.embedding
        if self.embedding_norm is not None:
            yield self.spec.embedding_norm.prefix, self.embedding_norm
        if self.position is not None:
            yield self.spec.position.prefix, self.position
        for layer, block in zip(self.spec.layers, self.blocks):
            yield from block.named_parts(layer)
        for spec, junction in zip(self.spec.junctions, self.junctions):
            yield spec.prefix, junction
        yield self.spec.final_norm.prefix, self.final_norm
        yield self.spec.head.prefix, self.head

    def expected_tensors(self) -> Dict[str, TensorSpec]:
        out: Dict[str, TensorSpec] = {}
        for prefix, part in self.named_parts():
            for name, spec in part.tensors().items():
                out[prefix + name] = spec
        for name, shape in self.spec.tolerated:
            out.setdefault(name, TensorSpec(tuple(shape), role="vector", optional=True))
        return out

    def load(self, tensors: Mapping[str, torch.Tensor], rt: Runtime) -> None:
        self.rt = rt
        for prefix, part in self.named_parts():
            mine = {name: tensors[prefix + name] for name in part.tensors() if prefix + name in tensors}
            part.load(mine, rt)

    def memory_needs(self) -> Tuple[List[Optional[CacheNeed]], List[Optional[StateNeed]], List[Optional[int]]]:
        needs, states, memory_of = [], [], []
        for run in self.spec.schedule:
            mixer = self.blocks[run.layer].memory_part()
            needs.append(None if mixer is None else mixer.cache_need())
            states.append(None if mixer is None else mixer.state_need())
            memory_of.append(run.memory_of)
        need = self.embedding.cache_need()
        if need is not None:        # one more entry, behind the runs'
            needs, states, memory_of = needs + [need], states + [None], memory_of + [None]
        # A run that reads another's memory may see further back than its owner: the owner keeps what both read.
        for i, j in enumerate(memory_of):
            if j is not None and needs[j] is not None and needs[i] is not None:
                needs[j] = needs[j].widened(needs[i])
        return needs, states, memory_of

    def more_state_needs(self) -> List[Dict[str, StateNeed]]:
        """For every run, the per-sequence state its block's other parts ask for, by role."""
        return [dict(self.blocks[run.layer].state_needs()) for run in self.spec.schedule]

    def forward(self, ctx: StepContext, cache, want_rows: Optional[torch.Tensor], n_want: int) -> torch.Tensor:
        """Scores [n_want, vocab] float32 at rows ``want_rows`` (all rows if None)."""
        rt = self.rt
        residual = torch.empty((ctx.rows, self.spec.hidden_size), dtype=torch.float32, device=rt.device)
        self._embed(ctx, cache, residual)
        if self.spec.streams:
            return self._forward_streams(residual, ctx, cache, want_rows, n_want)
        if self.embedding_norm is not None:
            self.embedding_norm.forward(residual.clone(), residual)
        if self.position is not None and not self.position_joined:
            self.position.on_embeddings(residual, ctx)
        embedded = None
        if any(j.needs_embedding for j in self.junctions):
            # The embedding's output is read again later: a second gather keeps it (the stream itself moves on).
            embedded = torch.empty_like(residual)
            self._embed(ctx, cache, embedded)
        for i, run in enumerate(self.spec.schedule):
            if run.enter is not None:
                self.junctions[run.enter[0]].forward(residual, embedded, ctx, run.enter[1])
            ctx.hand_over = self.hand_over[i]
            self.blocks[run.layer].forward(residual, ctx, cache.memory(i), rt)
            if self.after_run is not None and not ctx.extras.get("graph"):
                self.after_run(i, residual)
        h = torch.empty((n_want, self.spec.hidden_size), dtype=rt.dtype, device=rt.device)
        self.final_norm.forward(residual, h, want_rows)
        return self._scores(h)

    def _embed(self, ctx: StepContext, cache, out: torch.Tensor) -> None:
        if self.embedding.cache_need() is None:
            self.embedding.forward(ctx, out)
        else:
            self.embedding.forward(ctx, out, mem=cache.memory(len(self.spec.schedule)))

    def _scores(self, h: torch.Tensor) -> torch.Tensor:
        scores = torch.empty((h.shape[0], self.spec.vocab_size), dtype=torch.float32, device=self.rt.device)
        self.head.forward(h, scores, self.embedding.table())
        return scores

    def _forward_streams(self, embedded: torch.Tensor, ctx: StepContext, cache, want_rows: Optional[torch.Tensor], n_want: int) -> torch.Tensor:
        """``forward`` where a row's residual stream is a bundle of copies."""
        rt = self.rt
        bundle = StreamBundle(ctx.rows, self.spec.streams, self.spec.hidden_size, rt.device)
        bundle.start(embedded, self.embedding_norm)
        for i, run in enumerate(self.spec.schedule):
            self.blocks[run.layer].forward(bundle, ctx, cache.memory(i), rt)
            if self.after_run is not None and not ctx.extras.get("graph"):
                self.after_run(i, bundle.total())
        h = torch.empty((n_want, self.spec.hidden_size), dtype=rt.dtype, device=rt.device)
        bundle.finish(self.final_norm, h, want_rows)
        return self._scores(h)


def model_for_config(config: Mapping[str, Any], shapes: Optional[Mapping[str, tuple]] = None) -> Tuple[Any, DecoderModel]:
    """The typed configuration and the (unloaded) model a config.json dict describes.
    ``shapes`` (tensor name -> shape of what the folder holds) lets an architecture whose
    config.json leaves a size to the tensors fill it in."""
    arch = resolve(config)
    if arch.complete is not None and shapes is not None:
        config = arch.complete(config, shapes)
    typed = arch.parse_config(config)
    return typed, DecoderModel(arch.model_spec(typed))


def expected_tensors_for_config(config: Mapping[str, Any]) -> Dict[str, TensorSpec]:
    return model_for_config(config)[1].expected_tensors()
