"""The generic decoder: embedding, the layers in their given order, the final
norm and the output head on the rows whose logits are wanted
(mini_llm/model/base.py:55-89 for the traversal)."""

from __future__ import annotations

from typing import Any, Mapping

import torch

from ..cache.manager import CacheLayout, CacheManager, LayerCache
from ..parts.base import ResidualStream, Runtime
from ..weights.checkpoint import TensorSpec
from ..weights.view import TensorView
from .description import ModelDescription, build_parts, join_schemas, named_parts


class DecoderModel:
    def __init__(self, description: ModelDescription) -> None:
        self.description = description
        parts = build_parts(description)
        self.embedding_prefix, self.embedding = parts["embedding"]
        self.blocks = parts["blocks"]  # [(prefix, block)]
        self.final_norm_prefix, self.final_norm = parts["final_norm"]
        self.head_prefix, self.head = parts["head"]
        self.stream_steps = parts["stream_steps"]    # run -> (prefix, step)
        self._parts = parts
        self.order = description.order
        self.runtime: Runtime | None = None
        self._layer_caches: list[LayerCache] | None = None

    # ------------------------------------------------------------ weights
    def tensor_schema(self) -> dict[str, TensorSpec]:
        return join_schemas(named_parts(self._parts), self.description.stored_name)

    def load(self, tensors: Mapping[str, torch.Tensor], runtime: Runtime) -> None:
        """Place every weight.  ``tensors`` is keyed by checkpoint name and has
        been validated against ``tensor_schema()`` already."""

        self.runtime = runtime
        view = TensorView.of(tensors)
        if self.description.stored_name is not None:
            view = view.renamed(self.description.stored_name)
        self.embedding.load(view.sub(self.embedding_prefix), runtime)
        for prefix, block in self.blocks:
            block.load(view.sub(prefix), runtime)
        for prefix, step in self.stream_steps.values():
            step.load(view.sub(prefix), runtime)
        self.final_norm.load(view.sub(self.final_norm_prefix), runtime)
        self.head.load(view.sub(self.head_prefix), runtime, embedding=self.embedding)

    # -------------------------------------------------------------- cache
    def cache_layout(self) -> CacheLayout:
        """One requirement per *run* of a layer (a layer named twice in the order
        has two caches); a run that uses an earlier run's cache asks for none."""

        needs = []
        for layer_index, source in zip(self.order, self.description.cache_of):
            needs.append(None if source is not None else self.blocks[layer_index][1].cache_requirement())
        # an embedding that keeps something per request (the token before a step's first one) asks behind the last run
        embedding_need = getattr(self.embedding, "cache_requirement", lambda: None)()
        if embedding_need is not None:
            needs.append(embedding_need)
        return CacheLayout.from_requirements(needs)

    def bind_cache(self, manager: CacheManager) -> None:
        self._layer_caches = [
            manager.layer_cache(run if source is None else source)
            for run, source in enumerate(self.description.cache_of)
        ]
        self._embedding_cache = manager.layer_cache(len(self.order))

    def graph_safe(self) -> bool:
        """Whether every part allows its launches to be replayed from a CUDA graph."""

        parts = [self.embedding, *(block for _, block in self.blocks), *(step for _, step in self.stream_steps.values()),
                 self.final_norm, self.head]
        return all(part.capture_safe() for part in parts)

    # ------------------------------------------------------------ forward
    def forward(self, ctx: Any) -> torch.Tensor | None:
        """Run the batch in ``ctx``; return float32 logits ``[wanted, vocab]``
        (``None`` when no row is wanted: the cache is written all the same)."""

        blocks = [self.blocks[index][1] for index in self.order]
        # the norm that reads the stream after each block: the next block's first norm, at last the final norm
        readers = [block.first_norm() for block in blocks[1:]] + [self.final_norm]
        steps = self.stream_steps
        for run in steps:       # a stream step changes the rows before the norm reads them: nothing is prepared for it
            if run > 0:
                readers[run - 1] = None
        if getattr(self.embedding, "takes_context", False):      # it reads positions and entries, and may keep state per request
            first = self.embedding.forward(ctx, self._embedding_cache)
        elif getattr(self.embedding, "fuses_norms", False):
            first = self.embedding.forward(ctx.token_ids, next_norm=None if 0 in steps else blocks[0].first_norm())
        else:
            first = self.embedding.forward(ctx.token_ids)
        if isinstance(first, ResidualStream):
            stream = first
        elif isinstance(first, tuple):     # (rows, the same rows prepared for the first norm)
            stream = ResidualStream(first[0], weighted=first[1], weighted_for=blocks[0].first_norm())
        else:
            stream = ResidualStream(first)
        # the residual rows are updated in place; a step that reads the embedding's output gets a copy of it
        first_rows = stream.resid.clone() if any(step.reads_first_rows for _, step in steps.values()) else None
        for run, (block, reader) in enumerate(zip(blocks, readers)):
            if run in steps:
                if stream.delta is not None:
                    stream.resid += stream.delta
                stream.put(None, None)
                steps[run][1].forward(stream, ctx, first_rows)
            if block.fuses_norms:
                block.forward(stream, ctx, self._layer_caches[run], next_norm=reader)
            else:
                block.forward(stream, ctx, self._layer_caches[run])
        if ctx.num_logit_rows == 0:
            return None
        if stream.weighted is not None and stream.weighted_for is self.final_norm and getattr(ctx, "logits_at_every_row", False):
            x = stream.take_rows(self.final_norm, self.head)       # every row is wanted, in order: no gather
        else:
            x = self.final_norm.norm_rows(stream.resid, stream.delta, ctx.logit_rows)
        return self.head.forward(x)
