"""A decoder put together from a ``ModelSpec``: embedding, blocks in the
spec's order (with what joins the residual stream ahead of a run), final norm on the wanted rows only, output head
(crates/models/qwen/src/forward.rs:1562-1606)."""
from __future__ import annotations

from typing import Dict, List, Optional

import torch

from ..config.spec import CacheNeed, ModelSpec
from ..parts.block import open_streams, read_streams, sum_of_streams
from ..parts.registry import (CacheView, Runtime, StepContext, WeightStore, _BUILDERS, build_part, settle)


class DecoderModel:
    def __init__(self, spec: ModelSpec, tensors: Dict[str, torch.Tensor], runtime: Runtime,
                 consume: bool = False):
        """``consume``: the caller gives ``tensors`` away; entries are removed
        as the parts take them, so that a model close to the device's memory
        never holds its weights twice."""
        spec.validate()
        self.spec, self.runtime = spec, runtime
        weights = WeightStore(tensors)
        self.embedding = build_part("embedding", spec.embedding, weights, runtime)
        self.joins = [build_part("join", join, weights, runtime) for join in spec.joins]
        self.blocks = []
        for layer in spec.layers:
            builder = _BUILDERS.get(("block", layer.block.kind))
            if builder is None:
                raise KeyError(f"no block arrangement of kind {layer.block.kind!r}")
            self.blocks.append(builder(layer, weights, runtime))
            if consume:
                weights.drop_taken(keep=(spec.embedding.get("weight"), spec.head.get("weight")))
        self.final_norm = build_part("norm", spec.final_norm, weights, runtime)
        head_builder = _BUILDERS.get(("head", spec.head.kind))
        if head_builder is None:
            raise KeyError(f"no head of kind {spec.head.kind!r}")
        self.head = head_builder(spec.head, weights, runtime, self.embedding)
        if consume:
            weights.drop_taken()
        self.order = list(spec.order)
        self.vocab_size = spec.vocab_size

    def cache_needs(self) -> List[Optional[CacheNeed]]:
        """What each cache entry (one per layer index) must hold."""
        needs: List[Optional[CacheNeed]] = [None] * self.spec.num_cache_entries()
        for run in self.order:
            entry = run.cache_entry()
            block = self.blocks[run.layer]   # an arrangement that keeps state of its own beside its mixer's says so
            need = block.cache_need() if hasattr(block, "cache_need") else block.mixer.cache_need()
            if run.write_cache or needs[entry] is None:
                if needs[entry] is not None and needs[entry].group_key() != need.group_key() \
                        and run.write_cache:
                    raise ValueError(f"cache entry {entry} is written by layers with different needs")
                needs[entry] = need
        return needs

    def weight_bytes(self) -> int:
        """Bytes of every weight one step reads (a layer that runs several times counts each time)."""
        total = self.head.weight_bytes() if not self.head.tied else self.embedding.weight_bytes()
        for run in self.order:
            block = self.blocks[run.layer]
            total += self.joins[run.join].weight_bytes() if run.join is not None else 0
            for part in (block.mixer, getattr(block, "feed_forward", None)):
                total += part.weight_bytes() if hasattr(part, "weight_bytes") else 0
        return total

    def forward(self, token_ids: torch.Tensor, ctx: StepContext, views, wanted_rows: Optional[torch.Tensor],
                tap=None):
        """``views(entry, write) -> CacheView``. Returns float32 logits
        [wanted, vocab], or None when no row is wanted. ``tap(index, residual)``
        is called after every layer run with the residual stream
        ``[tokens, hidden]`` as that layer leaves it (the sums that otherwise
        ride along into the next layer's first kernel are made at once then)."""
        residual = self.embedding.forward(token_ids)
        ctx.token_ids = token_ids
        streams = self.spec.streams
        if streams:   # several copies of the stream: [tokens, streams, hidden]
            residual = open_streams(residual, streams)
        # the stream as the embedding left it, for joins that read it again: a copy where a layer changes it first
        first = None
        if self.joins:
            first = residual if self.order[0].join is not None else residual.clone()
        pending = None
        for index, run in enumerate(self.order):
            block = self.blocks[run.layer]
            if run.join is not None:
                residual, pending = self.joins[run.join].forward(residual, pending, first, run.turn)
            pending = block.forward(residual, pending, ctx, views(run.cache_entry(), run.write_cache))
            if tap is not None:
                settle(residual, pending)
                pending = None
                tap(index, sum_of_streams(residual) if streams else residual)
        if wanted_rows is None or wanted_rows.numel() == 0:
            return None
        if streams:   # what is pending joins, the streams are summed and normed, on the wanted rows only
            return self.head.forward(read_streams(residual, pending, None, self.final_norm, self.runtime.dtype,
                                                  rows_index=wanted_rows, keep_streams=False))
        settle(residual, pending)
        normed = self.final_norm.forward(residual, self.runtime.dtype, rows_index=wanted_rows)
        return self.head.forward(normed)
