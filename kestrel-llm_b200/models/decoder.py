"""A decoder as data: an embedding, a list of blocks, the order in which they run, a final
norm and an output head.

``order`` is a list of `LayerCall`s.  A call names the block it runs and the cache layer it
uses; a block may appear in several calls (its weights run twice, each call with a cache
layer of its own or a shared one), and a call with ``writes_cache=False`` reads a cache layer
that an earlier call of the same step filled; a call with ``add_embedding`` adds the embedded tokens
to the stream once more before its block runs (a model that runs a stretch of its layers several
times feeds them in at the start of each further pass); a call with ``add_row`` adds a learned vector of the
model's ``stream_rows`` to every token of the stream before its block runs.  The reference runs its layers in a fixed loop
(src/model/vllm_safetensors.c:16404-16812); here the loop walks this list.
"""
from __future__ import annotations

from dataclasses import dataclass
from typing import List, Optional, Sequence

import torch

from ..csrc import ops
from ..parts.base import Block, CacheSpec, Norm, Part, PositionEncoding, WeightSlot
from ..parts.embedding import LMHead, TokenEmbedding


@dataclass(frozen=True)
class LayerCall:
    block: int                  # index into DecoderModel.blocks
    cache: int = -1             # cache layer it uses, -1 for none
    writes_cache: bool = True   # False: attends over what an earlier call wrote
    add_embedding: bool = False  # the embedded tokens are added to the stream once more in front of this call
    add_row: int = -1            # row of the model's `stream_rows` that is added to every token of the stream in front of this call


class DecoderModel(Part):
    def __init__(self, config, dtype: torch.dtype, device, embedding: TokenEmbedding,
                 position: Optional[PositionEncoding], blocks: Sequence[Block],
                 order: Sequence[LayerCall], final_norm: Norm, lm_head: LMHead,
                 optional_tensors: Sequence[str] = (), shared_parts: Sequence[Part] = (), embedding_norm: Optional[Norm] = None,
                 stream_rows=None):
        self.config = config
        self.dtype = dtype
        self.device = torch.device(device)
        self.embedding = embedding
        self.position = position
        self.embedding_norm = embedding_norm                # a norm of the embedded tokens (after the position vector), or None
        self.blocks = list(blocks)
        self.order = list(order)
        self.final_norm = final_norm
        self.lm_head = lm_head
        self.optional_tensors = tuple(optional_tensors)   # may be in a checkpoint, are not used
        self.shared_parts = list(shared_parts)            # parts that several blocks use (a table all layers read): their weights are the model's
        self.stream_rows = stream_rows                      # `StreamRows`: vectors that layer calls add to the stream, or None
        if any(c.add_row >= 0 for c in order) and stream_rows is None:
            raise ValueError("a layer call adds a row to the stream, but the model has no stream rows")
        n_cache = 1 + max([c.cache for c in self.order], default=-1)
        owners: List[Optional[int]] = [None] * n_cache
        for c in self.order:
            if c.cache >= 0 and c.writes_cache:
                if owners[c.cache] is not None:
                    raise ValueError(f"cache layer {c.cache} is written by two layer calls")
                owners[c.cache] = c.block
        for c in self.order:
            if c.cache >= 0 and not c.writes_cache and owners[c.cache] is None:
                raise ValueError(f"cache layer {c.cache} is read but never written")
        seen = set()
        for c in self.order:        # a reader must come after the writer
            if c.cache >= 0:
                if c.writes_cache:
                    seen.add(c.cache)
                elif c.cache not in seen:
                    raise ValueError(f"cache layer {c.cache} is read before it is written")
        self._cache_owner = owners
        # the first block reads the stream unnormed, and the stream starts as rows of the table: the table's rows are that copy
        self._starts_with_copy = bool(self.order) and getattr(self.blocks[self.order[0].block], "reads_stream_copy", False) and \
            position is None and embedding_norm is None and self.order[0].add_row < 0 and embedding.copies_rows
        if any(c.add_embedding for c in self.order) and (embedding_norm is not None or (
                position is not None and type(position).add_to_embedding is not PositionEncoding.add_to_embedding)):
            raise ValueError("feeding the embedded tokens in again is built for models whose stream starts as the table's rows alone")

    @property
    def graph_safe(self) -> bool:
        """Whether a decode step through the whole model can be captured in a CUDA graph."""
        pos_ok = self.position is None or (getattr(self.position, "graph_safe", False)
                                           or type(self.position).add_to_embedding is PositionEncoding.add_to_embedding)
        return (pos_ok and all(b.graph_safe for b in self.blocks) and self.final_norm.graph_safe
                and (self.embedding_norm is None or self.embedding_norm.graph_safe)
                and self.embedding.graph_safe and self.lm_head.graph_safe)

    @property
    def vocab_size(self) -> int:
        return self.lm_head.vocab

    def cache_specs(self) -> List[CacheSpec]:
        """What each cache layer keeps, taken from the block that writes it."""
        return [self.blocks[b].cache_spec() if b is not None else None for b in self._cache_owner]

    def weight_slots(self) -> List[WeightSlot]:
        slots = self.embedding.weight_slots()
        if self.position is not None:
            slots += self.position.weight_slots()
        if self.embedding_norm is not None:
            slots += self.embedding_norm.weight_slots()
        for part in self.shared_parts:
            slots += part.weight_slots()
        if self.stream_rows is not None:
            slots += self.stream_rows.weight_slots()
        for b in self.blocks:
            slots += b.weight_slots()
        slots += self.final_norm.weight_slots() + self.lm_head.weight_slots()
        return slots

    def step_program(self, cache):
        """The whole step as a `StepProgram` for the native runner, or None if some part of the
        model has no ``emit`` (it then runs by the walk below).  ``cache`` is the `CacheManager`
        whose layers the program's attention operations point into."""
        from ..csrc import ops
        pos_ok = (self.position is None or type(self.position).add_to_embedding is PositionEncoding.add_to_embedding) \
            and self.embedding_norm is None
        blocks_ok = all(getattr(b, "emit", None) is not None and getattr(b, "emits", False) for b in self.blocks) \
            and not any(c.add_embedding or c.add_row >= 0 for c in self.order) and getattr(self.lm_head, "plain", True)
        if not (pos_ok and blocks_ok and all(getattr(p, "emit", None) is not None
                                              for p in (self.embedding, self.final_norm, self.lm_head))):
            return None
        prog = ops.StepProgram(self.dtype)
        x = self.embedding.emit(prog)
        pending = None
        for call in self.order:
            lc = cache.layer(call.cache, call.writes_cache) if call.cache >= 0 else None
            prog.begin_call()
            pending = self.blocks[call.block].emit(prog, x, pending, lc)
        prog.begin_call()
        n = self.final_norm.emit(prog, x, pending, self.dtype, logit_rows=True)
        self.lm_head.emit(prog, n)
        return prog

    def forward(self, batch, cache) -> Optional[torch.Tensor]:
        """Runs this step's tokens through every layer call; returns float32 logits
        [len(batch.logit_rows), vocab], or None if no logits are wanted."""
        x, pending = self.forward_embed(batch)
        x, pending = self.forward_calls(x, pending, batch, cache, 0, len(self.order))
        return self.forward_head(x, pending, batch)

    # The three stages of `forward`, for callers that run a step in pieces (a captured decode
    # step is two graphs, so that the second is submitted while the first already runs).
    def forward_embed(self, batch):
        if self._starts_with_copy:
            return self.embedding.forward_with_copy(batch.token_ids)
        x = self.embedding.forward(batch.token_ids)
        if self.position is not None:
            self.position.add_to_embedding(x, batch)
        if self.embedding_norm is not None:                 # the stream starts as the normed embedding, still float32
            x = self.embedding_norm.add_forward(x, None, torch.float32)
        return x, None

    def forward_calls(self, x, pending, batch, cache, lo: int, hi: int):
        """Layer calls order[lo:hi] on the residual stream ``x`` and the not yet added ``pending``."""
        for call in self.order[lo:hi]:
            lc = cache.layer(call.cache, call.writes_cache) if call.cache >= 0 else None
            if (call.add_embedding or call.add_row >= 0) and isinstance(pending, ops.StreamCopy):
                pending = None                  # a copy of the stream as it was: nothing to add, and about to be out of date
            if call.add_embedding:
                if pending is not None:         # what the call before left unadded goes in first
                    ops.add_two(x, pending, None, None)
                    pending = None
                self.embedding.add_forward(batch.token_ids, x)
            if call.add_row >= 0:
                if pending is not None:
                    ops.add_two(x, pending, None, None)
                    pending = None
                self.stream_rows.add_forward(call.add_row, x)
            x, pending = self.blocks[call.block].forward(x, pending, batch, lc)
        return x, pending

    def forward_head(self, x, pending, batch) -> Optional[torch.Tensor]:
        if batch.num_logit_rows == 0:
            return None
        if isinstance(pending, ops.StreamCopy):
            pending = None                      # the stream is complete
        n = self.final_norm.add_forward(x, pending, self.dtype, rows=batch.logit_rows)
        return self.lm_head.forward(n)
