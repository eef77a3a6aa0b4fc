"""The generic decoder that every registered architecture is built as.

Embedding (times ``ModelSpec.embedding_multiplier`` if the architecture has one, plus a learned position vector
and through a norm if it has those), the blocks of
``ModelSpec.layers`` in the order of ``ModelSpec.schedule`` (a list that may name a layer twice, let an
entry read another entry's cache, or have the embedding's output added again or joined to the stream by a matrix in
front of an entry), the final norm on the rows whose logits are wanted, the head, and the
architecture's ``logit_scale`` and ``logit_softcap`` if it has them. The head is the checkpoint's
head tensor when it has one, else the embedding:
src/akas/models/lfm2/weights.py:399-402 and _composition.py:363-380 in kreasof-ai/akas).
It holds weights and computes; caches belong to the cache manager and reach the
blocks through ``caches[entry]``.
"""

from __future__ import annotations

from typing import Callable, Dict, List, Optional

import torch

from ..config.specs import ModelSpec
from ..parts.base import Param, Runtime, build_part, load_norm, norm_params, project
from ..parts.block import Block


class Decoder:
    def __init__(self, spec: ModelSpec, runtime: Runtime):
        self.spec = spec
        self.rt = runtime
        self.blocks: List[Block] = [Block(layer, runtime) for layer in spec.layers]
        self.final_norm = build_part("norm", spec.final_norm, runtime)
        self.schedule = spec.run_order()
        for i, entry in enumerate(self.schedule):
            if not 0 <= entry.layer < len(self.blocks):
                raise ValueError(f"schedule entry {i} names layer {entry.layer}; there are {len(self.blocks)}")
            if entry.cache is not None:
                owner = self.schedule[entry.cache] if 0 <= entry.cache < i else None
                if owner is None or owner.cache is not None:
                    raise ValueError(f"schedule entry {i} reads cache {entry.cache}, which is no earlier owning entry")
                for which in (owner.layer, entry.layer):
                    mixer = self.blocks[which].mixer
                    if not mixer.shares_cache:
                        raise ValueError(f"schedule entry {i} reads the cache of entry {entry.cache}, but the mixer of layer "
                                         f"{which} ({type(mixer).__name__}) keeps a summary of the past that has moved on "
                                         "when a reader runs: give the entry a cache of its own")
        self.embedding_norm = build_part("norm", spec.embedding_norm, runtime)
        self.embedding = None
        self.positions = None  # learned absolute positions [max_context, hidden], where the architecture has them
        self.head = None
        self.joins: Dict[str, Optional[torch.Tensor]] = {e.join: None for e in self.schedule if getattr(e, "join", None)}

    # ------------------------------------------------------------------ weights

    def params(self) -> Dict[str, Param]:
        s = self.spec
        out = {s.embedding_name: Param((s.vocab_size, s.hidden_size))}
        out.update(norm_params(self.final_norm, s.final_norm_name))
        if s.head_name is not None:
            out[s.head_name] = Param((s.vocab_size, s.hidden_size), optional=s.head_optional)
        if s.position_table_name is not None:
            out[s.position_table_name] = Param((s.max_context, s.hidden_size))
        if self.embedding_norm is not None:
            out.update(norm_params(self.embedding_norm, s.embedding_norm_name))
        for name in self.joins:
            out[name] = Param((s.hidden_size, 2 * s.hidden_size))
        for block in self.blocks:
            out.update(block.params())
        return out

    def load(self, get: Callable[[str], torch.Tensor], has: Callable[[str], bool] = lambda name: True) -> None:
        s = self.spec
        self.embedding = get(s.embedding_name)
        load_norm(self.final_norm, s.final_norm_name, get)
        if s.position_table_name is not None:
            self.positions = get(s.position_table_name)
        if self.embedding_norm is not None:
            load_norm(self.embedding_norm, s.embedding_norm_name, get)
        self.head = get(s.head_name) if s.head_name is not None and has(s.head_name) else self.embedding
        for name in self.joins:
            self.joins[name] = get(name)
        for block in self.blocks:
            block.load(get)

    # ------------------------------------------------------------------ compute

    def cache_specs(self):
        """For each schedule entry that owns a cache: what its mixer needs (or None)."""
        return [self.blocks[e.layer].mixer.cache() if e.cache is None else None for e in self.schedule]

    def forward(self, ctx, caches) -> torch.Tensor:
        """Runs the tokens of ``ctx`` and returns float32 logits ``[len(ctx.logit_rows), vocab]``."""
        ops = self.rt.ops
        # A decode step is a chain of small operations; kernels that can run such a chain as one launch are told
        # where it begins and ends, and it is cut before any block that has not declared itself safe inside one.
        chained = ctx.decode_only and hasattr(ops, "chain_begin") and ops.chain_begin(ctx.num_tokens)
        try:
            return self._forward(ctx, caches, chained)
        finally:
            if chained:
                ops.chain_end()

    def _forward(self, ctx, caches, chained: bool) -> torch.Tensor:
        ops = self.rt.ops
        spec = self.spec
        h = ops.embedding(ctx.token_ids, self.embedding)
        if spec.embedding_multiplier is not None:
            h = ops.scale_cap(h, scale=spec.embedding_multiplier)
        if self.positions is not None:
            h = ops.add_rows(h, self.positions, ctx.positions)
        if self.embedding_norm is not None:
            h = self.embedding_norm.forward(h, out_dtype=torch.float32)  # the residual stream stays float32
        # entries that add the embedding's output again read a copy of it (the blocks add into h in place)
        first = None
        if any(entry.add_embedding for entry in self.schedule):
            if chained:
                ops.chain_flush()
            first = h.clone()
        # entries that join it to the stream read both side by side, in the compute dtype: the embedding's half is
        # written once, the stream's half in front of every such entry
        joined = None
        if self.joins:
            joined = torch.empty((h.shape[0], 2 * spec.hidden_size), dtype=self.rt.dtype, device=h.device)
            ops.round_rows(h, joined[:, spec.hidden_size :])
        for i, entry in enumerate(self.schedule):
            owner = i if entry.cache is None else entry.cache
            block = self.blocks[entry.layer]
            if chained and not block.chain_safe:
                ops.chain_flush()
            if entry.add_embedding:
                h = ops.scaled_add(h, first, None, None, None, 1.0)
            if joined is not None and entry.join is not None:
                ops.round_rows(h, joined[:, : spec.hidden_size])
                h = ops.linear(joined, self.joins[entry.join], out_dtype=torch.float32)
            h = block.forward(h, ctx, caches[owner], write=entry.cache is None)
        if chained and not getattr(self.final_norm, "chain_safe", False):
            ops.chain_flush()
        if ctx.num_logit_rows == 0:
            return torch.empty((0, self.spec.vocab_size), dtype=torch.float32, device=h.device)
        if hasattr(self.final_norm, "lazy"):
            x = self.final_norm.lazy(h, rows=ctx.logit_rows)
        else:
            x = self.final_norm.forward(h, rows=ctx.logit_rows)
        logits = project(self.rt, x, self.head, out_dtype=torch.float32)
        if spec.logit_scale is not None or spec.logit_softcap is not None:
            logits = ops.scale_cap(logits, scale=1.0 if spec.logit_scale is None else spec.logit_scale,
                                   cap=spec.logit_softcap or 0.0)
        return logits
