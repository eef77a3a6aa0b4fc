"""The generic decoder that every registered architecture is built as.

Embedding (plus a row picked by a hash of the token in front and the token, if the architecture has such a table; times ``ModelSpec.embedding_multiplier`` if the architecture has one, plus a learned position vector
and through a norm if it has those), the blocks of
``ModelSpec.layers`` in the order of ``ModelSpec.schedule`` (a list that may name a layer twice, let an
entry read another entry's cache, or have the embedding's output added again or joined to the stream by a matrix in
front of an entry, or be followed by a weighted sum of the embedding's output and of all entries' results so far), the
final norm on the rows whose logits are wanted, the head, and the
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
from ..parts.base import Param, Runtime, StateSpec, build_part, load_norm, norm_params, project
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
        self.bigram = None  # the second table [buckets + 1, hidden], where the architecture has one
        self.averages: Dict[str, Optional[torch.Tensor]] = {e.average: None for e in self.schedule if getattr(e, "average", None)}
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
        if s.bigram is not None:
            out[s.bigram.name] = Param((s.bigram.buckets + 1, s.hidden_size))
        for i, entry in enumerate(self.schedule):
            if getattr(entry, "average", None):
                out[entry.average] = Param((i + 2,), role="vector", mean=1.0 / (i + 2))
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
        if s.bigram is not None:
            self.bigram = get(s.bigram.name)
        for name in self.averages:
            self.averages[name] = get(name)
        for name in self.joins:
            self.joins[name] = get(name)
        for block in self.blocks:
            block.load(get)

    # ------------------------------------------------------------------ compute

    def cache_specs(self):
        """For each schedule entry that owns a cache: what its mixer needs (or None). Behind those, where the embedding
        looks at the token in front: the state that holds it, one integer per request, the last token plus one (0: no
        token yet, as admission leaves it)."""
        specs = [self.blocks[e.layer].mixer.cache() if e.cache is None else None for e in self.schedule]
        return specs if self.spec.bigram is None else specs + [StateSpec((1,), torch.int32)]

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
        # Where entries are followed by an average over all results so far, the results lie in one buffer: entry e's layer
        # adds in place into the rows [e + 1], which the average in front of it has written, and so leaves its result there.
        history = None
        if self.averages:
            words = ctx.num_tokens * spec.hidden_size
            pitch = -(-words // 64) * 64  # every entry's rows start on 256 bytes, as rows of their own would
            history = torch.empty((len(self.schedule) + 1, pitch), dtype=torch.float32, device=self.embedding.device)
            history = history[:, :words].view(-1, ctx.num_tokens, spec.hidden_size)
        started = False  # whether the embedding's output lies in the first two rows of the buffer already
        if spec.bigram is not None:
            b = spec.bigram
            started = history is not None and spec.embedding_multiplier is None and self.positions is None and self.embedding_norm is None
            h = ops.bigram_embedding(ctx.token_ids, self.embedding, self.bigram, b.mul_prev, b.mul_cur, caches[len(self.schedule)].state,
                                     ctx.cu_seqlens, ctx.seq_of_token, ctx.slots, out=history[:2] if started else None)
        else:
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
        if history is not None and not started:
            if chained:
                ops.chain_flush()
            history[:2] = h
            h = history[1]
        normed = None
        final_rows = None  # the rows the final norm wants, once an average has picked them
        last = len(self.schedule) - 1
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
            h = block.forward(h, ctx, caches[owner], write=entry.cache is None, **({} if normed is None else dict(normed=normed)))
            normed = None
            if history is not None:
                h, normed, final_rows = self._behind(i, h, history, ctx, i == last, chained)
        if chained and not getattr(self.final_norm, "chain_safe", False):
            ops.chain_flush()
        if ctx.num_logit_rows == 0:
            return torch.empty((0, self.spec.vocab_size), dtype=torch.float32, device=h.device)
        if normed is not None:
            x = normed
        elif final_rows is not None:  # h is those rows already
            x = self.final_norm.lazy(h) if hasattr(self.final_norm, "lazy") else self.final_norm.forward(h)
        elif hasattr(self.final_norm, "lazy"):
            x = self.final_norm.lazy(h, rows=ctx.logit_rows)
        else:
            x = self.final_norm.forward(h, rows=ctx.logit_rows)
        logits = project(self.rt, x, self.head, out_dtype=torch.float32)
        if spec.logit_scale is not None or spec.logit_softcap is not None:
            logits = ops.scale_cap(logits, scale=1.0 if spec.logit_scale is None else spec.logit_scale,
                                   cap=spec.logit_softcap or 0.0)
        return logits

    def _behind(self, i, h, history, ctx, last: bool, chained: bool):
        """What goes on behind entry ``i`` where results are kept: (stream, the next norm's output where it is made in the
        same pass, the rows of the final norm where ``stream`` is those rows alone). h is the entry's result."""
        ops = self.rt.ops
        entry = self.schedule[i]
        averages = bool(getattr(entry, "average", None))
        in_place = h.data_ptr() == history[i + 1].data_ptr()
        if chained and not (in_place and averages):
            ops.chain_flush()
        if not in_place:  # (a block that did not add in place)
            history[i + 1].copy_(h)
        following = self.schedule[i + 1] if not last else None
        plain = following is None or not (following.add_embedding or following.join)
        norm = self.final_norm if last else self.blocks[following.layer].mixer_norm
        takes = plain and (last or self.blocks[following.layer].takes_ready_norm) and getattr(norm.spec, "kind", None) == "rmsnorm"
        rows = ctx.logit_rows if last else None
        if not averages:
            if last:
                return h, None, None
            history[i + 2].copy_(h)  # the next layer adds into rows of its own
            return history[i + 2], None, None
        if last and ctx.num_logit_rows == 0:
            return h, None, None  # nobody reads it
        h, normed = ops.depth_average(history, i + 2, self.averages[entry.average], None if last else history[i + 2], rows=rows,
                                      norm=(norm.weight, norm.spec.eps, norm.spec.zero_centered, self.rt.dtype) if takes else None)
        return h, normed, rows
