"""A decoder assembled from a :class:`ModelSpec`: embedding, layers run in the schedule's order,
final norm and head on the rows whose logits are wanted.

This is the one forward pass of the package (the reference has three, one per batch shape:
ampere_kv/runner.py:219-290).  It runs exactly the tokens of the step's batch, reads earlier
tokens only through the cache, and returns float32 logits for ``ctx.logit_rows``
(the reference returns the last position only, runner.py:293-297).
"""

from __future__ import annotations

from dataclasses import replace

import torch

from ..config.spec import ModelSpec
from ..kernels import ops
from ..parts import (attention, block, embedding, feed_forward, gated_delta, hyper, latent_attention,  # noqa: F401
                     linear_memory, norm, parallel, position, rotary_attention, routed_experts,
                     scored_attention, state_space, stream_update)   # (importing them registers the built-in kinds)
from ..parts.base import BLOCKS, EMBEDDINGS, HEADS, NORMS, STREAM_UPDATES, Block, CacheSpec, ParamSpec, build_part


class DecoderModel:
    def __init__(self, spec: ModelSpec, *, dtype: torch.dtype, device: torch.device | str):
        spec.validate()
        if dtype not in (torch.float32, torch.bfloat16):
            raise ValueError(f"compute dtype must be float32 or bfloat16, got {dtype}")
        self.spec = spec
        self.dtype = dtype
        self.device = torch.device(device)
        kw = dict(hidden_size=spec.hidden_size, dtype=dtype, device=self.device)
        self.embedding = build_part(EMBEDDINGS, spec.embedding, **kw)
        self.blocks = [BLOCKS.get(layer.block)(layer, **kw) for layer in spec.layers]
        self.walk_entry = None if spec.walk_entry is None else build_part(STREAM_UPDATES, spec.walk_entry, **kw)
        self.final_norm = build_part(NORMS, spec.final_norm, **kw)
        self.head = build_part(HEADS, spec.head, **kw)
        self.loaded = False

    # ------------------------------------------------------------------ tensors

    def _parts(self):
        """Every part, a part's own children after it."""
        def walk(part):
            yield part
            for child in part.children():
                yield from walk(child)
        yield from walk(self.embedding)
        for blk in self.blocks:
            for part in blk.parts():
                yield from walk(part)
        if self.walk_entry is not None:
            yield from walk(self.walk_entry)
        yield from walk(self.final_norm)
        yield from walk(self.head)

    def param_specs(self) -> dict[str, ParamSpec]:
        """Every tensor of the checkpoint by its full name."""
        out: dict[str, ParamSpec] = {}
        for part in self._parts():
            for local, ps in part.param_specs().items():
                name = f"{part.spec.prefix}.{local}" if part.spec.prefix else local
                if name in out and out[name] != ps:
                    raise ValueError(f"tensor {name} is declared twice with different shapes")
                out[name] = ps
        for name, shape in self.spec.unused_tensors:
            out.setdefault(name, ParamSpec(tuple(shape), kind="vector", optional=True))
        return out

    def load_tensors(self, tensors: dict[str, torch.Tensor]) -> None:
        """``tensors``: full name -> tensor, already validated, cast and on the device."""
        for part in self._parts():
            local = {}
            for name in part.param_specs():
                full = f"{part.spec.prefix}.{name}" if part.spec.prefix else name
                if full in tensors:
                    local[name] = tensors[full]
            part.load(local)
        self.head.tie(self.embedding)
        self.loaded = True

    @property
    def graph_safe(self) -> bool:
        """Every part only enqueues device work that depends on the batch layout alone."""
        return all(getattr(part, "graph_safe", False) for part in self._parts())

    # ------------------------------------------------------------------ cache needs

    def cache_specs(self) -> list[CacheSpec]:
        """One per schedule position, and behind them one for the embedding if it keeps something per request (the
        cache manager treats it as one more position without pages)."""
        specs = [self.blocks[e.layer].cache_spec() for e in self.spec.schedule]
        # a position whose pages others read keeps them as far back as any of them looks; those name the same cache
        for pos, entry in enumerate(self.spec.schedule):
            if entry.cache_of is not None:
                specs[entry.cache_of] = specs[entry.cache_of].covering(specs[pos])
        for pos, entry in enumerate(self.spec.schedule):
            if entry.cache_of is not None and specs[pos].stored() == specs[entry.cache_of].stored():
                specs[pos] = replace(specs[entry.cache_of], state_shape=specs[pos].state_shape)
        own = self.embedding.cache_spec()
        if own.kind != "none":
            raise ValueError("an embedding keeps a state per request at most, no pages")
        return specs + [own] if own.state_shape else specs

    def q_tile(self) -> int:
        """Query tokens per attention tile of the batch layout: what every mixer with a preference asks for, if they
        agree."""
        wishes = {m.preferred_q_tile() for blk in self.blocks for m in [getattr(blk, "mixer", None)]
                  if m is not None and m.preferred_q_tile() is not None}
        return wishes.pop() if len(wishes) == 1 else ops.ATTENTION_Q_TILE

    def cache_of(self) -> list[int | None]:
        own = [None] if self.embedding.cache_spec().state_shape else []
        return [e.cache_of for e in self.spec.schedule] + own

    # ------------------------------------------------------------------ forward

    @torch.no_grad()
    def forward(self, ctx, cache_views) -> torch.Tensor | None:
        """Run the step's tokens through the schedule; logits [wanted, vocab] float32, or None if none wanted."""
        ops.stream_begin_step(self.device)
        if getattr(ctx, "shared", None):
            ctx.shared.clear()
        positions = len(self.spec.schedule)
        if len(cache_views) > positions:
            hidden = self.embedding.forward(ctx.token_ids, ctx, cache=cache_views[positions])
        else:
            hidden = self.embedding.forward(ctx.token_ids, ctx)
        # a schedule that sends the stream through layers again adds the embedding's output before each such pass, or
        # gives it to what stands before a pass
        start = None
        if any(e.add_embedding or e.begins_walk is not None for e in self.spec.schedule):
            start = hidden.clone()
        delta = None
        if self.spec.streams:
            hidden = ops.hyper_expand(hidden, self.spec.streams)
        for pos, entry in enumerate(self.spec.schedule):
            if entry.add_embedding:
                delta = ops.stream_add(hidden, start, delta)
            if entry.begins_walk is not None:
                hidden, delta = self.walk_entry.forward(hidden, [delta], ctx, start=start, walk=entry.begins_walk)
            hidden, delta = self.blocks[entry.layer].forward(hidden, delta, ctx, cache_views[pos])
        if ctx.num_logit_rows == 0:
            return None
        if self.spec.streams:
            # the copies' sum, with the last sublayer's result written on the way
            hidden, delta = ops.hyper_collapse(hidden, delta), None
        normed = Block.run_norm(self.final_norm, hidden, delta, ctx, rows=ctx.logit_rows)
        return self.head.forward(normed)
