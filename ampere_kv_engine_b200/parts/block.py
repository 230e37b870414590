"""Arrangements of a layer's parts around the residual stream.

``prenorm``: ``h += mixer(norm1(h)); h += feed_forward(norm2(h))`` (ampere_kv/runner.py:117-121
and 156-179).  The residual stream is float32; each branch output is handed to the next norm
as a pending ``delta`` so that the sum and the norm are one kernel.  On decode steps the branch's
last product may add to the stream itself and the next product apply the norm (``Summed``,
``LazyNorm``): then no kernel stands between the two products.  ``postnorm``: the norms sit on the
branches' outputs only.  ``sandwich``: a norm before and after every branch.  ``shared_norm``: one norm, whose output
mixer and feed-forward both read.
"""

from __future__ import annotations

import torch

from ..kernels import ops
from .base import NORMS, STREAM_UPDATES, Block, register_block


@register_block("prenorm")
class PreNormBlock(Block):
    """roles: ``mixer_norm``, ``mixer``, ``feed_forward_norm``, ``feed_forward``.  A layer spec without a
    feed-forward makes a layer of the mixer branch alone."""

    def __init__(self, layer, **kw):
        super().__init__(layer, **kw)
        self.mixer_norm = self.build_role("mixer_norm")
        self.mixer = self.build_role("mixer")
        self.feed_forward = self.feed_forward_norm = None
        if layer.feed_forward is not None:
            self.feed_forward_norm = self.build_role("feed_forward_norm")
            self.feed_forward = self.build_role("feed_forward")

    def forward(self, hidden, delta, ctx, cache):
        x = self.run_norm(self.mixer_norm, hidden, delta, ctx, consumer=self.mixer)
        attn = self.run_branch(self.mixer, hidden, x, ctx, cache)
        if self.feed_forward is None:
            return hidden, attn
        x = self.run_norm(self.feed_forward_norm, hidden, attn, ctx, consumer=self.feed_forward)
        return hidden, self.run_branch(self.feed_forward, hidden, x, ctx)


@register_block("postnorm")
class PostNormBlock(Block):
    """``h += norm1(mixer(h)); h += norm2(feed_forward(h))``: the branches read the stream itself and each norm sits
    on its branch's output.  roles as ``prenorm``; the norms must offer ``add_normed``.  The stream is float32; in
    bfloat16 every ``add_normed`` also leaves the stream's rounded copy, which the next branch reads and which
    travels to the next block as an ``ops.Mirrored`` in place of a pending delta."""

    def __init__(self, layer, **kw):
        super().__init__(layer, **kw)
        self.mixer = self.build_role("mixer")
        self.mixer_norm = self.build_role("mixer_norm")
        self.feed_forward = self.feed_forward_norm = None
        if layer.feed_forward is not None:
            self.feed_forward = self.build_role("feed_forward")
            self.feed_forward_norm = self.build_role("feed_forward_norm")
        for norm in (self.mixer_norm, self.feed_forward_norm):
            if norm is not None and not hasattr(norm, "add_normed"):
                raise ValueError(f"block kind 'postnorm': norm kind {norm.spec.kind!r} cannot norm a branch's output")

    def forward(self, hidden, delta, ctx, cache):
        if isinstance(delta, ops.Mirrored) and delta.hidden is hidden:
            x = delta.copy
        else:
            if isinstance(delta, ops.PendingPhases):
                delta.launch()
                delta = None
            if isinstance(delta, ops.NormedBranch):
                delta.apply(hidden)
                delta = None
            if delta is not None and not isinstance(delta, (ops.Summed, ops.Mirrored)):
                raise ValueError("block kind 'postnorm' follows a block that leaves its last branch unadded; "
                                 "put a norm that adds it between them")
            x = ops.stream_copy(hidden, self.dtype)
        x = self.mixer_norm.add_normed(hidden, self.mixer.forward(x, ctx, cache), ctx)
        if self.feed_forward is not None:
            # a feed-forward whose result is still a sum of rows leaves the sum to a norm that can do it
            if getattr(self.feed_forward, "defers_sum", False) and getattr(self.feed_forward_norm, "takes_parts", False):
                branch = self.feed_forward.forward(x, ctx, defer_sum=True)
            else:
                branch = self.feed_forward.forward(x, ctx)
            x = self.feed_forward_norm.add_normed(hidden, branch, ctx)
        return hidden, ops.Mirrored(hidden, x)


@register_block("sandwich")
class SandwichBlock(Block):
    """``h += norm1b(mixer(norm1(h))); h += norm2b(feed_forward(norm2(h)))``: a norm on either side of every branch (a
    constant on the branch's normed result is a ``factor`` of its out-norm).  roles as ``prenorm`` and beside them
    ``mixer_out_norm`` and ``feed_forward_out_norm``, which must offer ``of_branch``; without a feed-forward the layer is
    the mixer branch alone.  A branch's result stays a pending ``ops.NormedBranch`` until the next norm: that one
    kernel norms the branch, adds it to the float32 stream and norms the stream."""

    def __init__(self, layer, **kw):
        super().__init__(layer, **kw)
        self.mixer_norm = self.build_role("mixer_norm")
        self.mixer = self.build_role("mixer")
        self.mixer_out_norm = self.build_role("mixer_out_norm", NORMS)
        self.feed_forward = self.feed_forward_norm = self.feed_forward_out_norm = None
        if layer.feed_forward is not None:
            self.feed_forward_norm = self.build_role("feed_forward_norm")
            self.feed_forward = self.build_role("feed_forward")
            self.feed_forward_out_norm = self.build_role("feed_forward_out_norm", NORMS)
        for norm in (self.mixer_out_norm, self.feed_forward_out_norm):
            if norm is not None and not hasattr(norm, "of_branch"):
                raise ValueError(f"block kind 'sandwich': norm kind {norm.spec.kind!r} cannot norm a branch's output")

    def forward(self, hidden, delta, ctx, cache):
        x = self.run_norm(self.mixer_norm, hidden, delta, ctx, consumer=self.mixer)
        branch = self.mixer_out_norm.of_branch(self.mixer.forward(x, ctx, cache))
        if self.feed_forward is None:
            return hidden, branch
        x = self.run_norm(self.feed_forward_norm, hidden, branch, ctx, consumer=self.feed_forward)
        # a feed-forward whose result is still a sum of rows leaves the sum to the kernel that norms it
        if getattr(self.feed_forward, "defers_sum", False):
            return hidden, self.feed_forward_out_norm.of_branch(self.feed_forward.forward(x, ctx, defer_sum=True))
        return hidden, self.feed_forward_out_norm.of_branch(self.feed_forward.forward(x, ctx))


@register_block("shared_norm")
class SharedNormBlock(Block):
    """``h += mixer(n) + feed_forward(n)`` with ``n = norm(h)``: one norm, both branches read its output and their results
    join the stream together.  roles: ``mixer_norm``, ``mixer``, ``feed_forward`` (or none: the mixer branch alone) and
    ``after`` (a stream update that acts once the branches are in the stream; or none).

    Where both branches let someone else run their first and last products (``in_projection``, ``heads_forward``,
    ``out_projection``; neither product with a bias), the layer runs two products in all: one makes what both branches
    need of n, and one takes both branches' results, laid side by side, into the stream."""

    def __init__(self, layer, **kw):
        super().__init__(layer, **kw)
        roles = layer.roles()
        self.mixer_norm = self.build_role("mixer_norm")
        self.mixer = self.build_role("mixer")
        self.feed_forward = self.build_role("feed_forward") if layer.feed_forward is not None else None
        self.after = self.build_role("after", STREAM_UPDATES) if "after" in roles else None
        self.joined = None          # made at the first step: (first products, split, last products, split), or False

    def _join(self):
        parts = (self.mixer, self.feed_forward)
        self.joined = False
        if all(getattr(p, "joinable", None) is not None and p.joinable() for p in parts):
            w_in, w_out = [p.in_projection()[0] for p in parts], [p.out_projection()[0] for p in parts]
            first, last = torch.cat(w_in, dim=0).contiguous(), torch.cat(w_out, dim=1).contiguous()
            rows, cols = w_in[0].shape[0], w_out[0].shape[1]
            self.joined = (first, rows, last, cols)
            # the parts keep views of the joined matrices, not copies of their own
            self.mixer.adopt(first[:rows], last[:, :cols])
            self.feed_forward.adopt(first[rows:], last[:, cols:])

    def forward(self, hidden, delta, ctx, cache):
        x = self.run_norm(self.mixer_norm, hidden, delta, ctx)
        if self.joined is None and self.feed_forward is not None:
            self._join()
        if self.joined:
            first, rows, last, cols = self.joined
            both = ops.linear(x, first, status=ctx.status)
            out = torch.empty((x.shape[0], last.shape[1]), dtype=self.dtype, device=x.device)
            self.mixer.heads_forward(x, ctx, cache, projected=(both, 0), out=(out, 0))
            self.feed_forward.heads_forward(x, ctx, projected=(both, rows), out=(out, cols))
            branch = ops.linear_into_residual(out, last, hidden, status=ctx.status)
            branches = [branch if branch is not None else ops.linear(out, last, partial_ok=True, status=ctx.status)]
        else:
            branches = [self.run_branch(self.mixer, hidden, x, ctx, cache)]
            if self.feed_forward is not None:
                if getattr(self.feed_forward, "defers_sum", False):
                    branches.append(self.feed_forward.forward(x, ctx, defer_sum=True))
                else:
                    branches.append(self.run_branch(self.feed_forward, hidden, x, ctx))
        if self.after is not None:
            return self.after.forward(hidden, branches, ctx)
        if len(branches) == 1:
            return hidden, branches[0]
        ops.stream_sum(hidden, branches)
        return hidden, None
