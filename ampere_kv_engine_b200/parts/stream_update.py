"""Updates of the residual stream itself, beside the branches that add to it.

``token_gate``: after a layer's branches, a small gated branch that the token's id steers:

    g = gelu_tanh(W_gate x) * e;   y = W_proj g;   x <- x + y / sqrt(mean(y^2) + eps) * norm

with e a run of ``dim`` columns of the row that the token's id picks from a table (a layer has its own run; the table is
one tensor of the model).  x, the whole stream, is what the first product reads, so the branches' results join the stream
here, in the kernel that also rounds the copy for the product (``ops.stream_sum``); y joins through its norm in the kernel
of whatever norm comes next (``ops.NormedBranch``).

``concat_projection``: before a pass through a run of layers,

    x <- W_in [x | x0] + step[t]

with x0 the embedding's output and t the number of the pass.  The product leaves its float32 accumulators, which are the
new stream.
"""

from __future__ import annotations

import torch

from ..kernels import ops
from .base import ParamSpec, StreamUpdate, register_stream_update


@register_stream_update("token_gate")
class TokenGate(StreamUpdate):
    """params: ``dim``, ``runs`` (how many runs of ``dim`` columns the table has), ``run`` (which one is this layer's),
    ``vocab_size``, ``eps``, ``names`` (full tensor names of table, gate, proj, norm: the table is shared by layers, so
    the part has no prefix)."""

    graph_safe = True

    def __init__(self, spec, **kw):
        super().__init__(spec, **kw)
        p = spec.params
        self.dim, self.runs, self.run = int(p["dim"]), int(p["runs"]), int(p["run"])
        self.vocab_size, self.eps = int(p["vocab_size"]), float(p["eps"])
        if self.dim <= 0 or not 0 <= self.run < self.runs:
            raise ValueError(f"token_gate: run {self.run} of {self.runs} runs of {self.dim} columns")
        self.names = dict(p["names"])
        self.table = self.w_gate = self.w_proj = self.norm_weight = None

    def param_specs(self):
        n, h = self.names, self.hidden_size
        return {n["table"]: ParamSpec((self.vocab_size, self.runs * self.dim)), n["gate"]: ParamSpec((self.dim, h)),
                n["proj"]: ParamSpec((h, self.dim)), n["norm"]: ParamSpec((h,), kind="vector", init="norm")}

    def load(self, tensors):
        n = self.names
        self.table, self.w_gate = tensors[n["table"]].contiguous(), tensors[n["gate"]].contiguous()
        self.w_proj, self.norm_weight = tensors[n["proj"]].contiguous(), tensors[n["norm"]].float().contiguous()

    def forward(self, hidden, pending, ctx, *, start=None, walk=0):
        status = getattr(ctx, "status", None)
        x = ops.stream_sum(hidden, pending, copy_dtype=self.dtype)
        z = ops.linear(x, self.w_gate, status=status)
        g = ops.token_gate(z, ctx.token_ids, self.table, self.run * self.dim, sampled=getattr(ctx, "sampled", None),
                           status=status)
        y = ops.linear(g, self.w_proj, out_dtype=torch.float32, status=status)
        return hidden, ops.NormedBranch(y, self.norm_weight, self.eps)


@register_stream_update("concat_projection")
class ConcatProjection(StreamUpdate):
    """params: ``times`` (passes), ``names`` (local tensor names of the matrix ``in`` [width, 2 width] and of the rows
    ``step`` [times, width])."""

    graph_safe = True

    NAMES = {"in": "in.weight", "step": "step.weight"}

    def __init__(self, spec, **kw):
        super().__init__(spec, **kw)
        self.times = int(spec.params["times"])
        self.names = dict(self.NAMES, **(spec.params.get("names") or {}))
        self.w_in = self.step = None

    def param_specs(self):
        h, n = self.hidden_size, self.names
        return {n["in"]: ParamSpec((h, 2 * h)), n["step"]: ParamSpec((self.times, h), kind="vector", init="around_zero")}

    def load(self, tensors):
        self.w_in = tensors[self.names["in"]].contiguous()
        self.step = tensors[self.names["step"]].float().contiguous()

    def forward(self, hidden, pending, ctx, *, start=None, walk=0):
        ops.stream_sum(hidden, pending)
        both = ops.stream_concat(hidden, start, self.dtype)
        hidden = ops.linear(both, self.w_in, out_dtype=torch.float32, status=getattr(ctx, "status", None))
        return ops.stream_row_add(hidden, self.step[walk]), None
