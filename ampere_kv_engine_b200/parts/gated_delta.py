"""The gated delta rule: a linear-attention mixer whose memory is one matrix per head, carried from token to token.

    q, k, v   = silu(conv(W_q x)), silu(conv(W_k x)), silu(conv(W_v x))     short causal convolutions over time, per
                                                                            channel, zeros before the sequence's start
    q, k     <- q / sqrt(|q|^2 + unit_eps) * dim^-1/2,  k / sqrt(|k|^2 + unit_eps)          per head
    beta      = sigmoid(W_b x);   decay = exp(-exp(rate_log) * softplus(W_a x + step_bias))  one of each per head
    S        <- decay * S;   u = beta * (v - S^T k);   S <- S + k u^T;   o = S^T q           per head, S: [dim, vdim]
    y         = W_o concat_h( o_h / sqrt(mean(o_h^2) + norm_eps) * norm * silu(W_g x)_h )

Options: ``decay="channel"``: a decay per head and key channel, ``decay = exp(-exp(rate_log_h) * softplus(. + step_bias))``
laid out heads x dim, each multiplying its row of S.  ``low_rank``: step and gate come through two matrices each,
``W_a2 (W_a1 x)`` and ``W_g2 (W_g1 x)``; the inner widths are the checkpoint's.  ``gate="sigmoid"``.

``num_kv_heads`` heads of q and k serve ``num_heads`` heads of v in groups.  What a request carries from step to
step is float32 and lives in its state slot: every head's S and the last ``taps - 1`` inputs of the three
convolutions.  One product makes all projections of a token; a row-wise kernel (``ops.delta_prep``) turns them into
float32 q, k, v, beta and decay; one block per (sequence, head) walks the step's tokens of that sequence in order
(``ops.delta_scan``), so the state after a token is the same however the tokens were cut into steps.
"""

from __future__ import annotations

import torch

from ..kernels import ops
from .base import FREE_SIZE, CacheSpec, Mixer, ParamSpec, register_mixer


@register_mixer("gated_delta")
class GatedDelta(Mixer):
    """params: ``num_heads``, ``num_kv_heads``, ``head_dim`` (q / k width), ``v_dim``, ``taps`` (of the convolutions;
    1: none), ``unit_eps``, ``norm_eps``, ``decay`` (``"head"`` or ``"channel"``), ``low_rank`` (None, or a dict with
    ``step`` and ``gate``, the inner widths that random weights take: a checkpoint brings its own), ``gate`` (``"silu"``
    or ``"sigmoid"``), ``out_scale`` (a factor on the result, applied before the output projection), ``names`` (local
    tensor names of q, k, v, their convolutions, beta, step, rate_log, step_bias, gate, norm, out; with ``low_rank``
    step_in, step_out, gate_in, gate_out in place of step and gate)."""

    graph_safe = True
    #: ``heads_forward(..., out=)`` writes its result into columns of a wider matrix
    writes_into = True

    NAMES = {"q": "q_proj.weight", "k": "k_proj.weight", "v": "v_proj.weight", "q_conv": "q_conv.weight",
             "k_conv": "k_conv.weight", "v_conv": "v_conv.weight", "beta": "b_proj.weight", "step": "a_proj.weight",
             "rate_log": "A_log", "step_bias": "dt_bias", "gate": "g_proj.weight", "norm": "o_norm.weight",
             "out": "o_proj.weight", "step_in": "a_in.weight", "step_out": "a_out.weight", "gate_in": "g_in.weight",
             "gate_out": "g_out.weight"}

    def __init__(self, spec, **kw):
        super().__init__(spec, **kw)
        p = spec.params
        self.num_heads, self.num_kv_heads = int(p["num_heads"]), int(p["num_kv_heads"])
        self.head_dim, self.v_dim, self.taps = int(p["head_dim"]), int(p["v_dim"]), int(p["taps"])
        if self.num_heads <= 0 or self.num_kv_heads <= 0 or self.num_heads % self.num_kv_heads:
            raise ValueError(f"gated_delta: {self.num_heads} heads are not a multiple of {self.num_kv_heads} q/k heads")
        if ops.delta_shape(self.head_dim, self.v_dim) is None:
            raise ValueError(f"gated_delta: q/k width {self.head_dim} with value width {self.v_dim} is outside what "
                             f"the kernel takes (each up to {ops.DELTA_MAX_DIM})")
        if not 1 <= self.taps <= ops.DELTA_MAX_TAPS:
            raise ValueError(f"gated_delta: {self.taps} taps outside what the kernel takes (1 to {ops.DELTA_MAX_TAPS})")
        self.unit_eps = float(p.get("unit_eps", 1e-6))
        self.norm_eps = float(p.get("norm_eps", 1e-6))
        self.out_scale = float(p.get("out_scale", 1.0))
        self.gate = str(p.get("gate", "silu"))
        self.low_rank = dict(p["low_rank"]) if p.get("low_rank") else None
        if self.gate not in ops.DELTA_GATES or p.get("decay", "head") not in ("head", "channel"):
            raise ValueError(f"gated_delta: gate {self.gate!r} or decay {p.get('decay')!r} is not known")
        self.channel_decay = p.get("decay", "head") == "channel"
        if self.channel_decay and self.low_rank is None:
            raise ValueError("gated_delta: decays per channel come through a low-rank step")
        self.names = dict(self.NAMES, **(p.get("names") or {}))
        self.qk_width = self.num_kv_heads * self.head_dim
        self.v_width = self.num_heads * self.v_dim
        self.channels = 2 * self.qk_width + self.v_width            # what the convolutions run over
        # floats of all heads' S per request, and of the whole state with the convolutions' inputs behind it
        self.memory, self.state_floats = ops.delta_state_floats(self.num_heads, self.num_kv_heads, self.head_dim,
                                                                self.v_dim, self.taps)
        self.steps = self.num_heads * (self.head_dim if self.channel_decay else 1)
        self.w_in = self.w_o = self.conv = self.rate_log = self.step_bias = self.norm_weight = self.w_mid = None
        self.mid_width = self.qkv_off = 0       # columns of the inner low-rank values, where q, k, v begin

    def cache_spec(self) -> CacheSpec:
        return CacheSpec(kind="none", state_shape=(self.state_floats,))

    def param_specs(self):
        h, n = self.hidden_size, self.names
        if self.low_rank is None:
            step, gate = {n["step"]: ParamSpec((self.num_heads, h))}, {n["gate"]: ParamSpec((self.v_width, h))}
        else:
            a, g = int(self.low_rank["step"]), int(self.low_rank["gate"])
            step = {n["step_in"]: ParamSpec((FREE_SIZE, h), free_size=a),
                    n["step_out"]: ParamSpec((self.steps, FREE_SIZE), free_size=a)}
            gate = {n["gate_in"]: ParamSpec((FREE_SIZE, h), free_size=g),
                    n["gate_out"]: ParamSpec((self.v_width, FREE_SIZE), free_size=g)}
        return {
            n["q"]: ParamSpec((self.qk_width, h)), n["q_conv"]: ParamSpec((self.qk_width, self.taps), kind="vector", init="unit_interval"),
            n["k"]: ParamSpec((self.qk_width, h)), n["k_conv"]: ParamSpec((self.qk_width, self.taps), kind="vector", init="unit_interval"),
            n["v"]: ParamSpec((self.v_width, h)), n["v_conv"]: ParamSpec((self.v_width, self.taps), kind="vector", init="unit_interval"),
            n["beta"]: ParamSpec((self.num_heads, h)),
            n["rate_log"]: ParamSpec((self.num_heads,), kind="vector", init="around_zero"),
            n["norm"]: ParamSpec((self.v_dim,), kind="vector", init="norm"),
            **step,
            n["step_bias"]: ParamSpec((self.steps,), kind="vector", init="around_zero"),
            **gate,
            n["out"]: ParamSpec((h, self.v_width)),
        }

    def load(self, tensors):
        n = self.names
        if self.low_rank is None:
            # one product: [q | k | v | gate | beta | step]
            self.w_in = torch.cat([tensors[n[k]] for k in ("q", "k", "v", "gate", "beta", "step")], dim=0).contiguous()
        else:
            self._load_low_rank(tensors)
        self.conv = torch.cat([tensors[n[k]] for k in ("q_conv", "k_conv", "v_conv")], dim=0).float().contiguous()
        self.rate_log = tensors[n["rate_log"]].float().contiguous()
        self.step_bias = tensors[n["step_bias"]].float().contiguous()
        self.norm_weight = tensors[n["norm"]].float().contiguous()
        self.w_o = tensors[n["out"]].contiguous()

    def _load_low_rank(self, tensors):
        """One product [inner step | inner gate | q | k | v | beta], each of the inner parts padded to a multiple of
        eight columns, as all of it is; and one product from the inner parts to [steps | gates], a matrix with a block
        for each."""
        n = self.names
        inner, outer = [tensors[n["step_in"]], tensors[n["gate_in"]]], [tensors[n["step_out"]], tensors[n["gate_out"]]]
        for what, i, o in zip(("step", "gate"), inner, outer):
            if i.shape[0] != o.shape[1]:
                raise ValueError(f"{self.spec.prefix}: the low-rank {what} has an inner width of {i.shape[0]} in its first "
                                 f"matrix and {o.shape[1]} in its second")
        dtype, device = inner[0].dtype, inner[0].device
        wide = [-(-i.shape[0] // 8) * 8 for i in inner]
        self.mid_width = self.qkv_off = sum(wide)
        rows = []
        self.w_mid = torch.zeros((outer[0].shape[0] + outer[1].shape[0], self.mid_width), dtype=dtype, device=device)
        r, c = 0, 0
        for i, o, w in zip(inner, outer, wide):
            rows += [i, torch.zeros((w - i.shape[0], self.hidden_size), dtype=dtype, device=device)]
            self.w_mid[r:r + o.shape[0], c:c + o.shape[1]] = o
            r, c = r + o.shape[0], c + w
        rows += [tensors[n[k]] for k in ("q", "k", "v", "beta")]
        spare = -sum(m.shape[0] for m in rows) % 8
        rows.append(torch.zeros((spare, self.hidden_size), dtype=dtype, device=device))
        self.w_in = torch.cat(rows, dim=0).contiguous()

    def joinable(self) -> bool:
        return self.low_rank is not None

    def in_projection(self):
        return self.w_in, None

    def out_projection(self):
        return self.w_o, None

    def adopt(self, w_in, w_o):
        """Views of larger matrices in place of the part's own."""
        self.w_in, self.w_o = w_in, w_o

    def heads_forward(self, x, ctx, cache, projected=None, out=None):
        """Everything before the output projection: [tokens, heads * v_dim] times ``out_scale``.  ``projected``: (a
        product that holds this mixer's columns, the column where they begin; only with ``low_rank``); ``out``: (a wider
        matrix that receives the result, the first of its columns)."""
        if cache.state is None:
            raise ValueError("gated_delta: the cache manager gave this position no state")
        sizes = dict(num_heads=self.num_heads, num_kv_heads=self.num_kv_heads, head_dim=self.head_dim,
                     v_dim=self.v_dim, taps=self.taps)
        if projected is not None and self.low_rank is None:
            raise ValueError("gated_delta: only the low-rank form takes a product that is shared")
        x, off = projected if projected is not None else (ops.linear(x, self.w_in, status=ctx.status), 0)
        more, prep, scan = {}, {}, {"factor": self.out_scale, "gate": self.gate}
        if self.low_rank is not None:
            # steps and gates keep the accumulators' precision: the steps become the decays of a recurrence
            mid = ops.linear(x[:, off:off + self.mid_width], self.w_mid, out_dtype=torch.float32, status=ctx.status)
            at = off + self.qkv_off
            more = dict(channel_decay=self.channel_decay, x_off=at)
            prep = dict(steps=mid, step_off=0, beta_off=at + self.channels)
            scan.update(gates=mid, gate_off=self.steps)
        if out is not None:
            scan.update(out=out[0], out_off=out[1])
        qkv, coef = ops.delta_prep(x, self.conv, self.rate_log, self.step_bias, cache.state, ctx.cu_q,
                                   ctx.state_slots, unit_eps=self.unit_eps, **sizes, **more, **prep)
        return ops.delta_scan(qkv, coef, x, self.norm_weight, cache.state, ctx.cu_q, ctx.state_slots,
                              norm_eps=self.norm_eps, **sizes, **more, **scan)

    def forward(self, x, ctx, cache):
        return ops.linear(self.heads_forward(x, ctx, cache), self.w_o, status=ctx.status)
