"""A feed-forward of many small gated experts of which every token uses a few, plus an optional shared expert.

    z       = W_r x (+ bias)                router logits, float32
    s       = sigmoid(z)                    scores (``score="softmax"``: softmax of z over all experts)
    c       = s + correction                choice scores (the weights below use s)
    groups  : the experts form ``groups`` equal runs of neighbours; a group's score is the sum of its ``group_top``
              largest c; only experts of the ``keep_groups`` best groups can be chosen
    chosen  = the ``top`` allowed experts with the largest c
    w_e     = s_e / (sum of the chosen s + weight_eps) * route_scale   (``normalize=False``: s_e * route_scale)
    choices from ``experts`` on (``identity`` of them) are the identity: w_e x, no matrices; the router, the scores,
              the correction and the groups count them like experts
    expert  : g = min(W_gate x, limit); u = clamp(W_up x, -limit, limit); W_down (g * sigmoid(slope * g) * (u + 1))
              (``activation="silu"``: plain W_down (silu(W_gate x) * W_up x), no clamp; ``gated=False``:
              W_down act(W_up x))
    y       = sum_e w_e expert_e(x)  +  shared(x)

Everything runs on the device from the batch layout alone (no host read of the routing), so a decode step through it
can be replayed as a CUDA graph: the router's product (``ops.moe_router_logits``), one kernel that scores and chooses (``ops.moe_route``), a
counting sort of the (token, choice) pairs by expert (``ops.moe_sort``), two grouped products over the sorted rows
(``ops.moe_gate_up`` with the activation on its output, ``ops.moe_down`` with the token's weight), and a sum in a
fixed order (``ops.moe_combine``).  The experts' matrices are stacked [experts, rows, columns] at load.
"""

from __future__ import annotations

import torch

from ..kernels import ops
from .base import FeedForward, ParamSpec, register_feed_forward


@register_feed_forward("routed_experts")
class RoutedExperts(FeedForward):
    """params: ``experts``, ``top``, ``groups`` and ``keep_groups`` (default 1 / 1: no groups), ``group_top``
    (default 2; 1: a group is scored by its best expert), ``identity`` (choices beyond the experts that hand back their
    input, default 0), ``normalize`` (default True: the chosen scores are divided by their sum), ``route_scale``,
    ``weight_eps``, ``score`` (``"sigmoid"`` or
    ``"softmax"``), ``correction`` (bool, default True: a learned per-expert offset of the choice scores),
    ``router_bias`` (bool, default False: a learned number per choice added to the logits), ``activation``
    (``"clamped_swish"``, the default, with ``limit`` and ``swish_slope``; or ``"silu"``), ``gated`` (default True; False:
    experts of one first matrix, ``activation`` then one of ``ops.ACTIVATIONS``, and no shared expert),
    ``intermediate_size`` of an expert, ``shared`` (None, or ``{"intermediate_size", "limit"}``), ``names`` (``expert`` with ``{}`` for
    the index, ``gate``, ``up``, ``down``, ``router``, ``router_bias``, ``correction``, ``shared``)."""

    graph_safe = True
    #: ``forward(..., defer_sum=True)`` hands back an ``ops.ExpertParts`` for a norm that adds the rows up itself
    defers_sum = True

    NAMES = {"expert": "experts.{}", "gate": "gate_proj.weight", "up": "up_proj.weight", "down": "down_proj.weight",
             "router": "router.weight", "router_bias": "router.bias", "correction": "router.correction",
             "shared": "shared_expert"}

    def __init__(self, spec, **kw):
        super().__init__(spec, **kw)
        p = spec.params
        self.experts, self.top = int(p["experts"]), int(p["top"])
        self.identity = int(p.get("identity") or 0)
        if self.identity < 0:
            raise ValueError("routed_experts: identity must not be negative")
        self.choices = self.experts + self.identity       # what the router scores
        self.normalize = bool(p.get("normalize", True))
        self.groups, self.keep_groups = int(p.get("groups") or 1), int(p.get("keep_groups") or 1)
        self.group_top = int(p.get("group_top", 2))
        if self.experts <= 0 or self.choices % self.groups or not 0 < self.keep_groups <= self.groups:
            raise ValueError(f"routed_experts: {self.choices} experts do not form {self.groups} equal groups of which "
                             f"{self.keep_groups} are kept")
        if not 0 < self.top <= self.keep_groups * (self.choices // self.groups):
            raise ValueError(f"routed_experts: top {self.top} is more than the kept groups hold")
        if self.choices > ops.MOE_MAX_EXPERTS or self.top > ops.MOE_MAX_TOP:
            raise ValueError(f"routed_experts: the kernels take up to {ops.MOE_MAX_EXPERTS} experts and a top of "
                             f"{ops.MOE_MAX_TOP}")
        self.score = str(p.get("score", "sigmoid"))
        if self.score not in ops.MOE_SCORES:
            raise ValueError(f"routed_experts: score must be one of {sorted(ops.MOE_SCORES)}, got {self.score!r}")
        self.activation = str(p.get("activation", "clamped_swish"))
        self.gated, self.has_router_bias = bool(p.get("gated", True)), bool(p.get("router_bias", False))
        if not self.gated:
            if self.activation not in ops.ACTIVATIONS or p.get("shared"):
                raise ValueError(f"routed_experts: experts without a gate take an activation of {sorted(ops.ACTIVATIONS)} "
                                 f"and no shared expert; got {self.activation!r}")
        elif self.activation not in ("clamped_swish", "silu"):
            raise ValueError(f"routed_experts: activation must be 'clamped_swish' or 'silu', got {self.activation!r}")
        self.route_scale = float(p.get("route_scale", 1.0))
        self.weight_eps = float(p.get("weight_eps", 1e-20))
        self.has_correction = bool(p.get("correction", True))
        self.intermediate_size = int(p["intermediate_size"])
        shared = p.get("shared")
        self.shared_size = int(shared["intermediate_size"]) if shared else 0
        if not self.gated:
            self.limit = self.swish_slope = self.up_offset = self.shared_limit = 0.0
        elif self.activation == "silu":
            # the clamped form with nothing to clamp, a slope of one and no offset on the up half is SiLU times up
            self.limit, self.swish_slope, self.up_offset, self.shared_limit = float("inf"), 1.0, 0.0, float("inf")
        else:
            self.limit, self.swish_slope, self.up_offset = float(p["limit"]), float(p.get("swish_slope", 1.702)), 1.0
            self.shared_limit = float(shared["limit"]) if shared else 0.0
        self.names = dict(self.NAMES, **(p.get("names") or {}))
        self.router_bias = None
        self.w_router = self.correction = self.w_gate_up = self.w_down = self.shared_gate_up = self.shared_down = None

    def _expert(self, index: int, which: str) -> str:
        return f"{self.names['expert'].format(index)}.{self.names[which]}"

    def param_specs(self):
        f, h, n = self.intermediate_size, self.hidden_size, self.names
        specs = {}
        for e in range(self.experts):
            if self.gated:
                specs[self._expert(e, "gate")] = ParamSpec((f, h))
            specs[self._expert(e, "up")] = ParamSpec((f, h))
            specs[self._expert(e, "down")] = ParamSpec((h, f))
        specs[n["router"]] = ParamSpec((self.choices, h))
        if self.has_router_bias:
            specs[n["router_bias"]] = ParamSpec((self.choices,), kind="vector", init="around_zero")
        if self.has_correction:
            specs[n["correction"]] = ParamSpec((self.choices,), kind="vector", init="around_zero")
        if self.shared_size:
            specs[f"{n['shared']}.{n['gate']}"] = ParamSpec((self.shared_size, h))
            specs[f"{n['shared']}.{n['up']}"] = ParamSpec((self.shared_size, h))
            specs[f"{n['shared']}.{n['down']}"] = ParamSpec((h, self.shared_size))
        return specs

    def load(self, tensors):
        n = self.names
        # [experts, gate rows then up rows, hidden] and [experts, hidden, intermediate]
        self.w_gate_up = torch.stack([torch.cat((tensors[self._expert(e, "gate")], tensors[self._expert(e, "up")]), dim=0)
                                      if self.gated else tensors[self._expert(e, "up")]
                                      for e in range(self.experts)]).contiguous()      # (no gate rows: the up rows alone)
        self.router_bias = tensors[n["router_bias"]].float().contiguous() if self.has_router_bias else None
        self.w_down = torch.stack([tensors[self._expert(e, "down")] for e in range(self.experts)]).contiguous()
        self.w_router = tensors[n["router"]].contiguous()
        self.correction = tensors[n["correction"]].float().contiguous() if self.has_correction else None
        if self.shared_size:
            self.shared_gate_up = torch.cat((tensors[f"{n['shared']}.{n['gate']}"], tensors[f"{n['shared']}.{n['up']}"]),
                                            dim=0).contiguous()
            self.shared_down = tensors[f"{n['shared']}.{n['down']}"].contiguous()

    def forward(self, x, ctx, defer_sum: bool = False):
        status = getattr(ctx, "status", None)
        logits = ops.moe_router_logits(x, self.w_router, status=status)
        chosen, weights = ops.moe_route(logits, self.correction, top=self.top, groups=self.groups,
                                        keep_groups=self.keep_groups, group_top=self.group_top,
                                        scale=self.route_scale, weight_eps=self.weight_eps, score=self.score,
                                        normalize=self.normalize, bias=self.router_bias)
        order, offsets = ops.moe_sort(chosen, self.choices)
        if self.identity:
            offsets = offsets[:self.experts + 1]       # the identity choices' pairs sort behind the experts' runs
        if self.gated:
            act = ops.moe_gate_up(x, self.w_gate_up, order, offsets, top=self.top, limit=self.limit,
                                  slope=self.swish_slope, up_offset=self.up_offset)
        else:
            act = ops.moe_up(x, self.w_gate_up, order, offsets, top=self.top, activation=self.activation)
        parts = ops.moe_down(act, self.w_down, order, offsets, weights)
        shared = None
        if self.shared_size:
            if self.activation == "silu":
                shared = ops.linear(ops.gated_linear(x, self.shared_gate_up, 0, status=status), self.shared_down,
                                    status=status)
            else:
                both = ops.linear(x, self.shared_gate_up, status=status)
                shared = ops.linear(ops.glu(both, "clamped_swish", 0, self.shared_limit, self.swish_slope),
                                    self.shared_down, status=status)
        identity = ops.IdentityChoices(chosen, weights, x, self.experts) if self.identity else None
        result = ops.ExpertParts(parts, shared, self.top, identity)
        return result if defer_sum else result.materialize()
