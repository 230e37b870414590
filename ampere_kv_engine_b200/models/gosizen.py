"""The ``Gosizen`` decoder as a model spec.

A plain token embedding; layers of block kind ``shared_norm`` (one norm whose weight is stored around zero; mixer and
feed-forward both read its output, their results join the stream together) with a ``token_gate`` after each (a small
gated branch that the token's id steers); a run of layers may be walked several times on one set of weights, a cache and
a state per walk, with a ``concat_projection`` of the stream and the embedding's output before every walk; a final norm
and an untied head with capped logits.  Mixers, chosen layer by layer:

``latent_attention``   ``latent_attention`` behind a query latent, with a window, sinks and a gate per head
``parallel``           ``parallel`` of a ``rotary_attention`` (biases and short convolutions on q, k and v, the half
                       layout with rescaled frequencies, blocks of positions, sinks, a gate per element) and a
                       ``gated_delta`` (a decay per head and key channel through a low-rank step, a low-rank sigmoid gate)

Feed-forwards, chosen layer by layer: dense with tanh GELU and no gate, routed experts without a gate (GELU, the softmax
over the chosen logits, a bias on the router), or none.

Tensor names: ``embed``, ``loop.in|step``, ``side.embed``, ``l<i>.norm1``, ``l<i>.mix.*`` (``.left.*`` / ``.right.*`` in a
parallel layer), ``l<i>.mlp.*``, ``l<i>.side.gate|proj|norm``, ``final.norm``, ``head``.
"""

from __future__ import annotations

from ..config.model_config import GosizenConfig
from ..config.spec import LayerSpec, ModelSpec, PartSpec, ScheduleEntry
from .registry import register_architecture

#: constants the design fixes
UNIT_EPS = 1e-6             # inside the root that makes the delta rule's q and k unit vectors


def _norm(config: GosizenConfig, prefix: str, tensor: str) -> PartSpec:
    return PartSpec("rmsnorm", {"eps": config.norm_eps, "tensor": tensor, "unit_offset": True}, prefix)


def _rope(rot: dict, layout: str) -> PartSpec:
    # a factor of one where the configuration names none: the frequencies are then formed in float64 and rounded once
    return PartSpec("rope", {"theta": rot["base"], "rotary_dim": rot["dims"], "layout": layout,
                             "scaling": rot.get("scaling") or {"factor": 1.0}}, "")


def _mixer(config: GosizenConfig, kind: str, m: dict, prefix: str) -> PartSpec:
    if kind == "latent_attention":
        return PartSpec("latent_attention", {
            "num_heads": m["heads"], "head_dim": m["dim"], "rot_dim": m["rot_dim"], "v_dim": m["vdim"],
            "q_rank": m["q_rank"], "kv_rank": m["kv_rank"], "scale": m["scale"], "norm_eps": config.norm_eps,
            "position_encoding": _rope(m["rot"], "pairs"), "window": (m.get("mask") or {}).get("size"), "gated": True,
            "sink": True,
            "names": {"dq": "dq", "dq_norm": "dq.norm", "uq": "uq", "dkv": "dkv", "dkv_norm": "dkv.norm", "uk": "uk",
                      "uv": "uv", "gate": "g", "sink": "sink", "out": "o"}}, prefix)
    left, right = m["left"], m["right"]
    return PartSpec("parallel", {
        "left": PartSpec("rotary_attention", {
            "num_heads": left["heads"], "num_kv_heads": left["kv_heads"], "head_dim": left["dim"], "v_dim": left["vdim"],
            "scale": left["scale"], "position_encoding": _rope(left["rot"], "half"), "bias": ("q", "k", "v"),
            "bias_suffix": ".b", "taps": left["conv"], "chunk": (left.get("mask") or {}).get("size"), "sink": True,
            "gated": True,
            "names": {"q": "q", "k": "k", "v": "v", "gate": "g", "sink": "sink", "out": "o"}}, f"{prefix}.left"),
        "right": PartSpec("gated_delta", {
            "num_heads": right["heads"], "num_kv_heads": right["kv_heads"], "head_dim": right["dim"],
            "v_dim": right["vdim"], "taps": right["conv"], "unit_eps": UNIT_EPS, "norm_eps": config.norm_eps,
            "decay": "channel", "gate": "sigmoid",
            "low_rank": {"step": right.get("decay_rank") or right["dim"], "gate": right.get("gate_rank") or right["vdim"]},
            "names": {"q": "q", "k": "k", "v": "v", "q_conv": "q.conv", "k_conv": "k.conv", "v_conv": "v.conv",
                      "beta": "b", "step_in": "a1", "step_out": "a2", "gate_in": "g1", "gate_out": "g2",
                      "rate_log": "A_log", "step_bias": "dt_bias", "norm": "norm", "out": "o"}}, f"{prefix}.right"),
        "left_scale": m["left_scale"], "right_scale": m["right_scale"]}, prefix)


def _feed_forward(mlp: dict, prefix: str) -> PartSpec:
    if mlp.get("kind", "dense") == "dense":
        return PartSpec("dense_mlp", {"intermediate_size": mlp["ff"], "activation": "gelu_tanh", "up": "up",
                                      "down": "down"}, prefix)
    # the softmax over the chosen logits is the softmax over all of them divided by the chosen ones' sum
    return PartSpec("routed_experts", {
        "experts": mlp["router"]["experts"], "top": mlp["router"]["top"], "score": "softmax", "weight_eps": 0.0,
        "correction": False, "router_bias": True, "gated": False, "activation": "gelu",
        "intermediate_size": mlp["expert"]["ff"],
        "names": {"expert": "e{}", "up": "up", "down": "down", "router": "router", "router_bias": "router.b"}}, prefix)


def build_spec(config: GosizenConfig) -> ModelSpec:
    layers, count = [], len(config.layers)
    for i, layer in enumerate(config.layers):
        prefix, parts = f"l{i}", {}
        if config.side_dim is not None:
            parts["after"] = PartSpec("token_gate", {
                "dim": config.side_dim, "runs": count, "run": i, "vocab_size": config.vocab, "eps": config.norm_eps,
                "names": {"table": "side.embed", "gate": f"{prefix}.side.gate", "proj": f"{prefix}.side.proj",
                          "norm": f"{prefix}.side.norm"}}, "")
        layers.append(LayerSpec(
            block="shared_norm", mixer=_mixer(config, layer.type, layer.mixer, f"{prefix}.mix"),
            feed_forward=None if layer.mlp is None else _feed_forward(layer.mlp, f"{prefix}.mlp"),
            mixer_norm=_norm(config, prefix, "norm1"), parts=parts))
    entry, schedule = None, [ScheduleEntry(i) for i in range(count)]
    if config.loop is not None:
        start, stop, times = (config.loop[k] for k in ("start", "stop", "times"))
        entry = PartSpec("concat_projection", {"times": times, "names": {"in": "in", "step": "step"}}, "loop")
        schedule = [ScheduleEntry(i) for i in range(start)]
        for t in range(times):
            schedule += [ScheduleEntry(i, begins_walk=t if i == start else None) for i in range(start, stop)]
        schedule += [ScheduleEntry(i) for i in range(stop, count)]
    return ModelSpec(
        hidden_size=config.width,
        vocab_size=config.vocab,
        embedding=PartSpec("token_embedding", {"vocab_size": config.vocab, "tensor": "embed"}, ""),
        layers=tuple(layers),
        schedule=tuple(schedule),
        final_norm=_norm(config, "final", "norm"),
        head=PartSpec("linear_head", {"vocab_size": config.vocab, "tied": False, "tensor": "head",
                                      "softcap": config.logit_softcap}, ""),
        max_position=config.max_position_embeddings,
        eos_token_ids=config.eos_token_id,
        walk_entry=entry,
    )


register_architecture("Gosizen", GosizenConfig, build_spec)
