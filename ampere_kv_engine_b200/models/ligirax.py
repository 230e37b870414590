"""The ``Ligirax`` decoder as a model spec.

A plain token embedding; layers of block kind ``sandwich`` (every sublayer normed on the way in and on the way out, the
normed result times a constant added to the stream); ``latent_attention`` with queries straight from the mixer's input,
pairs of the rotated parts turned with frequencies rescaled by wavelength, a window and a sigmoid gate per head, in some
layers over the latents an earlier layer keeps; a feed-forward of ``routed_experts`` with softmax scores that are not
renormalised, some of whose choices are the identity, or none; the final norm and the embedding's matrix as the head,
its logits times a constant.  Tensor names: ``embed``, ``l<i>.norm1|norm1b|norm2|norm2b``, ``l<i>.mix.*``,
``l<i>.mlp.*``, ``final.norm``.

A layer with ``kv_from: j`` becomes a schedule position that reads the cache of position ``j``; how far back position
``j``'s pages are held follows from the windows of all that read them.
"""

from __future__ import annotations

from ..config.model_config import LigiraxConfig
from ..config.spec import LayerSpec, ModelSpec, PartSpec, ScheduleEntry
from .registry import register_architecture

#: constant the design fixes
SWISH_SLOPE = 1.702         # g * sigmoid(SWISH_SLOPE * g) in an expert


def _norm(config: LigiraxConfig, prefix: str, tensor: str, factor: float = 1.0) -> PartSpec:
    return PartSpec("rmsnorm", {"eps": config.norm_eps, "tensor": tensor, "factor": factor}, prefix)


def _mixer(config: LigiraxConfig, m: dict, prefix: str) -> PartSpec:
    rot = m["rot"]
    return PartSpec("latent_attention", {
        "num_heads": m["heads"], "head_dim": m["dim"], "rot_dim": m["rot_dim"], "v_dim": m["vdim"], "q_rank": None,
        "kv_rank": m["kv_rank"], "scale": m["scale"], "norm_eps": config.norm_eps,
        "position_encoding": PartSpec("rope", {"theta": rot["base"], "rotary_dim": rot["dims"], "layout": "pairs",
                                               "scaling": rot.get("scaling")}, ""),
        "window": (m.get("mask") or {}).get("size"), "gated": True, "own_kv": m.get("kv_from") is None,
        "names": {"q": "q", "dkv": "dkv", "dkv_norm": "dkv.norm", "uk": "uk", "uv": "uv", "gate": "g", "out": "o"},
    }, prefix)


def _feed_forward(mlp: dict, prefix: str) -> PartSpec:
    router = mlp["router"]
    return PartSpec("routed_experts", {
        "experts": router["experts"], "identity": router.get("identity") or 0, "top": router["top"],
        "score": "softmax", "normalize": False, "intermediate_size": mlp["expert"]["ff"],
        "limit": mlp["expert"]["limit"], "swish_slope": SWISH_SLOPE,
        "names": {"expert": "e{}", "gate": "gate", "up": "up", "down": "down", "router": "router",
                  "correction": "correction"}}, prefix)


def build_spec(config: LigiraxConfig) -> ModelSpec:
    layers, schedule, unused = [], [], []
    for i, layer in enumerate(config.layers):
        prefix = f"l{i}"
        # the constant on a sublayer's normed result is part of that norm's weight
        parts = {"mixer_out_norm": _norm(config, prefix, "norm1b", config.residual_mult)}
        ff = ff_norm = None
        if layer.mlp is not None:
            ff, ff_norm = _feed_forward(layer.mlp, f"{prefix}.mlp"), _norm(config, prefix, "norm2")
            parts["feed_forward_out_norm"] = _norm(config, prefix, "norm2b", config.residual_mult)
        else:
            # a layer without a feed-forward may still carry its norms
            unused += [(f"{prefix}.norm2", (config.width,)), (f"{prefix}.norm2b", (config.width,))]
        layers.append(LayerSpec(block="sandwich", mixer=_mixer(config, layer.mixer, f"{prefix}.mix"), feed_forward=ff,
                                mixer_norm=_norm(config, prefix, "norm1"), feed_forward_norm=ff_norm, parts=parts))
        schedule.append(ScheduleEntry(i, cache_of=layer.mixer.get("kv_from")))
    return ModelSpec(
        hidden_size=config.width,
        vocab_size=config.vocab,
        embedding=PartSpec("token_embedding", {"vocab_size": config.vocab, "tensor": "embed"}, ""),
        layers=tuple(layers),
        schedule=tuple(schedule),
        # the logits are linear in the final norm's weight: their constant rides on it
        final_norm=_norm(config, "final", "norm", config.logit_scale),
        head=PartSpec("linear_head", {"vocab_size": config.vocab, "tied": True, "tensor": "head"}, ""),
        max_position=config.max_position_embeddings,
        eos_token_ids=config.eos_token_id,
        unused_tensors=tuple(unused),
    )


register_architecture("Ligirax", LigiraxConfig, build_spec)
