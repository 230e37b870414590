"""Plain, slow Ligirax decoder: whole sequences, no cache, one function per mechanism.

The oracle of the Ligirax tests.  It shares no code with the package: it reads a ``dict`` of tensors keyed by
checkpoint name and the ``dict`` of config.json, works on one whole sequence with dense [T, T] score matrices, expands
every key and value, and runs in the dtype of the tensors it is given (float64 in the tests).

The design in short.  The stream x starts as the embedding row.  Every sublayer is normed on the way in and on the way
out: ``x += m * N_out(mixer(N_in(x)))``, then the same with the feed-forward (which a layer may lack); all norms are
RMS norms with a plain weight.  The mixer is attention through a latent: c_t (normed) and one rotated key part r_t are
all a token leaves behind, keys and values of every head come from them by two matrices; a layer may take both from an
earlier layer and only bring its own matrices, queries and window.  The feed-forward is a mixture of clamped gated
experts, some choices of which are the identity; the chosen ones are weighted by their share of a softmax over all
choices.
"""

from __future__ import annotations

import math

import torch


def rms_norm(x: torch.Tensor, w: torch.Tensor, eps: float) -> torch.Tensor:
    return x / torch.sqrt(x.square().mean(dim=-1, keepdim=True) + eps) * w


def turn_frequencies(rot: dict) -> tuple[torch.Tensor, float]:
    """(angle per position of every pair, factor on cos and sin)."""
    dims, base = rot["dims"], float(rot["base"])
    f = torch.tensor([base ** (-2.0 * i / dims) for i in range(dims // 2)], dtype=torch.float64)
    s = rot.get("scaling")
    if s is None:
        return f, 1.0

    def where(turns):
        return dims * math.log(s["original"] / (2.0 * math.pi * turns)) / (2.0 * math.log(base))

    lo, hi = max(math.floor(where(s["fast"])), 0), min(math.ceil(where(s["slow"])), dims - 1)
    out = []
    for i in range(dims // 2):
        r = min(max((i - lo) / max(hi - lo, 0.001), 0.0), 1.0)
        out.append(float(f[i]) / s["factor"] * r + float(f[i]) * (1.0 - r))
    return torch.tensor(out, dtype=torch.float64), 0.1 * math.log(s["factor"]) + 1.0


def turn(x: torch.Tensor, rot: dict) -> torch.Tensor:
    """x [T, ..., D]: the pairs (2i, 2i + 1) of the first ``dims`` dims of row t turned by t * f_i."""
    freq, factor = turn_frequencies(rot)
    dims = rot["dims"]
    angle = torch.arange(x.shape[0], dtype=torch.float64)[:, None] * freq[None, :]
    shape = [x.shape[0]] + [1] * (x.dim() - 2) + [dims // 2]
    cos, sin = ((factor * t).to(x.dtype).view(shape) for t in (angle.cos(), angle.sin()))
    out = x.clone()
    u, v = x[..., 0:dims:2], x[..., 1:dims:2]
    out[..., 0:dims:2], out[..., 1:dims:2] = u * cos - v * sin, v * cos + u * sin
    return out


def window_mask(length: int, size: int | None) -> torch.Tensor:
    """[T, T] bool: token i sees token j iff 0 <= i - j < size (no size: every earlier one)."""
    back = torch.arange(length)[:, None] - torch.arange(length)[None, :]
    return (back >= 0) & ((back < size) if size else torch.ones_like(back, dtype=torch.bool))


def latent_of(h: torch.Tensor, w: dict, m: dict, eps: float) -> tuple[torch.Tensor, torch.Tensor]:
    """(normed latent [T, rank], turned shared key part [T, rot_dim]): what a token leaves behind."""
    down = h @ w["dkv"].T
    return rms_norm(down[:, :m["kv_rank"]], w["dkv.norm"], eps), turn(down[:, m["kv_rank"]:], m["rot"])


def latent_attention(h: torch.Tensor, w: dict, m: dict, kept: tuple[torch.Tensor, torch.Tensor]) -> torch.Tensor:
    T, H, D = h.shape[0], m["heads"], m["dim"]
    c, r = kept
    q = (h @ w["q"].T).view(T, H, D + m["rot_dim"])
    k, v = (c @ w["uk"].T).view(T, H, D), (c @ w["uv"].T).view(T, H, m["vdim"])
    s = torch.einsum("ihd,jhd->hij", q[..., :D], k) + torch.einsum("ihd,jd->hij", turn(q[..., D:], m["rot"]), r)
    mask = window_mask(T, (m.get("mask") or {}).get("size"))
    p = torch.softmax((s * m["scale"]).masked_fill(~mask[None], -math.inf), dim=-1)
    out = torch.einsum("hij,jhd->ihd", p, v) * torch.sigmoid(h @ w["g"].T)[:, :, None]
    return out.reshape(T, -1) @ w["o"].T


def clamped_expert(h: torch.Tensor, gate: torch.Tensor, up: torch.Tensor, down: torch.Tensor, limit: float):
    g = (h @ gate.T).clamp(max=limit)
    u = (h @ up.T).clamp(min=-limit, max=limit)
    return (g * torch.sigmoid(1.702 * g) * (u + 1.0)) @ down.T


def route(h: torch.Tensor, router: torch.Tensor, correction: torch.Tensor, top: int):
    """(chosen choices [T, top], their weights, by how much each token's last chosen one leads the first left out)."""
    s = torch.softmax(h @ router.T, dim=-1)
    c = s + correction
    order = torch.sort(c, dim=-1, descending=True, stable=True)
    chosen = order.indices[:, :top]
    lead = order.values[:, top - 1] - order.values[:, top] if top < c.shape[1] else torch.full((h.shape[0],), math.inf)
    return chosen, s.gather(1, chosen), lead


def mixture(h: torch.Tensor, w: dict, mlp: dict, margins: list | None = None) -> torch.Tensor:
    real, r = mlp["router"]["experts"], mlp["router"]
    chosen, weights, lead = route(h, w["router"], w["correction"], r["top"])
    if margins is not None:
        margins.append(lead)
    out = torch.zeros_like(h)
    for e in sorted(set(chosen.flatten().tolist())):
        t, place = (chosen == e).nonzero(as_tuple=True)          # the tokens that chose e
        y = h[t] if e >= real else clamped_expert(h[t], w[f"e{e}.gate"], w[f"e{e}.up"], w[f"e{e}.down"],
                                                  mlp["expert"]["limit"])
        out[t] += weights[t, place][:, None] * y
    return out


def local(weights: dict, prefix: str) -> dict:
    return {k[len(prefix) + 1:]: v for k, v in weights.items() if k.startswith(prefix + ".")}


def forward(weights: dict, config: dict, tokens: list[int], margins: list | None = None, return_layers: bool = False):
    """Logits [T, vocab] of one whole sequence (and the stream after every layer, if asked).  ``margins`` receives per
    routed layer by how much every token's choice is decided."""
    eps, m = config["norm"]["eps"], config["residual_mult"]
    x = weights["embed"][torch.tensor(tokens)]
    kept: dict[int, tuple] = {}
    after = []
    for i, layer in enumerate(config["layers"]):
        mixer, mix, pre = layer["mixer"], local(weights, f"l{i}.mix"), f"l{i}"
        h = rms_norm(x, weights[f"{pre}.norm1"], eps)
        source = mixer.get("kv_from")
        if source is None:
            source = i
            kept[i] = latent_of(h, mix, mixer, eps)
        x = x + m * rms_norm(latent_attention(h, mix, mixer, kept[source]), weights[f"{pre}.norm1b"], eps)
        if layer.get("mlp") is not None:
            h = rms_norm(x, weights[f"{pre}.norm2"], eps)
            y = mixture(h, local(weights, f"{pre}.mlp"), layer["mlp"], margins)
            x = x + m * rms_norm(y, weights[f"{pre}.norm2b"], eps)
        after.append(x)
    logits = rms_norm(x, weights["final.norm"], eps) @ weights["embed"].T * config["logit_scale"]
    return (logits, torch.stack(after)) if return_layers else logits


def greedy_generate(weights: dict, config: dict, prompt: list[int], new_tokens: int) -> list[int]:
    ids, out = list(prompt), []
    for _ in range(new_tokens):
        out.append(int(forward(weights, config, ids)[-1].argmax()))
        ids.append(out[-1])
    return out
