"""The Gosizen decoder written out plainly: whole sequences, dense [T, T] score matrices, Python loops over time and
over experts, one function per mechanism.  It shares nothing with the package; the tests run it in float64 on the
weights the engine was given.

    x        = embed[token]                                                                  (x0 below)
    a layer  : h = norm(x);  x <- x + mixer(h) + ff(h)            (one norm, both branches read it; ff may be absent)
               then  y = P (gelu(G x) * e),  x <- x + y / rms(y) * w,   e: the layer's part of a row the token picks
    loop     : layers [start, stop) are walked `times` times; before a walk's first layer  x <- W [x; x0] + step[t]
    logits   = cap * tanh(head(norm(x)) / cap)
    norm     : x / sqrt(mean(x^2) + eps) * (1 + w)

``raw`` is the configuration as config.json holds it; ``w`` maps tensor names to tensors.
"""

from __future__ import annotations

import math

import torch


def rms_unit(x, eps):
    return x / torch.sqrt((x * x).mean(-1, keepdim=True) + eps)


def offset_norm(x, weight, eps):
    """The layers' norm: its weight is stored around zero."""
    return rms_unit(x, eps) * (1.0 + weight)


def gelu_tanh(z):
    return 0.5 * z * (1.0 + torch.tanh(math.sqrt(2.0 / math.pi) * (z + 0.044715 * z ** 3)))


def gelu_erf(z):
    return 0.5 * z * (1.0 + torch.erf(z / math.sqrt(2.0)))


def softplus(z):
    return torch.where(z > 40.0, z, torch.log1p(torch.exp(torch.clamp(z, max=40.0))))


# ------------------------------------------------------------------ positions and masks

def frequencies(rot):
    """Angle per position of every pair.  With ``scaling``: a pair whose wavelength is short keeps its frequency, one
    whose wavelength is long is slowed by ``factor``, and between the two bounds the two are mixed."""
    dims, base = int(rot["dims"]), float(rot["base"])
    out = []
    s = rot.get("scaling")
    for i in range(dims // 2):
        f = base ** (-2.0 * i / dims)
        if s is not None:
            wave = 2.0 * math.pi / f
            if wave > s["original"] / s["low"]:
                f = f / s["factor"]
            elif wave >= s["original"] / s["high"]:
                mix = (s["original"] / wave - s["low"]) / (s["high"] - s["low"])
                f = (1.0 - mix) * f / s["factor"] + mix * f
        out.append(f)
    return torch.tensor(out, dtype=torch.float64)


def turn(x, rot, layout):
    """x [T, heads, D]: row t's pairs turned by t * f_i.  ``layout`` "half": dims (i, i + dims / 2); "pairs": dims
    (2i, 2i + 1).  Dims from rot.dims on stay."""
    dims = int(rot["dims"])
    angle = torch.arange(x.shape[0], dtype=torch.float64)[:, None] * frequencies(rot)[None, :]
    cos, sin = angle.cos().to(x.dtype)[:, None, :], angle.sin().to(x.dtype)[:, None, :]
    out = x.clone()
    a, b = (slice(0, dims // 2), slice(dims // 2, dims)) if layout == "half" else (slice(0, dims, 2), slice(1, dims, 2))
    u, v = x[..., a], x[..., b]
    out[..., a], out[..., b] = u * cos - v * sin, v * cos + u * sin
    return out


def window_mask(T, size):
    back = torch.arange(T)[:, None] - torch.arange(T)[None, :]
    return (back >= 0) & (back < size)


def chunk_mask(T, size):
    i = torch.arange(T)
    return (i[:, None] >= i[None, :]) & (i[:, None] // size == i[None, :] // size)


def sink_softmax(scores, mask, sink):
    """Row-wise softmax over the visible keys with one more term exp(sink) in the denominator."""
    s = scores.masked_fill(~mask, -math.inf)
    top = torch.maximum(s.max(-1, keepdim=True).values, sink.expand(s.shape[0], 1))
    e = torch.exp(s - top)
    return e / (e.sum(-1, keepdim=True) + torch.exp(sink - top))


# ------------------------------------------------------------------ mixers

def latent_attention(h, w, prefix, m, eps):
    T, H, D, R, rank = h.shape[0], m["heads"], m["dim"], m["rot_dim"], m["kv_rank"]
    cq = rms_unit(h @ w[f"{prefix}.dq"].T, eps) * w[f"{prefix}.dq.norm"]
    q = (cq @ w[f"{prefix}.uq"].T).view(T, H, D + R)
    down = h @ w[f"{prefix}.dkv"].T
    c = rms_unit(down[:, :rank], eps) * w[f"{prefix}.dkv.norm"]
    rot = dict(m["rot"])
    shared = turn(down[:, None, rank:], rot, "pairs")[:, 0]
    turned = turn(q[..., D:], rot, "pairs")
    k = (c @ w[f"{prefix}.uk"].T).view(T, H, D)
    v = (c @ w[f"{prefix}.uv"].T).view(T, H, m["vdim"])
    gate = torch.sigmoid(h @ w[f"{prefix}.g"].T)
    mask = window_mask(T, m["mask"]["size"])
    heads = []
    for i in range(H):
        s = (q[:, i, :D] @ k[:, i].T + turned[:, i] @ shared.T) * float(m["scale"])
        heads.append(sink_softmax(s, mask, w[f"{prefix}.sink"][i]) @ v[:, i] * gate[:, i:i + 1])
    return torch.cat(heads, dim=-1) @ w[f"{prefix}.o"].T


def short_conv(x, taps):
    """x [T, C], taps [C, n]: y[t, c] = sum_j taps[c, j] * x[t - (n - 1) + j, c], zeros before the start."""
    T, n = x.shape[0], taps.shape[1]
    padded = torch.cat((x.new_zeros(n - 1, x.shape[1]), x), dim=0)
    y = torch.zeros_like(x)
    for j in range(n):
        y = y + padded[j:j + T] * taps[:, j]
    return y


def chunked_attention(h, w, prefix, m):
    """The left side: projections with biases, a short convolution on each, rotation, blocks of positions, a sink."""
    T, H, G, D, V = h.shape[0], m["heads"], m["kv_heads"], m["dim"], m["vdim"]

    def project(name):
        return short_conv(h @ w[f"{prefix}.{name}"].T + w[f"{prefix}.{name}.b"], w[f"{prefix}.{name}.conv"])

    q = turn(project("q").view(T, H, D), m["rot"], "half")
    k = turn(project("k").view(T, G, D), m["rot"], "half")
    v = project("v").view(T, G, V)
    mask = chunk_mask(T, m["mask"]["size"])
    heads = []
    for i in range(H):
        g = i // (H // G)
        s = (q[:, i] @ k[:, g].T) * float(m["scale"])
        heads.append(sink_softmax(s, mask, w[f"{prefix}.sink"][i]) @ v[:, g])
    out = torch.cat(heads, dim=-1) * torch.sigmoid(h @ w[f"{prefix}.g"].T)
    return out @ w[f"{prefix}.o"].T


def channel_delta_rule(q, k, v, beta, decay):
    """One head.  q, k, decay [T, D], v [T, V], beta [T].  S starts at zero; per token: row d of S times decay[d];
    u = beta (v - S^T k); S += k u^T; o = S^T q."""
    S = q.new_zeros(q.shape[1], v.shape[1])
    out = []
    for t in range(q.shape[0]):
        S = S * decay[t][:, None]
        u = beta[t] * (v[t] - S.T @ k[t])
        S = S + torch.outer(k[t], u)
        out.append(S.T @ q[t])
    return torch.stack(out)


def delta_mixer(h, w, prefix, m, eps):
    """The right side: the gated delta rule with a decay per head and key channel."""
    T, H, G, D, V = h.shape[0], m["heads"], m["kv_heads"], m["dim"], m["vdim"]

    def project(name):
        z = short_conv(h @ w[f"{prefix}.{name}"].T, w[f"{prefix}.{name}.conv"])
        return z * torch.sigmoid(z)

    def unit(z):
        return z / torch.sqrt((z * z).sum(-1, keepdim=True) + 1e-6)

    q = unit(project("q").view(T, G, D)) * D ** -0.5
    k = unit(project("k").view(T, G, D))
    v = project("v").view(T, H, V)
    beta = torch.sigmoid(h @ w[f"{prefix}.b"].T)
    step = softplus(h @ w[f"{prefix}.a1"].T @ w[f"{prefix}.a2"].T + w[f"{prefix}.dt_bias"]).view(T, H, D)
    decay = torch.exp(-torch.exp(w[f"{prefix}.A_log"])[None, :, None] * step)
    gate = torch.sigmoid(h @ w[f"{prefix}.g1"].T @ w[f"{prefix}.g2"].T).view(T, H, V)
    heads = []
    for i in range(H):
        g = i // (H // G)
        o = channel_delta_rule(q[:, g], k[:, g], v[:, i], beta[:, i], decay[:, i])
        heads.append(rms_unit(o, eps) * w[f"{prefix}.norm"] * gate[:, i])
    return torch.cat(heads, dim=-1) @ w[f"{prefix}.o"].T


def mixer(h, w, prefix, layer, eps):
    m = layer["mixer"]
    if layer["type"] == "latent_attention":
        return latent_attention(h, w, prefix, m, eps)
    return (float(m["left_scale"]) * chunked_attention(h, w, f"{prefix}.left", m["left"])
            + float(m["right_scale"]) * delta_mixer(h, w, f"{prefix}.right", m["right"], eps))


# ------------------------------------------------------------------ feed-forwards

def route(logits, top, margins=None):
    """logits [T, experts] -> (chosen [T, top], weights [T, top]: the softmax over the chosen logits).  ``margins`` (a
    list) receives by how much every token's last chosen logit leads the first one left out."""
    ranked = torch.sort(logits, dim=-1, descending=True, stable=True)
    chosen = ranked.indices[:, :top]
    if margins is not None:
        margins.append(ranked.values[:, top - 1] - ranked.values[:, top] if top < logits.shape[1]
                       else torch.full((logits.shape[0],), math.inf, dtype=logits.dtype))
    return chosen, torch.softmax(ranked.values[:, :top], dim=-1)


def experts_mixture(h, w, prefix, mlp, margins=None):
    chosen, weights = route(h @ w[f"{prefix}.router"].T + w[f"{prefix}.router.b"], mlp["router"]["top"], margins)
    out = torch.zeros_like(h)
    for e in sorted(set(chosen.flatten().tolist())):
        t, place = (chosen == e).nonzero(as_tuple=True)
        y = gelu_erf(h[t] @ w[f"{prefix}.e{e}.up"].T) @ w[f"{prefix}.e{e}.down"].T
        out[t] += weights[t, place][:, None] * y
    return out


def feed_forward(h, w, prefix, mlp, margins=None):
    if mlp.get("kind", "dense") == "dense":
        return gelu_tanh(h @ w[f"{prefix}.up"].T) @ w[f"{prefix}.down"].T
    return experts_mixture(h, w, prefix, mlp, margins)


# ------------------------------------------------------------------ the model

def side_input(x, e, w, prefix, eps):
    y = (gelu_tanh(x @ w[f"{prefix}.gate"].T) * e) @ w[f"{prefix}.proj"].T
    return x + rms_unit(y, eps) * w[f"{prefix}.norm"]


def schedule(raw):
    """(layer, walk that begins right before it or None) in run order."""
    count, loop = len(raw["layers"]), raw.get("loop")
    if loop is None:
        return [(i, None) for i in range(count)]
    order = [(i, None) for i in range(loop["start"])]
    for t in range(loop["times"]):
        order += [(i, t if i == loop["start"] else None) for i in range(loop["start"], loop["stop"])]
    return order + [(i, None) for i in range(loop["stop"], count)]


def forward(raw, w, tokens, margins=None, return_layers=False):
    """Logits of every position [T, vocab] in the dtype of the weights (and the stream after every layer run)."""
    eps = float(raw["norm"]["eps"])
    ids = torch.as_tensor(tokens, dtype=torch.long)
    x = start = w["embed"][ids]
    side = raw.get("token_side")
    after = []
    for i, walk in schedule(raw):
        layer, p = raw["layers"][i], f"l{i}"
        if walk is not None:
            x = torch.cat((x, start), dim=-1) @ w["loop.in"].T + w["loop.step"][walk]
        h = offset_norm(x, w[f"{p}.norm1"], eps)
        branch = mixer(h, w, f"{p}.mix", layer, eps)
        if layer.get("mlp") is not None:
            branch = branch + feed_forward(h, w, f"{p}.mlp", layer["mlp"], margins)
        x = x + branch
        if side is not None:
            dim = int(side["dim"])
            x = side_input(x, w["side.embed"][ids][:, i * dim:(i + 1) * dim], w, f"{p}.side", eps)
        after.append(x)
    logits = offset_norm(x, w["final.norm"], eps) @ w["head"].T
    cap = raw.get("logit_softcap")
    if cap:
        logits = cap * torch.tanh(logits / cap)
    return (logits, torch.stack(after)) if return_layers else logits


def greedy_generate(raw, w, prompt, count):
    ids, out = list(prompt), []
    for _ in range(count):
        out.append(int(forward(raw, w, ids)[-1].argmax()))
        ids.append(out[-1])
    return out
