"""Small Gosizen configurations of the tests, model folders with random weights for them (made in a temporary folder,
never committed), requests whose routing is decisive, models in which one token decides what is asked for, and the
plain implementation's logits.

The configurations differ from one another in every size, in the order of their layers and in what is present:

* ``G1``: a loop over the middle layers; left heads in groups of three, values narrower than keys, a rotation over part of
  the head; right heads in groups of two, values wider than keys, inner widths of five and nine; three and two taps; a
  dense feed-forward, experts of which two are used, and a layer without a feed-forward; sizes that are no multiple of 16.
* ``G2``: no loop, no token input, no logit cap; one tap on the left and five on the right; a single head; windows of one
  token and of a multiple of the page; frequencies without rescaling; all experts chosen; a top of one.
* ``G3``: sizes at which the tensor-core attention kernels, the small-batch products, the joined products, the 16-byte
  paths and the clusters of the row-wise kernels run; everything looped.

Random matrices of N(0, 0.02) would leave every softmax nearly flat and every memory forgotten within a few tokens; the
folders' query / key matrices, sinks, routers and decay rates are made so that they matter.
"""

from __future__ import annotations

import copy
import functools
import os
import random
import tempfile

import torch
from safetensors.torch import load_file, save_file

import replay_util as ru
from plain import gosizen_plain as plain


def rot(dims, base, scaling=None):
    out = {"base": base, "dims": dims}
    if scaling is not None:
        out["scaling"] = dict(zip(("factor", "low", "high", "original"), scaling))
    return out


def left(heads, kv_heads, dim, vdim, conv, scale, rotation, size):
    return {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "conv": conv, "scale": scale,
            "rot": copy.deepcopy(rotation), "mask": {"size": size}}


def right(heads, kv_heads, dim, vdim, conv, decay_rank, gate_rank):
    return {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "conv": conv, "decay_rank": decay_rank,
            "gate_rank": gate_rank}


def parallel(l, r, ls, rs, mlp):
    return {"type": "parallel", "mixer": {"left": l, "right": r, "left_scale": ls, "right_scale": rs}, "mlp": mlp}


def latent(heads, dim, rot_dim, vdim, q_rank, kv_rank, scale, base, size, mlp):
    return {"type": "latent_attention", "mlp": mlp,
            "mixer": {"heads": heads, "dim": dim, "rot_dim": rot_dim, "vdim": vdim, "q_rank": q_rank, "kv_rank": kv_rank,
                      "scale": scale, "rot": rot(rot_dim, base), "mask": {"size": size}}}


def dense(ff):
    return {"kind": "dense", "ff": ff}


def moe(experts, top, ff):
    return {"kind": "moe", "expert": {"ff": ff}, "router": {"experts": experts, "top": top}}


G1 = {
    "architecture": "Gosizen", "vocab": 211, "width": 72, "norm": {"eps": 1e-5}, "logit_softcap": 9.0,
    "token_side": {"dim": 12}, "loop": {"start": 1, "stop": 3, "times": 2},
    "layers": [
        parallel(left(6, 2, 20, 12, 3, 0.3, rot(12, 300.0, (4.0, 1.0, 8.0, 64)), 20), right(4, 2, 12, 20, 2, 5, 9), 0.7, 0.4,
                 dense(44)),
        latent(3, 7, 6, 9, 20, 24, 0.35, 500.0, 31, None),
        parallel(left(2, 2, 16, 28, 4, 0.25, rot(16, 1000.0, (2.0, 0.5, 2.0, 200)), 7), right(3, 1, 20, 7, 3, 11, 4), 0.5,
                 0.9, moe(5, 2, 24)),
        latent(5, 12, 8, 20, 9, 33, 0.25, 50.0, 50, moe(3, 1, 15)),
    ],
}
G2 = {
    "architecture": "Gosizen", "vocab": 97, "width": 48, "norm": {"eps": 1e-6},
    "layers": [
        latent(1, 24, 16, 16, 12, 64, 0.15, 1000.0, 1, moe(4, 4, 16)),
        parallel(left(4, 1, 24, 24, 1, 0.2, rot(8, 100.0), 64), right(1, 1, 33, 5, 5, 3, 3), 1.0, 1.0, None),
        latent(6, 8, 4, 32, 30, 40, 0.25, 20.0, 64, dense(30)),
        parallel(left(3, 3, 8, 40, 2, 0.35, rot(2, 30.0, (8.0, 0.25, 1.0, 16)), 33), right(6, 3, 4, 64, 1, 7, 6), 0.3, 1.2,
                 moe(7, 3, 8)),
    ],
}
G3 = {
    "architecture": "Gosizen", "vocab": 320, "width": 512, "norm": {"eps": 1e-6}, "logit_softcap": 20.0,
    "token_side": {"dim": 64}, "loop": {"start": 0, "stop": 3, "times": 2},
    "layers": [
        parallel(left(8, 2, 128, 128, 3, 0.09, rot(64, 20000.0, (8.0, 1.0, 4.0, 512)), 96), right(4, 2, 64, 128, 4, 32, 64),
                 0.6, 0.6, dense(640)),
        latent(20, 48, 32, 40, 160, 256, 0.1, 20000.0, 40, moe(6, 2, 128)),
        parallel(left(4, 4, 64, 64, 2, 0.12, rot(64, 500.0, (2.0, 1.0, 4.0, 128)), 64), right(2, 1, 128, 64, 3, 24, 16), 0.8,
                 0.5, moe(4, 3, 96)),
    ],
}
CONFIGS = {"G1": (G1, 16), "G2": (G2, 32), "G3": (G3, 16)}


def config(name: str) -> dict:
    return copy.deepcopy(CONFIGS[name][0])


def save_weights(tensors: dict, path: str) -> None:
    """bfloat16-representable values: both precisions then run on the same weights."""
    save_file({k: v.to(torch.bfloat16).to(torch.float32).contiguous() for k, v in tensors.items()}, path,
              metadata={"format": "pt"})


def write_folder(raw: dict, out: str, seed: int) -> dict:
    """config.json and random weights in ``out``; returns the tensors as they were drawn."""
    from ampere_kv_engine_b200.models.registry import config_from_dict
    from ampere_kv_engine_b200.weights.random_init import write_random_model
    _, cfg = config_from_dict(raw)
    write_random_model(cfg, seed, out, torch.float32)
    return load_file(os.path.join(out, "model.safetensors"))


@functools.lru_cache(maxsize=None)
def model_folder(name: str, seed: int = 3) -> str:
    raw = config(name)
    out = tempfile.mkdtemp(prefix=f"gosizen_{name}_")
    t = write_folder(raw, out, seed)
    g = torch.Generator().manual_seed(seed + 50)
    narrow = (72.0 / raw["width"]) ** 0.5                # products of about the same size at every width
    t["embed"] = t["embed"] * 20.0
    t["head"] = t["head"] * (10.0 * narrow)
    if "side.embed" in t:
        t["side.embed"] = t["side.embed"] * 40.0
    if "loop.in" in t:
        t["loop.in"] = t["loop.in"] * (3.0 * narrow)
    for i, lay in enumerate(raw["layers"]):
        p, m = f"l{i}.mix", lay["mixer"]
        if lay["type"] == "latent_attention":
            t[f"{p}.dq"] *= 9.0 * narrow
            t[f"{p}.uq"] *= 18.0 * (20.0 / m["q_rank"]) ** 0.5
            t[f"{p}.dkv"] *= 9.0 * narrow
            t[f"{p}.uk"] *= 18.0 * (24.0 / m["kv_rank"]) ** 0.5
            t[f"{p}.uv"] *= 10.0
            t[f"{p}.g"] *= 10.0 * narrow
            t[f"{p}.sink"] = torch.randn(m["heads"], generator=g) * 1.5 + 0.5
        else:
            for which in ("q", "k", "v"):
                t[f"{p}.left.{which}"] *= 12.0 * narrow
                t[f"{p}.left.{which}.b"] *= 4.0
                t[f"{p}.right.{which}"] *= 9.0 * narrow
                t[f"{p}.left.{which}.conv"] -= 0.3          # taps of both signs
                t[f"{p}.right.{which}.conv"] -= 0.3
            t[f"{p}.left.sink"] = torch.randn(m["left"]["heads"], generator=g) * 1.5 + 0.5
            t[f"{p}.left.g"] *= 10.0 * narrow
            t[f"{p}.right.b"] *= 10.0 * narrow
            # decays between about 0.5 and 0.995, unlike in every channel
            t[f"{p}.right.A_log"] = torch.randn(m["right"]["heads"], generator=g) * 0.7 - 2.5
            t[f"{p}.right.dt_bias"] = torch.randn(t[f"{p}.right.dt_bias"].shape, generator=g)
            for which in ("a1", "g1"):
                t[f"{p}.right.{which}"] *= 9.0 * narrow
            for which in ("a2", "g2"):
                t[f"{p}.right.{which}"] *= 30.0
            t[f"{p}.left.o"] *= 10.0
            t[f"{p}.right.o"] *= 10.0
        if f"{p}.o" in t:
            t[f"{p}.o"] *= 10.0
        if lay["mlp"] is not None and lay["mlp"]["kind"] == "moe":
            t[f"l{i}.mlp.router"] *= 9.0 * narrow
            t[f"l{i}.mlp.router.b"] *= 4.0
            for e in range(lay["mlp"]["router"]["experts"]):
                t[f"l{i}.mlp.e{e}.up"] *= 8.0 * narrow
                t[f"l{i}.mlp.e{e}.down"] *= 12.0
        elif lay["mlp"] is not None:
            t[f"l{i}.mlp.up"] *= 8.0 * narrow
            t[f"l{i}.mlp.down"] *= 10.0
        if f"l{i}.side.gate" in t:
            t[f"l{i}.side.gate"] *= 5.0 * narrow
            t[f"l{i}.side.proj"] *= 10.0
            t[f"l{i}.side.norm"] *= 0.5
    save_weights(t, os.path.join(out, "model.safetensors"))
    return out


def plain_weights(folder: str) -> dict:
    return {k: v.double() for k, v in load_file(os.path.join(folder, "model.safetensors")).items()}


def plain_logits(folder: str, raw: dict, requests: dict[str, list[int]]) -> dict[str, torch.Tensor]:
    """float64 logits of every request as a whole sequence, as float32."""
    w = plain_weights(folder)
    return {rid: plain.forward(raw, w, toks).float() for rid, toks in requests.items()}


def check(trace, outputs, expected, dtype: str, loose: float = 1.0) -> tuple[float, float]:
    """Every written row against the plain one, measured by the row's own scale (relative RMS error, worst element).
    float32: the two differ by summation order and by float32 angles.  bfloat16: a row's rounding error is a few per cent
    of its scale, while a row that is wrong as a whole (a wrong page, a wrong expert, a lost state) misses by all of it.
    ``loose``: a factor on the bounds for configurations drawn at random, some of which norm one or four numbers."""
    rms, peak = (1e-4, 5e-4) if dtype == "float32" else (0.15, 0.5)
    return ru.compare_rows_to_scale(trace, outputs, expected, rms_bound=rms * loose, peak_bound=peak * loose)


def decisive_requests(folder: str, raw: dict, lengths, seed: int, margin: float = 0.08, tries: int = 400
                      ) -> dict[str, list[int]]:
    """Random requests of the given lengths in which no expert choice is a close call: for every token and routed layer
    the last chosen logit leads the first left out by at least ``margin`` in the plain implementation.  Put together in
    pieces: a piece is drawn again, and halved, until it is decisive."""
    w = {k: v.float() for k, v in plain_weights(folder).items()}
    g = torch.Generator().manual_seed(seed)
    out = {}
    for i, n in enumerate(lengths):
        toks: list[int] = []
        size, left_tries = 4, tries
        while len(toks) < n:
            cand = toks + torch.randint(0, raw["vocab"], (min(size, n - len(toks)),), generator=g).tolist()
            margins: list = []
            plain.forward(raw, w, cand, margins=margins)
            if all(float(m[len(toks):].min()) >= margin for m in margins):
                toks, size = cand, min(8, size * 2)
            else:
                size, left_tries = max(1, size // 2), left_tries - 1
                assert left_tries > 0, "no decisive continuation found; lower the margin"
        out[f"r{i}"] = toks
    return out


def random_config(seed: int) -> dict:
    """A seeded random configuration of the design: 1 to 4 layers, every size drawn anew (odd head sizes, ranks and
    widths that are no multiples of 16 among them), windows and blocks of all kinds, one to six taps, grouped heads on
    either side, loops over any run of layers or none, with and without token input and logit cap."""
    rng = random.Random(seed)
    layers = []
    for _ in range(rng.randint(1, 4)):
        kind = rng.random()
        mlp = None if kind < 0.2 else dense(rng.choice((8, 30, 44, 64))) if kind < 0.5 else None
        if kind >= 0.5:
            experts = rng.randint(1, 7)
            mlp = moe(experts, rng.randint(1, min(4, experts)), rng.choice((8, 15, 24, 40)))
        if rng.random() < 0.4:
            rot_dim, dim = rng.choice((2, 4, 6, 16, 32)), rng.choice((3, 8, 12, 32))
            layers.append(latent(rng.choice((1, 2, 3, 5, 8)), dim, rot_dim, rng.choice((4, 7, 16, 24)),
                                 rng.choice((5, 16, 33, 40)), rng.choice((8, 20, 33, 64, 128)),
                                 round(rng.uniform(0.5, 1.5) * (dim + rot_dim) ** -0.5, 4), rng.choice((10.0, 500.0, 10000.0)),
                                 rng.choice((1, 2, 5, 16, 17, 33, 64)), mlp))
            continue
        kv, dim = rng.choice((1, 2, 3)), rng.choice((4, 9, 16, 20, 64))
        scaling = (rng.choice((1.0, 1.5, 4.0, 16.0)), rng.choice((0.25, 0.5, 1.0)), rng.choice((1.5, 4.0, 32.0)),
                   rng.choice((16, 100, 4096)))
        rotation = rot(2 * rng.randint(1, dim // 2), rng.choice((10.0, 500.0, 10000.0)), scaling if rng.random() < 0.7 else None)
        rk = rng.choice((1, 2, 3))
        layers.append(parallel(
            left(kv * rng.choice((1, 2, 4)), kv, dim, rng.choice((4, 11, 16, 64)), rng.choice((1, 2, 3, 4, 6)),
                 round(rng.uniform(0.5, 1.5) * dim ** -0.5, 4), rotation, rng.choice((1, 2, 5, 16, 17, 33, 64))),
            right(rk * rng.choice((1, 2, 3)), rk, rng.choice((3, 8, 12, 32, 70)), rng.choice((4, 7, 16, 40)),
                  rng.choice((1, 2, 4, 6)), rng.choice((1, 4, 13, 40)), rng.choice((1, 3, 16, 33))),
            rng.choice((0.3, 1.0, 1.4)), rng.choice((0.5, 1.0, 1.1)), mlp))
    raw = {"architecture": "Gosizen", "vocab": rng.choice((61, 128, 257)), "width": rng.choice((40, 48, 63, 72, 96)),
           "norm": {"eps": rng.choice((1e-5, 1e-6))}, "logit_softcap": rng.choice((None, 5.0, 12.0)), "layers": layers}
    if rng.random() < 0.7:
        raw["token_side"] = {"dim": rng.choice((1, 5, 8, 24))}
    if rng.random() < 0.7:
        start = rng.randint(0, len(layers) - 1)
        raw["loop"] = {"start": start, "stop": rng.randint(start + 1, len(layers)), "times": rng.randint(1, 3)}
    return raw


def random_model_folder(seed: int) -> str:
    CONFIGS[f"random{seed}"] = (random_config(seed), (16, 32, 64)[seed % 3])
    return model_folder(f"random{seed}", seed=seed)


MARK = 7          # the token of :func:`marked_model` whose key stands out


def marked_model(folder: str, kind: str, size: int) -> dict:
    """A model folder of one layer in which every query looks for the key of token ``MARK``: all tokens share a component
    that makes their queries point along one dim of the key (one that does not turn), which only the marked token's key
    fills; its value is unlike the others'.  What a position's logits say is then whether it sees the marked token.
    ``kind``: ``latent`` (a window of ``size``), ``left`` (blocks of ``size`` positions, the right side switched off) or
    ``right`` (the left side switched off: what is looked up is the memory, in which nothing fades and a key is found
    however far back it was written; ``size`` is not used)."""
    def layer_of():
        if kind == "latent":
            return latent(2, 8, 4, 12, 10, 16, 1.0, 100.0, size, None)
        return parallel(left(4, 2, 8, 12, 2, 1.0, rot(4, 100.0, (2.0, 1.0, 4.0, 64)), max(size, 1)),
                        right(2, 1, 8, 12, 2, 3, 2), 0.0 if kind == "right" else 0.9, 1.0 if kind == "right" else 0.0, None)
    raw = {"architecture": "Gosizen", "vocab": 61, "width": 40, "norm": {"eps": 1e-6}, "logit_softcap": 30.0,
           "token_side": {"dim": 4}, "layers": [layer_of()]}
    t = write_folder(raw, folder, 9)
    g = torch.Generator().manual_seed(2)
    embed = 0.05 * torch.randn(61, 40, generator=g)
    embed[:, 3] = 0.0
    embed[:, 5] = 1.0                                  # shared by all tokens: every query points the same way
    embed[MARK, 3] = 3.0
    t["embed"], p = embed, "l0.mix"
    small = lambda *shape: 0.01 * torch.randn(*shape, generator=g)      # noqa: E731
    if kind == "latent":
        t[f"{p}.dq"] = small(10, 40)
        t[f"{p}.dq"][0, 5] = 1.0                       # the query latent is the same unit vector for every token
        t[f"{p}.uq"] = small(2 * 12, 10)
        t[f"{p}.uq"].view(2, 12, 10)[:, 0, 0] = 2.0
        t[f"{p}.uk"] = small(2 * 8, 16)
        t[f"{p}.uk"].view(2, 8, 16)[:, 0, 0] = 1.5
        t[f"{p}.uv"] = 0.5 * torch.randn(2 * 12, 16, generator=g)
        t[f"{p}.dkv"] = small(20, 40)
        t[f"{p}.dkv"][0, 3] = 1.0                      # the first latent dim is the mark
        t[f"{p}.dkv"][1, 5] = 0.5
        t[f"{p}.sink"] = torch.full((2,), 3.0)
    else:
        for which, heads, at, value in (("q", 4, 5, 3.0), ("k", 2, 3, 1.5)):
            m = small(heads * 8, 40)
            m.view(heads, 8, 40)[:, 6, at] = value     # a dim behind the turned ones
            t[f"{p}.left.{which}"], t[f"{p}.left.{which}.b"] = m, small(heads * 8)
        t[f"{p}.left.v"] = 0.5 * torch.randn(24, 40, generator=g)
        for which in ("q", "k", "v"):                  # the current token alone
            t[f"{p}.left.{which}.conv"] = torch.tensor([[0.0, 1.0]]).repeat(t[f"{p}.left.{which}"].shape[0], 1)
            t[f"{p}.right.{which}.conv"] = torch.tensor([[0.0, 1.0]]).repeat(t[f"{p}.right.{which}"].shape[0], 1)
        t[f"{p}.left.sink"] = torch.full((4,), 2.0)
        # the memory: the marked token's key is one dim, everybody's query the same one, the others' keys another;
        # nothing fades (a step of zero)
        q, k = torch.zeros(8, 40), torch.zeros(8, 40)
        q[0, 5], k[0, 3], k[1, 5] = 2.0, 6.0, 1.0
        t[f"{p}.right.q"], t[f"{p}.right.k"] = q, k
        t[f"{p}.right.v"] = 0.5 * torch.randn(24, 40, generator=g)
        t[f"{p}.right.dt_bias"] = torch.full((16,), -30.0)
        t[f"{p}.right.b"] = torch.zeros(2, 40)
        t[f"{p}.right.b"][:, 5] = 3.0
    for name in [n for n in t if n.endswith(".o")]:
        t[name] = 0.3 * torch.randn(t[name].shape, generator=g)
    t["head"] = t["head"] * 20.0
    save_weights(t, os.path.join(folder, "model.safetensors"))
    return raw
