"""Small Ligirax configurations of the tests, model folders with random weights for them (made in a temporary folder,
never committed), requests whose routing is decisive, a model in which one token decides what is asked for, and the
plain implementation's logits.

The configurations differ from one another in every size, in the order of their layers and in what is present:

* ``L1``: latents of a layer with a window of 20 read by a later layer with a larger window and odd head sizes, and by
  another with a smaller one; latents of a second layer read without any window; frequencies rescaled in one rotation
  and not in the other; layers without a feed-forward; experts with several, with no and with one identity choice; a
  top of one, two and three; sizes that are no multiple of 16.
* ``L2``: every choice chosen (top = experts + identity); a window of one token and one that is a multiple of the page;
  a single head; a multiplier and a logit scale of one; latents at which the tensor-core kernel for shared rows runs.
* ``L3``: sizes at which the tensor-core attention, the small-batch product kernel, the 16-byte paths and the clusters
  of the row-wise kernels run; more heads than a row tile holds.

Random matrices of N(0, 0.02) would leave every softmax nearly flat and every expert choice to the correction; the
folders' query / key matrices, routers and experts are scaled up.
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
from plain import ligirax_plain as plain


def rot(dims, base, scaling=None):
    out = {"base": base, "dims": dims}
    if scaling is not None:
        out["scaling"] = dict(zip(("factor", "original", "fast", "slow"), scaling))
    return out


def latent(heads, dim, rot_dim, vdim, kv_rank, scale, rotation, size=None, kv_from=None):
    mixer = {"heads": heads, "dim": dim, "rot_dim": rot_dim, "vdim": vdim, "kv_rank": kv_rank, "scale": scale,
             "rot": copy.deepcopy(rotation)}
    if size is not None:
        mixer["mask"] = {"size": size}
    if kv_from is not None:
        mixer["kv_from"] = kv_from
    return mixer


def moe(experts, identity, top, ff, limit):
    return {"kind": "moe", "expert": {"ff": ff, "limit": limit},
            "router": {"experts": experts, "identity": identity, "top": top}}


def layer(mixer, mlp):
    return {"type": "latent_attention", "mixer": mixer, "mlp": mlp}


_A, _B = rot(8, 300.0, (4.0, 64, 4.0, 1.0)), rot(6, 50.0)
L1 = {
    "architecture": "Ligirax", "vocab": 211, "width": 72, "norm": {"eps": 1e-5}, "residual_mult": 0.7, "logit_scale": 1.6,
    "layers": [
        layer(latent(3, 12, 8, 20, 24, 0.25, _A, size=20), moe(5, 3, 3, 24, 0.8)),
        layer(latent(5, 7, 8, 9, 24, 0.4, _A, size=50, kv_from=0), None),
        layer(latent(1, 16, 6, 28, 36, 0.2, _B, size=7), moe(3, 0, 2, 40, 2.5)),
        layer(latent(2, 12, 8, 12, 24, 0.3, _A, size=9, kv_from=0), moe(2, 1, 1, 12, 1.5)),
        layer(latent(4, 8, 6, 8, 36, 0.3, _B, kv_from=2), None),
    ],
}
_C, _D = rot(16, 1000.0, (2.5, 32, 2.0, 0.25)), rot(32, 20000.0, (8.0, 512, 16.0, 2.0))
L2 = {
    "architecture": "Ligirax", "vocab": 97, "width": 48, "norm": {"eps": 1e-6}, "residual_mult": 1.0, "logit_scale": 1.0,
    "layers": [
        layer(latent(1, 24, 16, 16, 64, 0.15, _C, size=1), moe(2, 2, 4, 16, 3.0)),
        layer(latent(6, 8, 16, 32, 64, 0.2, _C, size=64), None),
        layer(latent(3, 20, 16, 24, 64, 0.15, _C, size=31, kv_from=1), moe(7, 1, 5, 8, 0.5)),
    ],
}
L3 = {
    "architecture": "Ligirax", "vocab": 320, "width": 512, "norm": {"eps": 1e-6}, "residual_mult": 0.4, "logit_scale": 3.0,
    "layers": [
        layer(latent(20, 48, 32, 40, 256, 0.08, _D, size=96), moe(6, 2, 2, 128, 1.0)),
        layer(latent(16, 64, 32, 32, 256, 0.07, _D, size=40, kv_from=0), moe(4, 4, 3, 96, 2.0)),
        layer(latent(8, 32, 32, 64, 128, 0.1, _D), moe(3, 1, 1, 256, 1.5)),
    ],
}
CONFIGS = {"L1": (L1, 16), "L2": (L2, 32), "L3": (L3, 16)}


def config(name: str) -> dict:
    return copy.deepcopy(CONFIGS[name][0])


def save_weights(tensors: dict, path: str) -> None:
    """bfloat16-representable values: both precisions then run on the same weights."""
    save_file({k: v.to(torch.bfloat16).to(torch.float32).contiguous() for k, v in tensors.items()}, path,
              metadata={"format": "pt"})


@functools.lru_cache(maxsize=None)
def model_folder(name: str, seed: int = 3) -> str:
    from ampere_kv_engine_b200.models.registry import config_from_dict
    from ampere_kv_engine_b200.weights.random_init import write_random_model
    _, cfg = config_from_dict(config(name))
    out = tempfile.mkdtemp(prefix=f"ligirax_{name}_")
    write_random_model(cfg, seed, out, torch.float32)
    path = os.path.join(out, "model.safetensors")
    t = load_file(path)
    narrow = (72.0 / cfg.width) ** 0.5                # products of about the same size at every width
    t["embed"] = t["embed"] * 20.0
    # of both signs: a tied head would otherwise answer every token with itself
    t["final.norm"] = torch.randn(cfg.width, generator=torch.Generator().manual_seed(seed + 100))
    for i, lay in enumerate(cfg.layers):
        m = lay.mixer
        # unrotated and rotated scores with a spread of a few units before the scale
        t[f"l{i}.mix.q"] = t[f"l{i}.mix.q"] * (9.0 * narrow)
        t[f"l{i}.mix.uk"] = t[f"l{i}.mix.uk"] * (18.0 * (24.0 / m["kv_rank"]) ** 0.5)
        t[f"l{i}.mix.uv"] = t[f"l{i}.mix.uv"] * 10.0
        t[f"l{i}.mix.g"] = t[f"l{i}.mix.g"] * (10.0 * narrow)
        t[f"l{i}.mix.o"] = t[f"l{i}.mix.o"] * 10.0
        if m.get("kv_from") is None:
            t[f"l{i}.mix.dkv"] = t[f"l{i}.mix.dkv"] * (9.0 * narrow)
        if lay.mlp is not None:
            t[f"l{i}.mlp.router"] = t[f"l{i}.mlp.router"] * (9.0 * narrow)
            t[f"l{i}.mlp.correction"] = t[f"l{i}.mlp.correction"] * 1.7
            for e in range(lay.mlp["router"]["experts"]):
                for which in ("gate", "up"):          # the clamps bite
                    t[f"l{i}.mlp.e{e}.{which}"] = t[f"l{i}.mlp.e{e}.{which}"] * (8.0 * narrow)
                t[f"l{i}.mlp.e{e}.down"] = t[f"l{i}.mlp.e{e}.down"] * 12.0
    save_weights(t, path)
    return out


def plain_weights(folder: str) -> dict:
    return {k: v.double() for k, v in load_file(os.path.join(folder, "model.safetensors")).items()}


def plain_logits(folder: str, raw: dict, requests: dict[str, list[int]]) -> dict[str, torch.Tensor]:
    """float64 logits of every request as a whole sequence, as float32."""
    w = plain_weights(folder)
    return {rid: plain.forward(w, raw, toks).float() for rid, toks in requests.items()}


def check(trace, outputs, expected, dtype: str) -> tuple[float, float]:
    """Every written row against the plain one, measured by the row's own scale (relative RMS error, worst element).
    float32: the two differ by summation order, which layers of peaked softmaxes and clamped experts enlarge to
    1e-5 of the scale.  bfloat16: a row's rounding error is a few per cent of it, while a row that is wrong as a
    whole (a wrong page, a wrong expert, a lost gate) misses by its whole scale."""
    rms, peak = (5e-5, 3e-4) if dtype == "float32" else (0.15, 0.5)
    return ru.compare_rows_to_scale(trace, outputs, expected, rms_bound=rms, peak_bound=peak)


def decisive_requests(folder: str, raw: dict, lengths, seed: int, margin: float = 0.05, tries: int = 300
                      ) -> dict[str, list[int]]:
    """Random requests of the given lengths in which no expert choice is a close call: for every token and routed layer
    the last chosen one leads the first left out by at least ``margin`` in the plain implementation, so that a rounding
    of the router's input cannot change the choice.  Put together one token at a time."""
    w = {k: v.float() for k, v in plain_weights(folder).items()}
    g = torch.Generator().manual_seed(seed)
    out = {}
    for i, n in enumerate(lengths):
        toks: list[int] = []
        while len(toks) < n:
            for _ in range(tries):
                cand = toks + torch.randint(0, raw["vocab"], (1,), generator=g).tolist()
                margins: list = []
                plain.forward(w, raw, cand, margins=margins)
                if all(float(m[len(toks):].min()) >= margin for m in margins):
                    toks = cand
                    break
            else:
                raise AssertionError("no decisive continuation found; lower the margin")
        out[f"r{i}"] = toks
    return out


def random_config(seed: int) -> dict:
    """A seeded random configuration of the design: 2 to 5 layers, every size drawn anew (odd head sizes, ranks and
    widths that are no multiples of 16 among them), windows of all kinds, borrowed latents with windows and heads of
    their own, experts with and without identity choices, layers without a feed-forward."""
    rng = random.Random(seed)
    layers, owners = [], []
    for i in range(rng.randint(2, 5)):
        source = None
        if owners and rng.random() < 0.5:
            source, rank, rot_dim, rotation = rng.choice(owners)
        else:
            rank = rng.choice((8, 20, 33, 48, 64, 128))
            rot_dim = rng.choice((2, 4, 6, 16, 32))
            scaling = (rng.choice((1.0, 1.5, 4.0, 16.0)), rng.choice((16, 100, 4096)), rng.choice((2.0, 8.0, 32.0)),
                       rng.choice((0.5, 1.0)))
            rotation = rot(rot_dim, rng.choice((10.0, 500.0, 10000.0)), scaling if rng.random() < 0.7 else None)
            owners.append((i, rank, rot_dim, rotation))
        dim = rng.choice((3, 8, 12, 16, 32))
        mixer = latent(rng.choice((1, 2, 3, 5, 8)), dim, rot_dim, rng.choice((4, 7, 16, 24)), rank,
                       round(rng.uniform(0.5, 1.5) * (dim + rot_dim) ** -0.5, 4), rotation,
                       size=rng.choice((None, 1, 2, 5, 16, 17, 33, 64)), kv_from=source)
        experts, identity = rng.randint(1, 6), rng.choice((0, 0, 1, 2, 4))
        layers.append(layer(mixer, None if rng.random() < 0.2 else moe(
            experts, identity, rng.randint(1, min(4, experts + identity)), rng.choice((8, 15, 24, 40)),
            rng.choice((0.5, 1.0, 2.0, 7.0)))))
    return {"architecture": "Ligirax", "vocab": rng.choice((61, 128, 257)), "width": rng.choice((40, 48, 63, 72, 96)),
            "norm": {"eps": rng.choice((1e-5, 1e-6))}, "residual_mult": rng.choice((0.25, 0.6, 1.0, 1.3)),
            "logit_scale": rng.choice((0.5, 1.0, 2.2)), "layers": layers}


def random_model_folder(seed: int) -> str:
    CONFIGS[f"random{seed}"] = (random_config(seed), (16, 32, 64)[seed % 3])
    return model_folder(f"random{seed}", seed=seed)


MARK = 7          # the token of :func:`marked_model` whose key stands out


def marked_model(folder: str, window: int | None, reader_window: int | None, page: int) -> dict:
    """A model folder in which every query looks for the key of token ``MARK``: two layers, the second reading the
    first's latents with a window of its own.  All tokens share a component that makes their queries point along the
    first latent dim, which only the marked token's latent fills; its value is unlike the others'.  What a position's
    logits say is then whether the marked token lies inside either window."""
    from ampere_kv_engine_b200.models.registry import config_from_dict
    from ampere_kv_engine_b200.weights.random_init import write_random_model
    turned = rot(4, 100.0, (2.0, 64, 4.0, 1.0))
    raw = {"architecture": "Ligirax", "vocab": 61, "width": 40, "norm": {"eps": 1e-6}, "residual_mult": 0.8,
           "logit_scale": 1.3,
           "layers": [layer(latent(2, 8, 4, 12, 16, 1.0, turned, size=window), moe(2, 1, 2, 16, 1.0)),
                      layer(latent(3, 6, 4, 8, 16, 1.0, turned, size=reader_window, kv_from=0), None)]}
    _, cfg = config_from_dict(raw)
    write_random_model(cfg, 9, folder, torch.float32)
    path = os.path.join(folder, "model.safetensors")
    t = load_file(path)
    g = torch.Generator().manual_seed(2)
    embed = 0.05 * torch.randn(61, 40, generator=g)
    embed[:, 3] = 0.0
    embed[:, 5] = 1.0                                  # shared by all tokens: every query points the same way
    embed[MARK, 3] = 3.0
    t["embed"] = embed
    for i, (heads, dim) in enumerate(((2, 8), (3, 6))):
        q = 0.01 * torch.randn(heads * (dim + 4), 40, generator=g)
        q.view(heads, dim + 4, 40)[:, 0, 5] = 1.5
        uk = 0.01 * torch.randn(heads * dim, 16, generator=g)
        uk.view(heads, dim, 16)[:, 0, 0] = 1.5
        t[f"l{i}.mix.q"], t[f"l{i}.mix.uk"] = q, uk
        t[f"l{i}.mix.uv"] = 0.5 * torch.randn(t[f"l{i}.mix.uv"].shape, generator=g)
        t[f"l{i}.mix.o"] = 0.3 * torch.randn(t[f"l{i}.mix.o"].shape, generator=g)
    dkv = 0.01 * torch.randn(20, 40, generator=g)
    dkv[0, 3] = 1.0                                    # the first latent dim is the mark
    dkv[1, 5] = 0.5
    t["l0.mix.dkv"] = dkv
    t["l0.mlp.correction"] = torch.tensor([2.0, 0.0, 1.0])       # the routing is settled: not what is looked at here
    save_weights(t, path)
    return raw
