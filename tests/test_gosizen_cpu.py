"""Gosizen without a GPU: configuration, the spec that is built from it, sizes that only the checkpoint says, closed
forms of the plain mechanisms, and the engine's host side (batch layout, cache manager, step function, scheduler, replay,
generation) driven through the stand-in kernels against the plain implementation."""

import math
import os

import pytest
import torch
from safetensors.torch import load_file, save_file

import gosizen_util as gu
import replay_util as ru
from plain import gosizen_plain as plain

LENGTHS = (1, 2, 19, 47, 90)


def _built(name):
    from ampere_kv_engine_b200.models.registry import config_from_dict
    arch, cfg = config_from_dict(gu.config(name))
    return arch, cfg, arch.build_spec(cfg)


def test_configuration_reads_every_size_and_names_what_is_wrong():
    from ampere_kv_engine_b200.config.model_config import ConfigError
    from ampere_kv_engine_b200.models.registry import config_from_dict
    arch, cfg, _ = _built("G1")
    assert arch.name == "Gosizen" and cfg.vocab_size == 211 and cfg.width == 72 and len(cfg.layers) == 4
    assert cfg.side_dim == 12 and cfg.logit_softcap == 9.0 and cfg.loop == {"start": 1, "stop": 3, "times": 2}
    for name in gu.CONFIGS:
        assert config_from_dict(_built(name)[1].to_dict())[1] == _built(name)[1]
    for path, value, word in ((("layers", 1, "type"), "mamba2", "type"), (("layers", 0, "mixer", "left", "heads"), 5, "heads"),
                              (("layers", 0, "mixer", "left", "conv"), 0, "conv"),
                              (("layers", 0, "mixer", "left", "rot", "dims"), 13, "dims"),
                              (("layers", 0, "mixer", "left", "rot", "dims"), 22, "dims"),
                              (("layers", 0, "mixer", "left", "rot", "scaling", "low"), 8.0, "low"),
                              (("layers", 0, "mixer", "left", "rot", "scaling", "original"), 0, "original"),
                              (("layers", 0, "mixer", "left", "mask", "size"), 0, "size"),
                              (("layers", 0, "mixer", "right", "kv_heads"), 3, "heads"),
                              (("layers", 0, "mixer", "right", "vdim"), -1, "vdim"),
                              (("layers", 0, "mixer", "left_scale"), None, "left_scale"),
                              (("layers", 1, "mixer", "q_rank"), 0, "q_rank"), (("layers", 1, "mixer", "scale"), "x", "scale"),
                              (("layers", 1, "mixer", "rot", "dims"), 8, "dims"), (("layers", 1, "mixer", "mask", "size"), 0, "size"),
                              (("layers", 0, "mlp", "kind"), "gated", "kind"), (("layers", 0, "mlp", "ff"), 0, "ff"),
                              (("layers", 2, "mlp", "router", "top"), 6, "top"), (("layers", 2, "mlp", "expert", "ff"), None, "ff"),
                              (("loop", "stop"), 5, "stop"), (("loop", "times"), 0, "times"), (("token_side", "dim"), 0, "dim"),
                              (("norm", "eps"), 0, "eps"), (("logit_softcap",), -1.0, "logit_softcap"), (("vocab",), -1, "vocab")):
        raw = gu.config("G1")
        node = raw
        for key in path[:-1]:
            node = node[key]
        node[path[-1]] = value
        with pytest.raises(ConfigError, match=word):
            config_from_dict(raw)


def test_spec_walks_the_loop_and_every_walk_keeps_its_own():
    from ampere_kv_engine_b200.cache.manager import CacheManager
    from ampere_kv_engine_b200.models.decoder import DecoderModel
    _, _, spec = _built("G1")
    assert [l.block for l in spec.layers] == ["shared_norm"] * 4 and [l.feed_forward is None for l in spec.layers] == [False, True, False, False]
    assert [(e.layer, e.begins_walk) for e in spec.schedule] == [(0, None), (1, 0), (2, None), (1, 1), (2, None), (3, None)]
    model = DecoderModel(spec, dtype=torch.float32, device="cpu")
    specs = model.cache_specs()
    assert [(s.kind, s.chunk, s.window) for s in specs] == [("chunk", 20, None), ("window", None, 31), ("chunk", 7, None),
                                                            ("window", None, 31), ("chunk", 7, None), ("window", None, 50)]
    # the left convolution's inputs, then the memory and the right one's, side by side in one slot
    assert model.blocks[0].mixer.state_sizes[0] == 2 * (8 * 20 + 2 * 12) and specs[0].state_shape[0] == sum(model.blocks[0].mixer.state_sizes)
    assert specs[1].state_shape == ()
    manager = CacheManager(specs, model.cache_of(), page_size=4, num_pages=40, max_seqs=2)
    views = [manager.layer_view(i) for i in range(6)]
    assert views[2].group == views[4].group and views[1].group == views[3].group and len(manager.groups) == 4
    assert views[2].state.data_ptr() != views[4].state.data_ptr()
    names = set(model.param_specs())
    assert {"loop.in", "loop.step", "side.embed", "l1.side.gate", "l0.mix.left.q.b", "l0.mix.left.q.conv", "l0.mix.left.sink",
            "l0.mix.left.g", "l0.mix.right.a1", "l0.mix.right.g2", "l0.mix.right.dt_bias", "l1.mix.sink", "l1.mix.g",
            "l2.mlp.e4.up", "l2.mlp.router.b", "l0.mlp.up", "final.norm", "head"} <= names
    assert not ({"l1.mlp.up", "l2.mlp.e0.gate", "l2.mlp.e5.up", "l0.norm2", "l0.mix.right.q.b"} & names)
    # without the options: no walk entry, no side, no cap
    _, _, spec = _built("G2")
    assert spec.walk_entry is None and all("after" not in l.roles() for l in spec.layers) and not spec.head.params["softcap"]


def test_inner_widths_are_the_checkpoints(fake_ext, tmp_path):
    """config.json does not say how wide the low-rank decay and gate are inside: a checkpoint with other widths than the
    configuration's hint loads and runs; one whose two halves disagree is refused by name."""
    from ampere_kv_engine_b200.models.decoder import DecoderModel
    from ampere_kv_engine_b200.weights.loader import WeightError, load_weights
    raw = gu.config("G1")
    t = gu.write_folder(raw, str(tmp_path), 1)
    assert t["l0.mix.right.a1"].shape == (5, 72) and t["l0.mix.right.g2"].shape == (80, 9)
    g = torch.Generator().manual_seed(0)
    for i in (0, 2):
        for a, b, r in (("a1", "a2", 17), ("g1", "g2", 2)):
            t[f"l{i}.mix.right.{a}"] = 0.1 * torch.randn(r, 72, generator=g)
            t[f"l{i}.mix.right.{b}"] = 0.3 * torch.randn(t[f"l{i}.mix.right.{b}"].shape[0], r, generator=g)
    path = os.path.join(str(tmp_path), "model.safetensors")
    gu.save_weights(t, path)
    requests = ru.make_requests(raw["vocab"], (9, 30), seed=1)
    trace = ru.trace_portions(requests)
    outputs = ru.run_inprocess(str(tmp_path), "float32", trace, 128, page_size=16)
    gu.check(trace, outputs, gu.plain_logits(str(tmp_path), raw, requests), "float32")
    model = DecoderModel(_built("G1")[2], dtype=torch.float32, device="cpu")
    t = load_file(path)
    save_file({**t, "l0.mix.right.a2": torch.zeros(48, 16)}, path)
    with pytest.raises(ValueError, match="l0.mix.right.*17.*16"):
        load_weights(model, str(tmp_path))
    save_file({**t, "l0.mix.right.a2": torch.zeros(47, 17)}, path)
    with pytest.raises(WeightError, match=r"l0.mix.right.a2 is \[47, 17\], expected \[48, any\]"):
        load_weights(model, str(tmp_path))


def test_closed_forms_of_the_plain_mechanisms():
    g = torch.Generator().manual_seed(0)
    # frequencies: short wavelengths stay, long ones are divided by the factor, between them a mixture
    r = gu.rot(64, 10000.0, (8.0, 1.0, 4.0, 512))
    f, plain_f = plain.frequencies(r), plain.frequencies(gu.rot(64, 10000.0))
    wave = 2 * math.pi / plain_f
    assert torch.equal(f[wave < 128], plain_f[wave < 128]) and torch.allclose(f[wave > 512], plain_f[wave > 512] / 8)
    between = (wave > 128) & (wave < 512)
    assert between.any() and bool(((f < plain_f) & (f > plain_f / 8))[between].all())
    from ampere_kv_engine_b200.config.spec import PartSpec
    from ampere_kv_engine_b200.parts.base import POSITION_ENCODINGS, build_part
    from ampere_kv_engine_b200.parts import position  # noqa: F401
    rope = build_part(POSITION_ENCODINGS, PartSpec("rope", {"theta": 10000.0, "rotary_dim": 64, "scaling": r["scaling"]}, ""),
                      hidden_size=8, dtype=torch.float32, device=torch.device("cpu"))
    assert torch.equal(rope.inv_freq, f.float()) and rope.factor == 1.0
    # a turn keeps lengths, and scores depend on the distance alone, in either layout
    x = torch.randn(1, 1, 8, generator=g, dtype=torch.float64).expand(12, 1, 8)
    for layout in ("half", "pairs"):
        y = plain.turn(x, gu.rot(6, 50.0), layout)
        assert torch.allclose(y.norm(dim=-1), x.norm(dim=-1)) and torch.equal(y[..., 6:], x[..., 6:])
        assert torch.allclose((y[3] * y[7]).sum(), (y[5] * y[9]).sum())
    # masks: a window of one, blocks counted from position 0
    assert torch.equal(plain.window_mask(4, 1), torch.eye(4, dtype=torch.bool))
    assert plain.chunk_mask(7, 3).sum(1).tolist() == [1, 2, 3, 1, 2, 3, 1]
    # a sink takes its share: with one visible key of score s its weight is sigmoid(s - sink)
    s = torch.randn(3, 3, generator=g, dtype=torch.float64)
    w = plain.sink_softmax(s, torch.eye(3, dtype=torch.bool), torch.tensor(0.7, dtype=torch.float64))
    assert torch.allclose(w, torch.diag(torch.sigmoid(s.diagonal() - 0.7)))
    # equal decays in every channel are the rule with one decay: a token's own write is read back whole
    k = torch.nn.functional.normalize(torch.randn(5, 4, generator=g, dtype=torch.float64), dim=-1)
    v = torch.randn(5, 3, generator=g, dtype=torch.float64)
    one = torch.ones(5, dtype=torch.float64)
    o = plain.channel_delta_rule(k, k, v, one, 0.5 * torch.ones(5, 4, dtype=torch.float64))
    assert torch.allclose(o, v)
    # a key in a channel that does not fade is found, one in a channel that fades is gone
    k = torch.eye(4, dtype=torch.float64)[[0, 1, 2, 2, 2]]
    q = torch.eye(4, dtype=torch.float64)[[0, 1, 0, 1, 1]]
    decay = torch.tensor([1.0, 0.5, 1.0, 1.0], dtype=torch.float64).expand(5, 4)
    o = plain.channel_delta_rule(q, k, v, one, decay)
    assert torch.allclose(o[2], v[0]) and torch.allclose(o[4], v[1] * 0.5 ** 3)
    # the softmax over the chosen logits alone
    z = torch.tensor([[1.0, 3.0, 2.0, -5.0]], dtype=torch.float64)
    chosen, weights = plain.route(z, 2)
    assert chosen.tolist() == [[1, 2]] and torch.allclose(weights, torch.softmax(torch.tensor([[3.0, 2.0]], dtype=torch.float64), -1))


@pytest.mark.parametrize("name", ["G1", "G2"])
@pytest.mark.parametrize("mode", ["whole", "last32", "portions", "mixed"])
def test_replay_matches_plain(fake_ext, name, mode):
    raw, page = gu.CONFIGS[name]
    folder = gu.model_folder(name)
    requests = ru.make_requests(raw["vocab"], LENGTHS + ((60, 45) if mode == "mixed" else ()), seed=11)
    expected = gu.plain_logits(folder, raw, requests)
    max_tokens = 64 * 6
    trace = {"whole": ru.trace_whole, "last32": ru.trace_last_decoded, "portions": ru.trace_portions,
             "mixed": lambda r: ru.trace_mixed(r, max_tokens, seed=5)}[mode](requests)
    outputs = ru.run_inprocess(folder, "float32", trace, max_tokens, page_size=page)
    gu.check(trace, outputs, expected, "float32")


def test_greedy_generation_through_the_scheduler(fake_ext):
    from ampere_kv_engine_b200.engine.engine import Engine
    raw, page = gu.CONFIGS["G1"]
    folder = gu.model_folder("G1")
    engine = Engine.from_pretrained(folder, dtype="float32", device="cpu", page_size=page, num_pages=12,
                                    max_batch_tokens=24, max_seqs=2)
    prompts = list(ru.make_requests(raw["vocab"], (3, 30, 41), seed=2).values())
    got = engine.generate(prompts, max_new_tokens=5, ignore_eos=True)       # three requests through two state slots
    w = gu.plain_weights(folder)
    assert got == [plain.greedy_generate(raw, w, p, 5) for p in prompts]
    assert engine.manager.free_pages() == [12] * len(engine.manager.groups)
    engine.manager.check_invariants()


@pytest.mark.parametrize("kind,size", [("latent", 20), ("left", 33), ("right", 0)])
def test_a_marked_token_shows_exactly_where_it_is_seen(fake_ext, tmp_path, kind, size):
    """The plain implementation's logits move when the marked token is taken away exactly where the window or the block
    holds it (and, in the memory, everywhere after it); the engine agrees, in portions and token by token."""
    raw = gu.marked_model(str(tmp_path / "m"), kind, size)
    w = gu.plain_weights(str(tmp_path / "m"))
    tokens = [t if t != gu.MARK else 8 for t in ru.make_requests(61, (80,), seed=4)["r0"]]
    tokens[16] = gu.MARK
    blank = list(tokens)
    blank[16] = 9
    moved = (plain.forward(raw, w, tokens) - plain.forward(raw, w, blank)).abs().amax(dim=1)
    stop = {"latent": 16 + size, "left": 33, "right": 80}[kind]
    assert float(moved[16:stop].min()) > 0.02 and float(moved[:16].max()) == 0.0
    assert stop == 80 or float(moved[stop:].max()) == 0.0
    requests = {"r0": tokens}
    expected = gu.plain_logits(str(tmp_path / "m"), raw, requests)
    for trace in (ru.trace_portions(requests), ru.trace_last_decoded(requests, last=60)):
        outputs = ru.run_inprocess(str(tmp_path / "m"), "float32", trace, 128, page_size=16)
        gu.check(trace, outputs, expected, "float32")


@pytest.mark.parametrize("seed", [1, 2, 3, 4, 5, 6])
def test_random_configurations_replay(fake_ext, seed):
    folder = gu.random_model_folder(seed)
    raw, page = gu.CONFIGS[f"random{seed}"]
    requests = ru.make_requests(raw["vocab"], (1, 2, 23, 51, 37), seed=seed)
    expected = gu.plain_logits(folder, raw, requests)
    trace = ru.trace_mixed(requests, 64 * 4, seed=seed)
    outputs = ru.run_inprocess(folder, "float32", trace, 64 * 4, page_size=page)
    gu.check(trace, outputs, expected, "float32", loose=5.0)
