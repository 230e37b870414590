"""Ligirax without a GPU: configuration, the spec that is built from it, how far back borrowed latents are held, closed
forms of the plain mechanisms, and the engine's host side (batch layout, cache manager, step function, scheduler,
replay, generation) driven through the stand-in kernels against the plain implementation."""

import math

import pytest
import torch

import ligirax_util as lu
import replay_util as ru
from plain import ligirax_plain as plain

LENGTHS = (1, 2, 19, 47, 130)


def test_configuration_reads_every_size_and_names_what_is_wrong():
    from ampere_kv_engine_b200.config.model_config import ConfigError
    from ampere_kv_engine_b200.models.registry import config_from_dict
    arch, cfg = config_from_dict(lu.config("L1"))
    assert arch.name == "Ligirax" and cfg.vocab_size == 211 and cfg.width == 72 and len(cfg.layers) == 5
    assert cfg.residual_mult == 0.7 and cfg.logit_scale == 1.6 and cfg.norm_eps == 1e-5
    assert config_from_dict(cfg.to_dict())[1] == cfg
    for path, value, word in ((("layers", 1, "type"), "attention", "type"), (("layers", 0, "mixer", "heads"), 0, "heads"),
                              (("layers", 0, "mixer", "rot", "dims"), 7, "dims"), (("layers", 0, "mixer", "rot", "dims"), 10, "dims"),
                              (("layers", 0, "mixer", "rot", "base"), 1.0, "base"),
                              (("layers", 0, "mixer", "rot", "scaling", "factor"), 0, "factor"),
                              (("layers", 0, "mixer", "mask", "size"), 0, "size"),
                              (("layers", 1, "mixer", "kv_from"), 1, "kv_from"),        # not an earlier layer
                              (("layers", 3, "mixer", "kv_from"), 1, "kv_from"),        # which has no latents of its own
                              (("layers", 3, "mixer", "kv_from"), 2, "kv_from"),        # another rank and rotation
                              (("layers", 1, "mixer", "rot", "base"), 301.0, "kv_from"),
                              (("layers", 0, "mlp", "kind"), "dense", "kind"), (("layers", 0, "mlp", "expert", "limit"), 0, "limit"),
                              (("layers", 0, "mlp", "router", "top"), 9, "top"),
                              (("layers", 0, "mlp", "router", "identity"), -1, "identity"),
                              (("norm", "eps"), 0, "eps"), (("residual_mult",), "x", "residual_mult"),
                              (("logit_scale",), None, "logit_scale"), (("vocab",), -1, "vocab")):
        raw = lu.config("L1")
        node = raw
        for key in path[:-1]:
            node = node[key]
        node[path[-1]] = value
        with pytest.raises(ConfigError, match=word):
            config_from_dict(raw)


def test_spec_gives_layers_their_parts_and_borrowers_their_source():
    from ampere_kv_engine_b200.models.decoder import DecoderModel
    from ampere_kv_engine_b200.models.registry import config_from_dict
    arch, cfg = config_from_dict(lu.config("L1"))
    spec = arch.build_spec(cfg)
    assert [l.block for l in spec.layers] == ["sandwich"] * 5
    assert [e.cache_of for e in spec.schedule] == [None, 0, None, 0, 2]
    assert [l.feed_forward is None for l in spec.layers] == [False, True, False, False, True]
    model = DecoderModel(spec, dtype=torch.float32, device="cpu")
    specs = model.param_specs()
    wanted = {name for name, ps in specs.items() if not ps.optional}
    assert {"embed", "final.norm", "l0.norm1", "l0.norm1b", "l0.norm2", "l0.norm2b", "l0.mix.q", "l0.mix.dkv",
            "l0.mix.dkv.norm", "l0.mix.g", "l1.mix.uk", "l0.mlp.e4.down", "l0.mlp.router", "l0.mlp.correction"} <= wanted
    assert not ({"l1.mix.dkv", "l1.mix.dkv.norm", "l0.mlp.e5.gate", "l1.mlp.router"} & set(specs))
    assert specs["l1.norm2"].optional and specs["l1.norm2b"].optional
    # a tied head may be carried by a checkpoint; the router scores experts and identity choices
    assert specs["head"].optional and specs["l0.mlp.router"].shape == (8, 72) and specs["l2.mlp.router"].shape == (3, 72)
    assert specs["l1.mix.q"].shape == (5 * 15, 72) and specs["l1.mix.o"].shape == (72, 45)
    # the constants of the configuration ride on norm weights
    assert model.blocks[0].mixer_out_norm.factor == 0.7 and model.final_norm.factor == 1.6
    assert model.blocks[0].mixer_norm.factor == 1.0


def test_borrowed_latents_are_held_as_far_back_as_any_reader_looks():
    from ampere_kv_engine_b200.cache.manager import CacheManager
    from ampere_kv_engine_b200.models.decoder import DecoderModel
    from ampere_kv_engine_b200.models.registry import config_from_dict
    from ampere_kv_engine_b200.parts.base import CacheSpec, CacheTensor
    arch, cfg = config_from_dict(lu.config("L1"))
    model = DecoderModel(arch.build_spec(cfg), dtype=torch.float32, device="cpu")
    specs = model.cache_specs()
    assert [(s.kind, s.window) for s in specs] == [("window", 50), ("window", 50), ("full", None), ("window", 50), ("full", None)]
    manager = CacheManager(specs, model.cache_of(), page_size=4, num_pages=40, max_seqs=2)
    assert len(manager.groups) == 2 and manager.groups[0].window == 50 and manager.groups[1].window is None
    assert [manager.layer_view(i).writes for i in range(5)] == [True, False, True, False, False]
    seq = manager.open("a")
    manager.reserve(seq, 90)
    manager.commit(seq, 90)
    # the next query, at 90, of the reader with 50 keys sees 41 ..: the page of 40 .. 43 is the first that is held
    assert [p >= 0 for p in seq.pages[0]] == [j >= 10 for j in range(23)] and all(p >= 0 for p in seq.pages[1])
    manager.check_invariants()
    row = (CacheTensor("latent", 1, 8),)
    small, large = CacheSpec(kind="window", window=3, tensors=row), CacheSpec(kind="window", window=9, keep_first=2, tensors=row)
    assert small.covering(large) == large and large.covering(small) == large and small.covering(small) is small
    assert large.covering(CacheSpec(kind="full", tensors=row)).kind == "full"
    assert CacheSpec(kind="chunk", chunk=4, tensors=row).covering(small) == CacheSpec(kind="full", tensors=row)
    other = CacheSpec(kind="full", tensors=(CacheTensor("latent", 1, 9),))
    assert small.covering(other) is small                   # the manager refuses such a pair


def test_a_borrowing_mixer_must_be_scheduled_behind_its_source(fake_ext):
    import dataclasses
    from ampere_kv_engine_b200.config.spec import ScheduleEntry
    from ampere_kv_engine_b200.engine.batch import SeqStep
    from ampere_kv_engine_b200.engine.step import ModelRunner
    from ampere_kv_engine_b200.models.decoder import DecoderModel
    from ampere_kv_engine_b200.models.registry import config_from_dict
    from ampere_kv_engine_b200.weights.random_init import init_random
    arch, cfg = config_from_dict(lu.config("L1"))
    spec = arch.build_spec(cfg)
    spec = dataclasses.replace(spec, schedule=tuple(ScheduleEntry(i) for i in range(len(spec.layers))))
    model = DecoderModel(spec, dtype=torch.float32, device="cpu")
    init_random(model, 0)
    runner = ModelRunner(model, page_size=4, num_pages=8, max_seqs=2, cuda_graphs=False)
    with pytest.raises(ValueError, match="cache_of"):
        runner.step([SeqStep(runner.open("a"), [1, 2, 3], [2])])


def test_closed_forms_of_the_plain_mechanisms():
    # a pair's turn keeps its length (times the factor), and scores of turned pairs depend on the distance alone
    r = lu.rot(6, 50.0, (4.0, 64, 4.0, 1.0))
    g = torch.Generator().manual_seed(0)
    x = torch.randn(1, 6, generator=g, dtype=torch.float64).expand(12, 6)
    y = plain.turn(x, r)
    factor = 0.1 * math.log(4.0) + 1.0
    assert torch.allclose(y.norm(dim=-1), x.norm(dim=-1) * factor)
    assert torch.allclose((y[3] * y[7]).sum(), (y[5] * y[9]).sum())
    # frequencies: the fastest pair is kept, the slowest divided by the factor
    freq, _ = plain.turn_frequencies(lu.rot(32, 10000.0, (4.0, 256, 32.0, 1.0)))
    assert freq[0] == 1.0 and math.isclose(float(freq[-1]), 10000.0 ** (-30 / 32) / 4.0)
    # a window of one sees the token itself
    assert torch.equal(plain.window_mask(4, 1), torch.eye(4, dtype=torch.bool))
    assert plain.window_mask(5, 3).sum(1).tolist() == [1, 2, 3, 3, 3]
    # a mixture whose choices are all the identity is the input times the chosen scores
    h = torch.randn(3, 4, generator=g, dtype=torch.float64)
    w = {"router": torch.zeros(3, 4, dtype=torch.float64), "correction": torch.tensor([0.0, 5.0, 4.0], dtype=torch.float64)}
    out = plain.mixture(h, w, {"expert": {"limit": 1.0}, "router": {"experts": 1, "identity": 2, "top": 2}})
    assert torch.allclose(out, h * (2.0 / 3.0))


def test_weights_are_not_renormalised_and_the_out_norm_hides_a_common_factor(fake_ext):
    """Two routings that differ by a common factor give the same normed branch, so a renormalisation only shows beside
    the norm's eps; the router part alone is looked at here."""
    from ampere_kv_engine_b200.kernels import ops
    logits = torch.randn(5, 7, generator=torch.Generator().manual_seed(3))
    correction = torch.randn(7, generator=torch.Generator().manual_seed(4))
    chosen, weights = ops.moe_route(logits, correction, top=3, groups=1, keep_groups=1, group_top=1, scale=1.0,
                                    weight_eps=0.0, score="softmax", normalize=False)
    want, s, _ = plain.route(logits.double(), torch.eye(7, dtype=torch.float64), correction.double(), 3)
    assert torch.equal(chosen.long(), want) and torch.allclose(weights.double(), s, atol=1e-6)


@pytest.mark.parametrize("name", ["L1", "L2"])
@pytest.mark.parametrize("mode", ["whole", "last32", "portions", "mixed"])
def test_replay_matches_plain(fake_ext, name, mode):
    raw, page = lu.CONFIGS[name]
    folder = lu.model_folder(name)
    requests = ru.make_requests(raw["vocab"], LENGTHS + ((70, 45) if mode == "mixed" else ()), seed=11)
    expected = lu.plain_logits(folder, raw, requests)
    max_tokens = 64 * 6
    trace = {"whole": ru.trace_whole, "last32": ru.trace_last_decoded, "portions": ru.trace_portions,
             "mixed": lambda r: ru.trace_mixed(r, max_tokens, seed=5)}[mode](requests)
    outputs = ru.run_inprocess(folder, "float32", trace, max_tokens, page_size=page)
    lu.check(trace, outputs, expected, "float32")


def test_greedy_generation_through_the_scheduler(fake_ext):
    from ampere_kv_engine_b200.engine.engine import Engine
    raw, page = lu.CONFIGS["L1"]
    folder = lu.model_folder("L1")
    engine = Engine.from_pretrained(folder, dtype="float32", device="cpu", page_size=page, num_pages=12,
                                    max_batch_tokens=24, max_seqs=4)
    prompts = list(ru.make_requests(raw["vocab"], (3, 30, 61), seed=2).values())
    got = engine.generate(prompts, max_new_tokens=6, ignore_eos=True)
    w = lu.plain_weights(folder)
    assert got == [plain.greedy_generate(w, raw, p, 6) for p in prompts]
    assert engine.manager.free_pages() == [12] * len(engine.manager.groups)
    engine.manager.check_invariants()


@pytest.mark.parametrize("window,reader_window", [(20, 45), (45, 20), (33, None)])
def test_a_marked_token_shows_exactly_inside_the_windows(fake_ext, tmp_path, window, reader_window):
    """The plain implementation's logits move when the marked token is taken away exactly where one of the two windows
    reaches it; the engine agrees at every position, in portions and token by token."""
    raw = lu.marked_model(str(tmp_path / "m"), window, reader_window, 16)
    w = lu.plain_weights(str(tmp_path / "m"))
    tokens = ru.make_requests(61, (90,), seed=4)["r0"]
    tokens = [t if t != lu.MARK else 8 for t in tokens]
    tokens[16] = lu.MARK
    blank = list(tokens)
    blank[16] = 9
    moved = (plain.forward(w, raw, tokens) - plain.forward(w, raw, blank)).abs().amax(dim=1)
    # both layers read latents made before either of them: nothing reaches further back than the larger window
    reach = 90 - 16 if reader_window is None else max(window, reader_window)
    assert float(moved[16:16 + reach].min()) > 0.02
    assert float(moved[:16].max()) == 0.0 and (16 + reach == 90 or float(moved[16 + reach:].max()) == 0.0)
    requests = {"r0": tokens}
    expected = lu.plain_logits(str(tmp_path / "m"), raw, requests)
    for trace in (ru.trace_portions(requests), ru.trace_last_decoded(requests, last=60)):
        outputs = ru.run_inprocess(str(tmp_path / "m"), "float32", trace, 128, page_size=16)
        lu.check(trace, outputs, expected, "float32")


@pytest.mark.parametrize("seed", [1, 2, 3, 4, 5, 6])
def test_random_configurations_replay(fake_ext, seed):
    folder = lu.random_model_folder(seed)
    raw, page = lu.CONFIGS[f"random{seed}"]
    requests = ru.make_requests(raw["vocab"], (1, 2, 23, 61, 37), seed=seed)
    expected = lu.plain_logits(folder, raw, requests)
    trace = ru.trace_mixed(requests, 64 * 4, seed=seed)
    outputs = ru.run_inprocess(folder, "float32", trace, 64 * 4, page_size=page)
    lu.check(trace, outputs, expected, "float32")
