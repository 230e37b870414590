"""The Gosizen decoder through the engine on the GPU, in both precisions, against the plain implementation: whole
prompts, the last tokens one by one (replayed as CUDA graphs), portions down to two tokens, mixed batches in which
pages and slots are used again, decoding from the very first token, a token that stands out just inside and just outside
every window and block at page borders, and in a memory, random configurations, greedy generation through the engine's entry point and the command
line, and the replay program as a subprocess."""

import json
import subprocess
import sys

import numpy as np
import pytest
import torch

import gosizen_util as gu
import replay_util as ru
from plain import gosizen_plain as plain

pytestmark = pytest.mark.gpu

LENGTHS = (1, 2, 19, 47, 115, 70, 45)
MODES = ["whole", "last32", "portions", "mixed"]
_REQUESTS: dict = {}


def _requests(name, dtype):
    """Requests r0 .. r6 of LENGTHS and their logits; bfloat16 runs take some whose expert choices are no close calls."""
    key = (name, dtype)
    if key not in _REQUESTS:
        raw, folder = gu.CONFIGS[name][0], gu.model_folder(name)
        requests = (gu.decisive_requests(folder, raw, LENGTHS, 11) if dtype == "bfloat16"
                    else ru.make_requests(raw["vocab"], LENGTHS, seed=11))
        _REQUESTS[key] = (requests, gu.plain_logits(folder, raw, requests))
    return _REQUESTS[key]


def _trace(mode, requests, max_tokens):
    return {"whole": ru.trace_whole, "last32": ru.trace_last_decoded, "portions": ru.trace_portions,
            "mixed": lambda r: ru.trace_mixed(r, max_tokens, seed=5)}[mode](requests)


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("mode", MODES)
@pytest.mark.parametrize("name", ["G1", "G2", "G3"])
def test_replay_matches_plain(name, mode, dtype):
    raw, page = gu.CONFIGS[name]
    requests, expected = _requests(name, dtype)
    if mode != "mixed":
        requests = dict(list(requests.items())[:5])
    max_tokens = 64 * 6
    trace = _trace(mode, requests, max_tokens)
    outputs, engine = ru.run_on_device(gu.model_folder(name), dtype, trace, max_tokens, page_size=page, max_seqs=4)
    print(gu.check(trace, outputs, expected, dtype))
    if mode == "last32":
        assert engine.runner.graph_replays > 0, "single-token steps were not replayed as CUDA graphs"
    assert engine.manager.free_pages() == [g.pool.count for g in engine.manager.groups]
    engine.manager.check_invariants()


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("name", ["G1", "G3"])
def test_decoding_from_the_first_token(name, dtype):
    """Every token a step of its own for 115 positions: keys, latents and memories were written one at a time over several pages, and
    every window and block has moved past its beginning."""
    raw, page = gu.CONFIGS[name]
    requests, expected = _requests(name, dtype)
    trace = ru.trace_last_decoded({"r4": requests["r4"]}, last=114)
    outputs, engine = ru.run_on_device(gu.model_folder(name), dtype, trace, 192, page_size=page, max_seqs=2)
    print(gu.check(trace, outputs, expected, dtype))
    assert engine.runner.graph_replays >= 100


def test_eager_and_captured_single_token_steps_agree():
    raw, page = gu.CONFIGS["G1"]
    requests = ru.make_requests(raw["vocab"], (40, 33), seed=3)
    trace = ru.trace_last_decoded(requests, last=12)
    folder = gu.model_folder("G1")
    with_graphs, engine = ru.run_on_device(folder, "float32", trace, 128, page_size=page, max_seqs=4)
    assert engine.runner.graph_replays > 0
    without, _ = ru.run_on_device(folder, "float32", trace, 128, page_size=page, max_seqs=4, cuda_graphs=False)
    for step in trace.expect:
        torch.testing.assert_close(torch.from_numpy(with_graphs[step]), torch.from_numpy(without[step]), atol=1e-5, rtol=1e-5)


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_a_requests_logits_do_not_depend_on_its_neighbours(dtype):
    """Four unequal requests decoding together, each also alone on an engine of its own."""
    raw, page = gu.CONFIGS["G3"]
    requests = {r: t for r, t in _requests("G3", "bfloat16")[0].items() if r in ("r2", "r3", "r5", "r6")}
    tail = 5
    together = ru.Trace()
    together.add([(r, t[:-tail], 0, [len(t) - tail - 1] if len(t) > tail else []) for r, t in requests.items() if len(t) > tail])
    for k in range(tail):
        together.add([(r, [t[len(t) - tail + k]], len(t) - tail + k, [0]) for r, t in requests.items()],
                     end=list(requests) if k == tail - 1 else [])
    folder = gu.model_folder("G3")
    outputs, _ = ru.run_on_device(folder, dtype, together, 64 * 6, page_size=page, max_seqs=4)
    both = {}
    for step, rows in together.expect.items():
        for (rid, pos), row in zip(rows, outputs[step].reshape(len(rows), -1)):
            both[rid, pos] = row
    for rid, toks in requests.items():
        trace = ru.trace_last_decoded({rid: toks}, last=tail)
        alone, _ = ru.run_on_device(folder, dtype, trace, 64 * 6, page_size=page, max_seqs=4)
        for step, rows in trace.expect.items():
            got = alone[step].reshape(len(rows), -1)
            for (_, pos), row in zip(rows, got):
                if (rid, pos) in both:
                    scale = float(np.sqrt((row ** 2).mean()))
                    assert float(np.abs(row - both[rid, pos]).max()) <= (2e-5 if dtype == "float32" else 0.1) * scale


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("kind,size,page", [("latent", 64, 16), ("latent", 97, 64), ("latent", 16, 64), ("left", 64, 16),
                                            ("left", 100, 64), ("left", 33, 16), ("right", 0, 16)])
def test_a_marked_token_shows_exactly_where_it_is_seen(dtype, kind, size, page, tmp_path):
    """Every query looks for one token's key: its logits say whether it sees it.  The token stands at page borders, at a
    sequence's first place and far back; each position just inside and just outside the window or the block is looked at
    in a prompt's portion, in portions of changing size and decoded alone.  The plain logits are asserted to move when
    the token is taken away exactly where it is seen (in the memory: for hundreds of tokens)."""
    folder = str(tmp_path / "marked")
    raw = gu.marked_model(folder, kind, size)
    w = gu.plain_weights(folder)
    length = 250
    others = [t for t in range(61) if t != gu.MARK]
    requests, stops = {}, {}
    for i, where in enumerate((0, page - 1, page, 2 * page + 1)):
        g = torch.Generator().manual_seed(i)
        tokens = [others[int(k)] for k in torch.randint(0, len(others), (length,), generator=g)]
        tokens[where] = gu.MARK
        requests[f"r{i}"] = tokens
        stops[f"r{i}"] = min(length, {"latent": where + size, "left": size and (where // size + 1) * size, "right": length}[kind])
    blank = list(requests["r2"])
    blank[page] = others[0]
    expected = gu.plain_logits(folder, raw, requests)
    moved = (plain.forward(raw, w, blank).float() - expected["r2"]).abs().amax(dim=1)
    stop = stops["r2"]
    assert float(moved[page:stop].min()) > 0.02, "the test's weights do not make the token show"
    assert float(moved[:page].max()) == 0.0 and (stop == length or float(moved[stop:].max()) == 0.0)
    max_tokens = 64 * 8
    for trace in (ru.trace_whole(requests), ru.trace_portions(requests)):
        outputs, _ = ru.run_on_device(folder, dtype, trace, max_tokens, page_size=page, max_seqs=2)
        gu.check(trace, outputs, expected, dtype)
    # decoded alone across the edge
    trace, edge = ru.Trace(), min(stop, length - 4)
    trace.add([("r2", requests["r2"][:edge - 4], 0, [])])
    for p in range(edge - 4, edge + 4):
        trace.add([("r2", requests["r2"][p:p + 1], p, [0])])
    trace.add([], end=["r2"])
    outputs, _ = ru.run_on_device(folder, dtype, trace, max_tokens, page_size=page, max_seqs=2)
    gu.check(trace, outputs, expected, dtype)


@pytest.mark.parametrize("seed", list(range(1, 13)))
def test_random_configuration(seed):
    folder = gu.random_model_folder(seed)
    raw, page = gu.CONFIGS[f"random{seed}"]
    requests = ru.make_requests(raw["vocab"], (1, 2, 23, 61, 90, 37), seed=seed)
    expected = gu.plain_logits(folder, raw, requests)
    max_tokens = 64 * 5
    mixed = ru.trace_mixed(requests, max_tokens, seed=seed)
    outputs, engine = ru.run_on_device(folder, "float32", mixed, max_tokens, page_size=page, max_seqs=4)
    gu.check(mixed, outputs, expected, "float32", loose=5.0)
    engine.manager.check_invariants()
    tail = ru.trace_last_decoded(requests, last=20)
    outputs, engine = ru.run_on_device(folder, "float32", tail, max_tokens, page_size=page, max_seqs=4)
    gu.check(tail, outputs, expected, "float32", loose=5.0)
    assert engine.runner.graph_replays > 0
    outputs, engine = ru.run_on_device(folder, "bfloat16", mixed, max_tokens, page_size=page, max_seqs=4)
    assert all(np.isfinite(rows).all() for rows in outputs.values())


@pytest.mark.parametrize("name", ["G1", "G3"])
def test_greedy_generation_through_the_entry_point(name):
    from ampere_kv_engine_b200.engine.engine import Engine
    raw, page = gu.CONFIGS[name]
    folder = gu.model_folder(name)
    w = gu.plain_weights(folder)
    prompts = list(ru.make_requests(raw["vocab"], (3, 30, 61), seed=41).values())
    engine = Engine.from_pretrained(folder, dtype="float32", device="cuda", page_size=page, num_pages=16,
                                    max_batch_tokens=24, max_seqs=4)
    got = engine.generate(prompts, max_new_tokens=8, ignore_eos=True)
    assert got == [plain.greedy_generate(raw, w, p, 8) for p in prompts]
    # five requests through four slots: one waits, then takes pages and a slot that were used before
    more = prompts + [prompts[1][:7], prompts[2][:11]]
    again = engine.generate(more, max_new_tokens=8, ignore_eos=True)
    assert again[:3] == got and again[3:] == [plain.greedy_generate(raw, w, p, 8) for p in more[3:]]
    engine.manager.check_invariants()
    # bfloat16: every chosen token is (nearly) the best one of the plain logits
    prompts = [t[:61] for t in list(_requests(name, "bfloat16")[0].values())[1:4]]
    engine = Engine.from_pretrained(folder, dtype="bfloat16", device="cuda", page_size=page, num_pages=16, max_seqs=4)
    for prompt, out in zip(prompts, engine.generate(prompts, max_new_tokens=2, ignore_eos=True)):
        logits = plain.forward(raw, w, list(prompt))[-1]
        assert float(logits.max() - logits[out[0]]) <= 0.05 * float(logits.max() - logits.min()), \
            "bfloat16 picked a token far from the best"


def test_command_line_and_replay_program():
    raw, page = gu.CONFIGS["G1"]
    folder = gu.model_folder("G1")
    prompt = list(ru.make_requests(raw["vocab"], (17,), seed=51).values())[0]
    cmd = [sys.executable, "-m", "ampere_kv_engine_b200.runner", "--model", folder, "--mode", "generate", "--dtype",
           "float32", "--prompt-ids", ",".join(map(str, prompt)), "--max-new-tokens", "5", "--ignore-eos",
           "--page-size", str(page)]
    proc = subprocess.run(cmd, cwd=ru.ROOT, capture_output=True, text=True, timeout=600)
    assert proc.returncode == 0, proc.stderr[-3000:]
    line = next(l for l in proc.stdout.splitlines() if l.startswith("generated_token_ids"))
    assert json.loads(line.split("=", 1)[1]) == plain.greedy_generate(raw, gu.plain_weights(folder), prompt, 5)
    # the replay program itself, as a user starts it
    requests = ru.make_requests(raw["vocab"], (5, 40), seed=8)
    trace = ru.trace_portions(requests)
    outputs = ru.run_subprocess(folder, "float32", trace, 128, page_size=page)
    gu.check(trace, outputs, gu.plain_logits(folder, raw, requests), "float32")
