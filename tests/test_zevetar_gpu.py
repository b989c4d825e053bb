"""Whole Zevetar models through the engine on the GPU against the plain restatement (``plain_zevetar.py``): prompts at once, decoding
through the latents' pages and the recurrences' states, portions of every size, mixed batches with pages and slots that are freed and
used again, rows at the edges of every window and far back in a state, long decoding, and greedy generation through the entry points."""

from __future__ import annotations

import copy
import json

import numpy as np
import pytest
import torch

import plain_zevetar as plain
from tiny_zevetar import CONFIGS, latent, layer, model, retention, write_model

pytestmark = pytest.mark.gpu

FLOAT32_LIMIT = 2e-4   # of the logits' spread; 32-bit sums of a few hundred terms stay far below
# In bfloat16 three rows in a hundred may be over the limit, by no more than five times: a recurrence's read-out that nearly cancels (at a
# request's first tokens) is divided by its root mean square with its rounding.
BFLOAT16_LIMIT = 0.08
MAX_SLACK = 0.12   # by how much a left-out expert's score may beat a chosen one's where bfloat16 rounding turned a close call


@pytest.fixture(scope="module")
def models(tmp_path_factory):
    root = tmp_path_factory.mktemp("zevetar")
    return {name: write_model(root / name, config, 70 + seed) for seed, (name, config) in enumerate(CONFIGS.items())}


def tokens_for(config: dict, count: int, seed: int) -> list[int]:
    return np.random.default_rng(seed).integers(0, config["vocab"], size=count).tolist()


def routers(config: dict) -> list[int]:
    return [index for index, entry in enumerate(config["layers"]) if entry["mlp"] is not None and entry["mlp"]["kind"] == "moe"]


def follows_choices(config: dict, dtype: str) -> bool:
    """bfloat16 rounding of a router's input can turn a close call between two experts, which no limit on rounding errors covers: there
    the plain implementation is given the engine's choices, which are checked against its own scores."""
    return dtype == "bfloat16" and bool(routers(config))


def expected(config: dict, weights: dict, tokens: list[int], choices: dict | None = None) -> np.ndarray:
    slack: list[float] = []
    logits = plain.forward(config, weights, tokens, choices=choices, slack=slack).numpy()
    assert sum(value > MAX_SLACK for value in slack) <= max(1, 0.01 * len(tokens)), sorted(slack)[-3:]   # the few rows over the limit choose from another input
    return logits


def load_engine(folder, dtype: str, max_tokens: int = 1024, config: dict | None = None, **options):
    from lalamo_b200.engine.engine import Engine, EngineConfig

    if config is not None and follows_choices(config, dtype):
        options.setdefault("cuda_graphs", False)   # the routers' choices are read after every launch
    return Engine.load(folder, EngineConfig(dtype=dtype, page_size=16, max_tokens=max_tokens, max_requests=4, poison_freed=True, **options))


def row_errors(got: np.ndarray, want: np.ndarray) -> np.ndarray:
    """Per row: the spread of the difference (its mean taken off) over the spread of the wanted logits."""
    difference = got - want
    difference = difference - difference.mean(axis=-1, keepdims=True)
    centred = want - want.mean(axis=-1, keepdims=True)
    return np.sqrt((difference**2).mean(axis=-1)) / np.sqrt((centred**2).mean())


def run_schedule(engine, requests: dict[str, list[int]], schedule: list[list[tuple[str, int]]], choices: dict | None = None) -> dict[str, np.ndarray]:
    """Feeds the requests' tokens in the schedule's portions (every step one batch), asks for every position's logits, ends a request
    with its last token, and checks the cache's books after every step.  ``choices`` (a dict) receives what the routers chose: request ->
    router (in the order they run) -> list of [tokens, top]; needs an engine that replays nothing."""
    from lalamo_b200 import ops
    from lalamo_b200.engine.executor import StepEntry

    done = {name: 0 for name in requests}
    rows: dict[str, list[np.ndarray]] = {name: [] for name in requests}
    seen: list[torch.Tensor] = []
    route = ops.moe_route

    def recording_route(*args, **kwargs):
        result = route(*args, **kwargs)
        seen.append(result[0])
        return result

    if choices is not None:
        ops.moe_route = recording_route
    try:
        for step in schedule:
            entries = []
            for name, count in step:
                if done[name] == 0:
                    engine.admit(name)
                entries.append(StepEntry(name, requests[name][done[name] : done[name] + count], list(range(count))))
            seen.clear()
            logits = engine.step(entries).float().cpu().numpy()
            offset = 0
            for name, count in step:
                rows[name].append(logits[offset : offset + count])
                if choices is not None:
                    for router, chosen in enumerate(seen):
                        choices.setdefault(name, {}).setdefault(router, []).append(chosen[offset : offset + count].cpu())
                offset += count
                done[name] += count
                if done[name] == len(requests[name]):
                    engine.release(name)
            engine.executor.check_status()
            engine.cache.check()
    finally:
        ops.moe_route = route
    assert all(done[name] == len(tokens) for name, tokens in requests.items())
    return {name: np.concatenate(parts) for name, parts in rows.items()}


def compare(engine, config: dict, weights: dict, requests: dict[str, list[int]], schedule: list, dtype: str) -> dict[str, np.ndarray]:
    """Runs the schedule and holds every request's rows to the limit of the type against the plain implementation."""
    follow = follows_choices(config, dtype)
    recorded: dict = {}
    got = run_schedule(engine, requests, schedule, recorded if follow else None)
    for name, tokens in requests.items():
        choices = {index: torch.cat(recorded[name][router]) for router, index in enumerate(routers(config))} if follow else None
        errors = row_errors(got[name], expected(config, weights, tokens, choices))
        worst = (name, int(errors.argmax()), float(errors.max()))
        if dtype == "float32":
            assert errors.max() < FLOAT32_LIMIT, worst
        else:
            assert errors.max() < 5 * BFLOAT16_LIMIT and (errors > BFLOAT16_LIMIT).sum() <= max(1, 0.03 * len(errors)), worst
    return got


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("name", list(CONFIGS))
def test_a_prompt_at_once_and_token_by_token(models, name, dtype):
    folder, weights = models[name]
    config = CONFIGS[name]
    tokens = tokens_for(config, 90, 5)
    engine = load_engine(folder, dtype, config=config)
    compare(engine, config, weights, {"a": tokens}, [[("a", len(tokens))]], dtype)
    # the first 21 at once, the rest one by one: windows pass over decoded tokens, steps replay from recordings
    compare(engine, config, weights, {"b": tokens}, [[("b", 21)]] + [[("b", 1)]] * (len(tokens) - 21), dtype)
    # from the very first token on, one by one: empty states, a cache of one key
    compare(engine, config, weights, {"c": tokens[:40]}, [[("c", 1)]] * 40, dtype)
    assert engine.cache.free_pages() == engine.cache.num_pages


@pytest.mark.parametrize("name", ["A", "B", "C", "D"])
def test_the_stream_after_every_layer(models, name):
    from lalamo_b200 import ops

    folder, weights = models[name]
    config = CONFIGS[name]
    tokens = tokens_for(config, 70, 8)
    wanted: list = []
    plain.forward(config, weights, tokens, wanted)
    engine = load_engine(folder, "float32", cuda_graphs=False)
    seen: list[torch.Tensor] = []
    for block in engine.model.blocks:
        def tapped(residual, pending, step, cache, inner=block.forward):
            terms = inner(residual, pending, step, cache)
            stream = residual.clone()
            ops.residual_add(stream, terms)
            seen.append(stream.double().cpu())
            return terms
        block.forward = tapped
    run_schedule(engine, {"a": tokens}, [[("a", len(tokens))]])
    assert len(seen) == len(wanted) == len(config["layers"])
    for index, (got, want) in enumerate(zip(seen, wanted)):
        assert float((got - want).abs().max()) < 2e-4 * float(want.abs().max()), index


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("name", list(CONFIGS))
def test_portions_of_every_size(models, name, dtype):
    folder, weights = models[name]
    config = CONFIGS[name]
    tokens = tokens_for(config, 150, 6)
    engine = load_engine(folder, dtype, config=config)
    for cuts in ([2, 3, 2, 5, 1, 17, 1, 1, 33, 2, 16, 31, 36], [64, 2, 2, 2, 48, 32], [7] * 21 + [3], [1, 2, 147]):
        assert sum(cuts) == len(tokens)
        compare(engine, config, weights, {"a": tokens}, [[("a", count)] for count in cuts], dtype)


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("name", ["A", "B", "C", "D"])
def test_mixed_batches_with_pages_and_slots_used_again(models, name, dtype):
    """Up to four live requests of unequal lengths, portions beside single tokens; requests end and others take their
    slots and pages (which were overwritten with NaN when they were given back); a pool smaller than the sum."""
    folder, weights = models[name]
    config = CONFIGS[name]
    lengths = {"a": 70, "b": 1, "c": 33, "d": 2, "e": 95, "f": 18, "g": 64}
    requests = {key: tokens_for(config, count, 10 + index) for index, (key, count) in enumerate(lengths.items())}
    schedule = [
        [("a", 30), ("b", 1), ("c", 2)],
        [("a", 1), ("c", 1), ("d", 1), ("e", 17)],
        [("a", 1), ("c", 14), ("d", 1), ("e", 1)],
        [("a", 16), ("c", 1), ("e", 40), ("f", 3)],
        [("a", 1), ("c", 15), ("e", 1), ("f", 15)],
        [("a", 21), ("e", 2), ("g", 33)],
        [("e", 33), ("g", 1)],
        [("e", 1), ("g", 30)],
    ]
    engine = load_engine(folder, dtype, max_tokens=288, config=config)
    got = compare(engine, config, weights, requests, schedule, dtype)
    if dtype == "float32":
        # each request alone, in one piece, on the same engine: what the batch and the cutting change is rounding
        for key in ("a", "e"):
            alone = run_schedule(engine, {key: requests[key]}, [[(key, len(requests[key]))]])[key]
            assert row_errors(got[key], alone).max() < 5e-5, key
    assert engine.cache.free_pages() == engine.cache.num_pages


def test_a_request_left_out_of_steps_goes_on_later(models):
    folder, weights = models["A"]
    config = CONFIGS["A"]
    requests = {key: tokens_for(config, count, 90 + count) for key, count in (("a", 60), ("b", 45), ("c", 12))}
    schedule = [[("a", 9)], [("b", 40)], [("b", 5), ("c", 3)], [("a", 1), ("c", 9)], [("a", 50)]]
    compare(load_engine(folder, "float32", max_tokens=160), config, weights, requests, schedule, "float32")


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_long_decoding(models, dtype):
    folder, weights = models["C"]
    config = CONFIGS["C"]
    tokens = tokens_for(config, 320, 22)
    compare(load_engine(folder, dtype, config=config), config, weights, {"a": tokens}, [[("a", 4)]] + [[("a", 1)]] * 316, dtype)


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("name", ["A", "C"])
def test_long_portions_beside_a_short_request(models, name, dtype):
    folder, weights = models[name]
    config = CONFIGS[name]
    requests = {"a": tokens_for(config, 1000, 41), "b": tokens_for(config, 30, 42)}
    # 800 tokens at once: long enough for the recurrence to run as chunks side by side where its head shape makes that pay
    schedule = [[("a", 800), ("b", 5)], [("a", 1), ("b", 20)], [("a", 190), ("b", 1)], [("b", 4), ("a", 9)]]
    compare(load_engine(folder, dtype, max_tokens=2048, config=config), config, weights, requests, schedule, dtype)


@pytest.mark.parametrize("name", ["E", "F"])
def test_recorded_steps_in_bfloat16(models, name):
    """Decoding replayed from recordings in bfloat16, in models that choose no experts (the routed ones run unrecorded in bfloat16
    above, and recorded in 32-bit)."""
    folder, weights = models[name]
    config = CONFIGS[name]
    requests = {"a": tokens_for(config, 80, 51), "b": tokens_for(config, 50, 52)}
    schedule = [[("a", 30), ("b", 1)]] + [[("a", 1), ("b", 1)]] * 49 + [[("a", 1)]]
    compare(load_engine(folder, "bfloat16", cuda_graphs=True), config, weights, requests, schedule, "bfloat16")


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("name", ["A", "C"])
def test_sublayers_on_two_streams_change_nothing(models, name, dtype, monkeypatch):
    """The two sublayers of a block side by side on two streams, recorded and not, against one after the other: the same bits."""
    from lalamo_b200.parts import block

    folder, _ = models[name]
    requests = {key: tokens_for(CONFIGS[name], count, 60 + count) for key, count in (("a", 190), ("b", 70), ("c", 45))}
    schedule = [[("a", 150), ("b", 2), ("c", 1)], [("a", 1), ("b", 40), ("c", 17)]] + [[("a", 1), ("b", 1), ("c", 1)]] * 27 + [[("a", 12), ("b", 1)]]
    results = []
    for together in (True, False):
        monkeypatch.setattr(block, "PARALLEL_STREAMS", together)
        for graphs in (True, False):
            results.append(run_schedule(load_engine(folder, dtype, cuda_graphs=graphs), requests, schedule))
    for other in results[1:]:
        assert all(np.array_equal(results[0][key], other[key]) for key in requests)


# One row that stands out.  The weights are made so that a cached row's score is tens of units above the others if its token is the marker:
# a position that sees a marker gets the marker's value, one that sees none about the mean of all others.  A marker that is seen one position
# early or late, or lost (far back, at a page's border, among the first tokens), changes that row's logits by a good part of their spread.
MARKER, OWN_WINDOW, BORROWED_WINDOW = 7, 19, 37
MARKER_POSITIONS = (0, 47, 96, 143, 200, 263)   # further apart than either window


def marker_config(heads: int, dim: int, rot_dim: int, vdim: int, q_rank: int, kv_rank: int, width: int) -> dict:
    """Two layers of latent attention, the second on the first one's rows under a longer window."""
    base = dict(heads=heads, dim=dim, rot_dim=rot_dim, vdim=vdim, q_rank=q_rank, kv_rank=kv_rank, scale=1.0, base=10.0, scaling=None)
    return model(96, width, [layer("latent_attention", latent(size=OWN_WINDOW, **base), None), layer("latent_attention", latent(size=BORROWED_WINDOW, kv_from=0, **base), None)],
                 scale=1.0, logit_scale=1.0, cap=0.0)


def make_marker_model(directory, config: dict):
    """Channel 0 of the stream is large for the marker and zero otherwise, channel 1 a constant (no layer writes to either); the first channel
    of the rows' latent reads channel 0, that of the queries' latent channel 1; the last unrotated channel of every head reads these."""
    from lalamo_b200.weights.safetensors_io import write_safetensors

    folder, weights = write_model(directory, config, 9)
    weights["embed"][:, 0] = 0.0
    weights["embed"][MARKER, 0] = 8.0
    weights["embed"][:, 1] = 4.0
    for index in range(len(config["layers"])):
        root, c = f"l{index}.", config["layers"][index]["mixer"]
        weights[root + "norm1"][:2] = 1.0
        weights[root + "ls1"].mul_(2.0)[:2] = 0.0
        weights[root + "mix.dq"][0].zero_()[1] = 4.0
        weights[root + "mix.dq.norm"][0] = 1.0
        if f"{root}mix.dkv" in weights:
            weights[root + "mix.dkv"][:, 0] = 0.0
            weights[root + "mix.dkv"][0].zero_()[0] = 4.0
            weights[root + "mix.dkv.norm"][0] = 1.0
        for name, per_head, factor in (("uq", c["dim"] + c["rot_dim"], 3.0), ("uk", c["dim"], 3.0)):
            rows = weights[f"{root}mix.{name}"]
            rows.zero_()
            for head in range(c["heads"]):
                rows[head * per_head + c["dim"] - 1, 0] = factor
    write_safetensors(folder / "model.safetensors", {name: tensor.to(torch.bfloat16) for name, tensor in weights.items()})
    return folder, weights


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("shape", [(4, 16, 8, 24, 24, 32, 64), (4, 64, 32, 64, 64, 128, 128), (3, 10, 6, 7, 13, 27, 70)], ids=str)
def test_single_rows_at_the_edges_of_both_windows(tmp_path, shape, dtype):
    config = marker_config(*shape)
    folder, weights = make_marker_model(tmp_path / "m", config)
    length = 330
    tokens = [token if token != MARKER else MARKER + 1 for token in tokens_for(config, length, 3)]
    for position in MARKER_POSITIONS:
        tokens[position] = MARKER
    want = expected(config, weights, tokens)
    # a window one position longer (shorter) keeps (loses) a marker at the row where it should leave (be seen last): the test shows what it is meant to
    for which, size in ((0, OWN_WINDOW), (1, BORROWED_WINDOW)):
        for change, rows in ((1, [p + size for p in MARKER_POSITIONS]), (-1, [p + size - 1 for p in MARKER_POSITIONS])):
            other = copy.deepcopy(config)
            other["layers"][which]["mixer"]["mask"]["size"] += change
            assert row_errors(expected(other, weights, tokens), want)[rows].min() > 3 * BFLOAT16_LIMIT
    engine = load_engine(folder, dtype, max_tokens=512)
    compare(engine, config, weights, {"a": tokens}, [[("a", length)]], dtype)
    compare(engine, config, weights, {"a": tokens}, [[("a", 2)], [("a", 15)], [("a", 118)], [("a", 2)], [("a", 100)]] + [[("a", 1)]] * 93, dtype)
    compare(engine, config, weights, {"a": tokens[:120]}, [[("a", 1)]] * 120, dtype)


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("shape", [(4, 16, 24, 12, 64), (2, 64, 128, 32, 128), (3, 12, 10, 6, 70)], ids=str)
def test_a_far_token_stays_in_the_state(tmp_path, shape, dtype):
    """Retention whose keys are nearly nothing but for two markers: every later read-out is what their values left in a state that forgets slowly,
    from one portion (or decoded token) to the next."""
    from lalamo_b200.weights.safetensors_io import write_safetensors

    heads, dim, vdim, dims, width = shape
    config = model(96, width, [layer("retention", retention(heads=heads, dim=dim, vdim=vdim, decay=[0.9995 - 0.001 * head for head in range(heads)], dims=dims, base=50.0), None)],
                   scale=1.0, logit_scale=1.0, cap=0.0)
    folder, weights = write_model(tmp_path / "m", config, 9)
    first, second = MARKER, MARKER + 1
    weights["embed"][:, 0] = 0.0
    weights["embed"][first, 0], weights["embed"][second, 0] = 5.0, 5.0
    weights["embed"][:, 1] = 4.0
    weights["l0.norm1"][:2] = 1.0
    weights["l0.ls1"].mul_(16.0)   # the mixer decides the logits
    for name, source in (("q", 1), ("k", 0)):
        rows = weights[f"l0.mix.{name}"]
        rows.zero_()
        rows[dim - 1 :: dim, source] = 2.0   # a channel past the rotated ones
    write_safetensors(folder / "model.safetensors", {name: tensor.to(torch.bfloat16) for name, tensor in weights.items()})
    length = 420
    tokens = [token if token not in (first, second) else 20 for token in tokens_for(config, length, 4)]
    tokens[3], tokens[17] = first, second
    want = expected(config, weights, tokens)
    for position in (3, 17):   # without either marker every later row is another
        other = list(tokens)
        other[position] = 20
        changed = row_errors(expected(config, weights, other), want)[40:]
        assert changed.min() > BFLOAT16_LIMIT and np.median(changed) > 3 * BFLOAT16_LIMIT
    engine = load_engine(folder, dtype, max_tokens=512)
    compare(engine, config, weights, {"a": tokens}, [[("a", length)]], dtype)
    compare(engine, config, weights, {"a": tokens}, [[("a", 10)], [("a", 190)], [("a", 2)], [("a", 158)]] + [[("a", 1)]] * 60, dtype)


def test_windows_give_pages_back_when_the_last_reader_has_passed(models):
    """The rows' owner looks back less far than one of its borrowers: pages stay for the borrower's window, and no longer."""
    folder, weights = models["A"]
    config = CONFIGS["A"]
    longest = max(entry["mixer"]["mask"]["size"] for entry in config["layers"] if entry["type"] == "latent_attention")
    engine = load_engine(folder, "float32")
    from lalamo_b200.engine.executor import StepEntry

    tokens = tokens_for(config, 200, 12)
    engine.admit("a")
    for at in range(0, 200, 50):
        engine.step([StepEntry("a", tokens[at : at + 50], [])])
    held = [sum(page >= 0 for page in blocks) for blocks in engine.cache.requests["a"].blocks.values()]
    assert held == [-(-200 // 16) - (200 - longest + 1) // 16]
    engine.release("a")
    assert engine.cache.free_pages() == engine.cache.num_pages


@pytest.mark.parametrize("name", ["A", "C"])
def test_greedy_generation_through_the_entry_point(models, name):
    from lalamo_b200 import GenerationConfig, LanguageModel

    folder, weights = models[name]
    config = CONFIGS[name]
    model_ = LanguageModel.load(folder, dtype="float32", max_tokens=1024, max_requests=4)
    prompts = [tokens_for(config, count, 30 + count) for count in (1, 9, 30, 47, 2, 18)]
    produced = model_.generate_tokens(prompts, GenerationConfig(temperature=0.0), max_output_length=12, eos_token_ids=[])
    compared = 0
    for prompt, generated in zip(prompts, produced):
        assert len(generated) == 12
        sequence = list(prompt)
        for token in generated:
            logits = expected(config, weights, sequence)[-1]
            best = np.sort(logits)[-2:]
            if best[1] - best[0] < 1e-4:
                break   # a tie within 32-bit rounding: either token is right, and what follows depends on it
            assert token == int(np.argmax(logits))
            sequence.append(token)
        else:
            compared += 1
    assert compared >= 4   # sequences compared to their end
    model_.engine.executor.check_status()
    assert model_.engine.cache.free_pages() == model_.engine.cache.num_pages


def test_command_line_and_step_replay(models, tmp_path):
    """The same model through the two programs a user runs: `generate` (greedy ids of the plain implementation) and the
    step replay that writes logits (portions, two live requests, a request that ends and another in its slot)."""
    import subprocess
    import sys
    from pathlib import Path

    from trace_client import TraceRun

    root = Path(__file__).resolve().parent.parent
    folder, weights = models["B"]
    config = CONFIGS["B"]
    prompt = tokens_for(config, 11, 77)
    prompt_file = tmp_path / "prompts.txt"
    prompt_file.write_text(" ".join(str(token) for token in prompt) + "\n")
    command = [sys.executable, "-m", "lalamo_b200", "generate", str(folder), "--prompt-ids-file", str(prompt_file), "--max-tokens", "5", "--temperature", "0",
               "--dtype", "float32", "--max-cache-tokens", "256"]
    result = subprocess.run(command, cwd=root, capture_output=True, text=True, timeout=600)
    assert result.returncode == 0, result.stderr
    produced = [json.loads(line) for line in result.stdout.splitlines() if line.startswith("{")][0]["token_ids"]
    sequence = list(prompt)
    for token in produced:
        logits = expected(config, weights, sequence)[-1]
        best = np.sort(logits)[-2:]
        if best[1] - best[0] < 1e-4:
            break
        assert token == int(np.argmax(logits))
        sequence.append(token)

    requests = {name: tokens_for(config, count, 80 + count) for name, count in (("a", 40), ("b", 9), ("c", 21))}
    wanted = {name: expected(config, weights, tokens) for name, tokens in requests.items()}
    run = TraceRun(folder, "float32", tmp_path / "out", 128, config["vocab"], poison_freed=True)
    steps = [([("a", 0, 17), ("b", 0, 2)], []), ([("a", 17, 18), ("b", 2, 9)], ["b"]), ([("a", 18, 40), ("c", 0, 21)], ["a", "c"])]
    for entries, ended in steps:
        got = run.step([{"id": name, "tokens": requests[name][lo:hi], "want": list(range(hi - lo))} for name, lo, hi in entries], ended)
        want = np.concatenate([wanted[name][lo:hi] for name, lo, hi in entries])
        assert row_errors(got, want).max() < FLOAT32_LIMIT
    assert run.close() == 0
