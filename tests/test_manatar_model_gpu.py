"""The Manatar decoder through the engine's own model, cache manager and step function, against
the plain implementation: every way of cutting the same requests into steps gives the plain
logits at every position.  Pools are small, so pages and slots are used again (free pages are
filled with NaN); layers that use another layer's keys keep a filter state of their own, and the
embedding keeps the previous token.
"""
from __future__ import annotations

import json
import os
import subprocess
import sys

import numpy as np
import pytest

import traces
from conftest import ROOT, random_tokens
from engine_harness import Harness, assert_close
from manatar_configs import CONFIGS, PAGE_SIZE, make_folder
from plain_manatar import PlainManatar, to_bfloat16

pytestmark = pytest.mark.gpu

LENGTHS = {"mixed": (1, 2, 9, 33, 90), "plain": (3, 17, 40, 75), "fast": (5, 70, 150, 420),
           "odd": (4, 11, 50, 100)}
NAMES = ("mixed", "plain", "fast", "odd")
CASES = [(name, dtype) for dtype in ("float32", "bfloat16") for name in NAMES]
# float32: double against float32 sums and recurrences, in values of logits whose spread is
# about one.  bfloat16: see check_rows.
FLOAT32 = dict(atol=2e-4, rtol=2e-4)


def relative_error(got: np.ndarray, want: np.ndarray) -> np.ndarray:
    """Per row: the root mean square of the difference (its mean taken off) over the spread of
    the wanted logits."""
    difference = got.astype(np.float64) - want
    difference -= difference.mean(axis=-1, keepdims=True)
    spread = want - want.mean(axis=-1, keepdims=True)
    return np.sqrt((difference ** 2).mean(axis=-1)) / np.sqrt((spread ** 2).mean())


def make_requests(name: str, extra: int = 0):
    vocab = CONFIGS[name]["vocab"]
    return {f"r{index}": random_tokens(vocab, length + extra, seed=61 * len(name) + index)
            for index, length in enumerate(LENGTHS[name])}


@pytest.fixture(scope="module")
def models(model_root):
    cache = {}

    def get(name: str, dtype: str):
        if (name, dtype) not in cache:
            folder = make_folder(model_root, name, dtype)
            cache[(name, dtype)] = (folder, PlainManatar(folder, dtype))
        return cache[(name, dtype)]
    return get


def shaken(folder: str, seed: int) -> PlainManatar:
    """The plain implementation with a relative change of 6e-8 wherever it can round: rows where the maps
    or a recurrence's terms nearly cancel, and are normed to their usual size again, carry it a
    thousandfold."""
    rng = np.random.default_rng(seed)
    plain = PlainManatar(folder, "float32")
    plain.round = lambda values: values * (1.0 + 6e-8 * rng.normal(size=np.shape(values)))
    return plain


class Expected:
    """The plain logits of a set of requests, and how far rounding alone moves each row (``noise`` for
    float32, ``moved`` for bfloat16)."""

    def __init__(self, folder, plain, dtype, requests) -> None:
        self.dtype = dtype
        self.logits, self.held = {}, {}
        for name, tokens in requests.items():
            self.logits[name] = plain.forward(tokens)
            # bfloat16: from the first close call of a router on, a row may rest on another choice
            close_calls = np.nonzero(plain.margins < CLOSE_CALL)[0] if dtype == "bfloat16" else []
            self.held[name] = int(close_calls[0]) if len(close_calls) else len(tokens)
        self.moved, self.noise = {}, {name: np.zeros(len(tokens)) for name, tokens in requests.items()}
        for seed in range(2 if dtype == "float32" else 0):
            other = shaken(folder, seed)
            for name, tokens in requests.items():
                change = np.abs(other.forward(tokens) - self.logits[name]).max(axis=1)
                self.noise[name] = np.maximum(self.noise[name], change)
        if dtype == "bfloat16":
            exact = PlainManatar(folder, "float32")
            self.moved = {name: relative_error(self.logits[name], exact.forward(tokens))
                          for name, tokens in requests.items()}
            # what rounding does to a row is one draw; a row where the maps or the recurrence's terms
            # nearly cancel shows in others (every rounded value moved by half a unit or so first)
            for seed in range(3):
                rng = np.random.default_rng(seed)
                other = PlainManatar(folder, "bfloat16")
                other.round = lambda values: to_bfloat16(
                    values * (1.0 + 2.0 ** -9 * rng.normal(size=np.shape(values))))
                for name, tokens in requests.items():
                    self.moved[name] = np.maximum(
                        self.moved[name], 0.7 * relative_error(other.forward(tokens), self.logits[name]))
            # and the rows of the model that it moves most say how large the draws are
            self.floor = float(np.quantile(np.concatenate(list(self.moved.values())), 0.9))


@pytest.fixture(scope="module")
def expectations(models):
    cache = {}

    def get(name: str, dtype: str, extra: int = 0):
        if (name, dtype, extra) not in cache:
            folder, plain = models(name, dtype)
            cache[(name, dtype, extra)] = Expected(folder, plain, dtype, make_requests(name, extra))
        return cache[(name, dtype, extra)]
    return get


# Distance of a router's last chosen logit from the best one left out that rounding its input to
# bfloat16 may turn around.
CLOSE_CALL = 0.02


def check_rows(out, expected, rows, what):
    """float32: value by value.  bfloat16: the plain implementation rounds where the engine
    stores, so what is left are activations on the other side of a rounding boundary; a row may
    differ by a few per cent of the logits' spread or by a multiple of what rounding all
    activations moves it, or moves the model's more sensitive rows."""
    want = np.stack([expected.logits[name][position] for name, position in rows])
    if expected.dtype == "float32":
        steady = np.array([expected.noise[name][position] < 1e-5 for name, position in rows])
        assert_close(out[steady], want[steady].astype(np.float32), what, **FLOAT32)
        for index in np.nonzero(~steady)[0]:
            name, position = rows[index]
            assert_close(out[index:index + 1], want[index:index + 1].astype(np.float32),
                         f"{what} {name} position {position}",
                         atol=FLOAT32["atol"] + 30.0 * expected.noise[name][position], rtol=FLOAT32["rtol"])
        return
    assert np.isfinite(out).all(), what
    error = relative_error(out, want)
    allowed = np.array([max(0.05, 4.0 * max(expected.moved[name][position], expected.floor))
                        for name, position in rows])
    resting = np.array([position >= expected.held[name] for name, position in rows])
    bad = np.nonzero((error > allowed) & ~resting)[0]
    assert bad.size == 0, (f"{what}: row {rows[bad[0]]} differs by {error[bad[0]]:.3f} of the "
                           f"logits' spread, allowed {allowed[bad[0]]:.3f}")


def replay(harness: Harness, steps, expected, what: str):
    positions = {}
    for step in steps:
        rows = traces.labels(step, positions)
        out = harness.run([(e["id"], e["tokens"], e["want"]) for e in step["entries"]])
        for name in step["end"]:
            harness.end(name)
        if rows:
            check_rows(out, expected, rows, f"{what} step {step['step']}")
        harness.cache.check()
    assert not harness.cache.live_requests()


def test_most_bfloat16_rows_are_held_to_the_tolerance(expectations):
    for name in NAMES:
        expected = expectations(name, "bfloat16", 30)
        moved = np.concatenate([rows[:expected.held[request]] for request, rows in expected.moved.items()])
        assert (4.0 * moved > 0.1).mean() <= 0.5, name
        lengths = [len(rows) for rows in expected.moved.values()]
        assert sum(min(expected.held[request], length) for request, length
                   in zip(expected.moved, lengths)) >= 0.5 * sum(lengths), name


@pytest.mark.parametrize("name,dtype", CASES)
def test_whole_requests(name, dtype, models, expectations):
    harness = Harness(models(name, dtype)[0], dtype, PAGE_SIZE[name], num_pages=48)
    replay(harness, traces.whole(make_requests(name)), expectations(name, dtype),
           f"{name} {dtype} whole")


@pytest.mark.parametrize("name", NAMES)
def test_residual_after_every_layer_run(name, models):
    folder, plain = models(name, "float32")
    harness = Harness(folder, "float32", PAGE_SIZE[name], num_pages=48)
    tokens = make_requests(name)["r3"]
    seen = []
    harness.model.after_entry = lambda index, rows: seen.append(rows.float().cpu().numpy().copy())
    harness.whole("a", tokens)
    states = plain.hidden_states(tokens)
    assert len(seen) == len(states)
    moved = [np.abs(other - want).max(axis=1)
             for other, want in zip(shaken(folder, 0).hidden_states(tokens), states)]
    for index, (got, want, noise) in enumerate(zip(seen, states, moved)):
        spread = float(np.abs(want).max())
        error = np.abs(got - want).max(axis=1)
        assert (error <= 3e-5 * spread + 30.0 * noise).all(), \
            f"{name} layer {index}: row {error.argmax()} differs by {error.max():.2e}"


@pytest.mark.parametrize("name,dtype", CASES)
def test_tail_decoded_one_by_one(name, dtype, models, expectations):
    harness = Harness(models(name, dtype)[0], dtype, PAGE_SIZE[name], num_pages=48)
    replay(harness, traces.tail_decoded(make_requests(name, extra=30), tail=60),
           expectations(name, dtype, 30), f"{name} {dtype} tail")


@pytest.mark.parametrize("name,dtype", CASES)
def test_portions_of_changing_size(name, dtype, models, expectations):
    harness = Harness(models(name, dtype)[0], dtype, PAGE_SIZE[name], num_pages=48)
    replay(harness, traces.chunked(make_requests(name, extra=30)), expectations(name, dtype, 30),
           f"{name} {dtype} portions")


@pytest.mark.parametrize("name,dtype", [("mixed", "float32"), ("odd", "float32"),
                                        ("mixed", "bfloat16"), ("plain", "bfloat16")])
def test_portions_of_two_tokens(name, dtype, models, expectations):
    harness = Harness(models(name, dtype)[0], dtype, PAGE_SIZE[name], num_pages=48)
    replay(harness, traces.chunked(make_requests(name), portions=(2,)), expectations(name, dtype),
           f"{name} {dtype} twos")


@pytest.mark.parametrize("name", NAMES)
def test_every_token_alone_from_the_first(name, models, expectations):
    """Decoding from position 0: the filter reaches in front of the sequence, the recurrence's state
    and its maximum are zero, and the first token has its own row of the table of pairs."""
    harness = Harness(models(name, "float32")[0], "float32", PAGE_SIZE[name], num_pages=48)
    tokens = make_requests(name)["r2"]
    expected = expectations(name, "float32")
    for position, token in enumerate(tokens):
        out = harness.run([("a", [token], [0])])
        check_rows(out, expected, [("r2", position)], f"{name} position {position}")
    harness.end("a")


@pytest.mark.parametrize("name,dtype", CASES)
@pytest.mark.parametrize("seed", [0, 1])
def test_mixed_batches_over_a_small_pool(name, dtype, seed, models, expectations):
    requests = make_requests(name, extra=30)
    steps = traces.mixed(requests, max_live=3, seed=seed)
    page = PAGE_SIZE[name]
    pages = -(-traces.live_token_need(steps, round_to=page) // page)
    harness = Harness(models(name, dtype)[0], dtype, page, num_pages=pages, max_requests=3)
    replay(harness, steps, expectations(name, dtype, 30), f"{name} {dtype} mixed")
    stats = harness.cache.stats()
    assert stats["groups"] and all(group["reuses"] > 0 for group in stats["groups"]), \
        "no page was used again"


@pytest.mark.parametrize("name", ["mixed", "odd"])
def test_a_long_request_with_a_long_decoded_tail(name, models):
    """300 tokens, the last 120 decoded one by one."""
    folder, plain = models(name, "float32")
    tokens = random_tokens(CONFIGS[name]["vocab"], 300, seed=5)
    harness = Harness(folder, "float32", PAGE_SIZE[name], num_pages=40, max_requests=1)
    expected = Expected(folder, plain, "float32", {"long": tokens})
    cursor = 0
    sizes = [13, 8, 8, 3, 11, 2, 29] * 5
    while cursor < len(tokens):
        size = 1 if cursor >= 180 else min(sizes.pop(0), 180 - cursor)
        out = harness.run([("long", tokens[cursor:cursor + size], range(size))])
        check_rows(out, expected, [("long", cursor + i) for i in range(size)],
                   f"positions from {cursor}")
        cursor += size
        harness.cache.check()
    harness.end("long")


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_a_batch_gives_what_each_request_gives_alone(dtype, models):
    """The same engine, requests of very different lengths side by side and one after the other."""
    folder, plain = models("fast", dtype)
    requests = {f"r{i}": random_tokens(640, length, seed=90 + i)
                for i, length in enumerate((1, 2, 40, 97, 250))}
    harness = Harness(folder, dtype, 16, num_pages=64, max_requests=5)
    alone = {name: harness.whole(name, tokens) for name, tokens in requests.items()}
    together = harness.run([(name, tokens, range(len(tokens))) for name, tokens in requests.items()])
    cursor = 0
    for name, tokens in requests.items():
        part = together[cursor:cursor + len(tokens)]
        cursor += len(tokens)
        if dtype == "float32":
            assert_close(part, alone[name], name, atol=1e-4, rtol=1e-4)
        else:
            error = relative_error(part, alone[name].astype(np.float64))
            plain.forward(tokens)
            calls = np.nonzero(plain.margins < CLOSE_CALL)[0]
            assert error[:int(calls[0]) if len(calls) else len(tokens)].max(initial=0.0) < 0.08, name
        harness.end(name)


@pytest.mark.parametrize("name,dtype", [("mixed", "float32"), ("fast", "bfloat16"),
                                        ("plain", "float32"), ("odd", "float32")])
def test_greedy_generation_through_the_engine(name, dtype, models):
    """``Engine.generate``: scheduler, continuous batching, CUDA graphs and sampling, several
    requests at once.  Each generated token must be (within rounding) the best token of the
    plain logits for the sequence so far."""
    from helix_runtime_b200 import Engine
    folder, plain = models(name, dtype)
    vocab = CONFIGS[name]["vocab"]
    prompts = [random_tokens(vocab, length, seed=300 + length) for length in (3, 25, 61)]
    engine = Engine.from_pretrained(folder, dtype=dtype, page_size=PAGE_SIZE[name], num_pages=64,
                                    max_running_requests=3, max_tokens_per_iteration=64,
                                    max_prefill_chunk=24, poison_free_pages=True)
    results = engine.generate(prompts, max_new_tokens=24)
    assert engine.graphs is not None and engine.graphs.captures > 0
    exact = PlainManatar(folder, "float32")
    for prompt, result in zip(prompts, results):
        assert len(result.generated_tokens) == 24
        tokens = list(prompt) + result.generated_tokens
        moved = np.zeros(len(tokens))
        logits = plain.forward(tokens)
        if dtype == "bfloat16":
            moved = np.abs(exact.forward(tokens) - logits).max(axis=1)
        calls = np.nonzero(plain.margins < CLOSE_CALL)[0] if dtype == "bfloat16" else []
        until = min(len(tokens), int(calls[0]) + 1 if len(calls) else len(tokens))
        for place in range(len(prompt), until):
            row = logits[place - 1]
            slack = 1e-3 if dtype == "float32" else max(0.1, 3.0 * moved[place - 1])
            assert row[tokens[place]] >= row.max() - slack, \
                f"token {tokens[place]} at position {place} is not the plain model's choice"


@pytest.mark.parametrize("name", ["mixed", "fast"])
def test_the_next_turn_adopts_pages_and_state(name, models):
    """A conversation's next turn with the prefix index on: what the engine keeps of the first
    prompt (pages, the filters' inputs, the recurrences' state, the previous token) gives the logits'
    choices of a sequence computed from the start."""
    from helix_runtime_b200 import Engine
    folder, plain = models(name, "float32")
    vocab, page = CONFIGS[name]["vocab"], PAGE_SIZE[name]
    engine = Engine.from_pretrained(folder, dtype="float32", page_size=page, num_pages=96,
                                    max_running_requests=2, max_tokens_per_iteration=64,
                                    prefix_cache_entries=8, poison_free_pages=True)
    for length in (page * 5 + 3, page * 8 + 1, page * 13 + page - 1):
        first = random_tokens(vocab, length, seed=length)
        engine.generate([first], max_new_tokens=2)
        again = first + random_tokens(vocab, 9, seed=length + 1)
        result = engine.generate([again], max_new_tokens=6)[0]
        assert engine.request(result.request_id).reused_tokens == length // page * page
        tokens = again + result.generated_tokens
        logits = plain.forward(tokens)
        for place in range(len(again), len(tokens)):
            assert logits[place - 1][tokens[place]] >= logits[place - 1].max() - 1e-3
    engine.cache.check()


def test_trace_replay_as_a_user_runs_it(models, expectations, tmp_path):
    """``bin/trace_run`` in a process of its own, fed a trace of mixed batches over a pool made
    for the live requests only; the logits it writes are the plain implementation's."""
    name, dtype = "mixed", "float32"
    folder = models(name, dtype)[0]
    expected = expectations(name, dtype, 30)
    steps = traces.mixed(make_requests(name, extra=30), max_live=4, seed=7)
    out_dir = str(tmp_path / "out")
    process = subprocess.Popen(
        [sys.executable, os.path.join(ROOT, "bin", "trace_run"), "--model", folder, "--dtype", dtype,
         "--out", out_dir, "--max-tokens", str(traces.live_token_need(steps, 64))],
        stdin=subprocess.PIPE, stdout=subprocess.PIPE, text=True, cwd=ROOT)
    try:
        positions = {}
        for step in steps:
            process.stdin.write(json.dumps(step) + "\n")
            process.stdin.flush()
            assert process.stdout.readline().strip() == f"done {step['step']}"
            rows = traces.labels(step, positions)
            data = np.fromfile(os.path.join(out_dir, f"{step['step']}.f32"), dtype="<f4")
            check_rows(data.reshape(len(rows), -1), expected, rows, f"step {step['step']}")
        process.stdin.close()
        assert process.wait(timeout=120) == 0
    finally:
        if process.poll() is None:
            process.kill()


def test_generation_from_the_command_line(models):
    """``bin/helix_generate`` chooses the model by ``config.json`` and prints the plain
    implementation's greedy tokens."""
    folder, plain = models("odd", "float32")
    prompt = random_tokens(CONFIGS["odd"]["vocab"], 19, seed=3)
    done = subprocess.run(
        [sys.executable, os.path.join(ROOT, "bin", "helix_generate"), "--model", folder,
         "--dtype", "float32", "--max-new-tokens", "12", *[str(token) for token in prompt]],
        capture_output=True, text=True, cwd=ROOT, timeout=300)
    assert done.returncode == 0, done.stderr
    lines = done.stdout.strip().splitlines()
    generated = [int(token) for token in lines[0].split(":")[1].split()]
    assert len(generated) == 12 and lines[1] == "stop_reason: max_new_tokens"
    tokens = list(prompt) + generated
    logits = plain.forward(tokens)
    for place in range(len(prompt), len(tokens)):
        assert logits[place - 1][tokens[place]] >= logits[place - 1].max() - 1e-3
