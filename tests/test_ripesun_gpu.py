"""Ripesun models on the GPU against the plain implementation (``oracle.ripesun_model``, float64).

In fp32 the two agree to fp32 rounding, so every mechanism, cache and state path and schedule is pinned sharply there;
the bf16 runs pin the serving kernels within bf16 rounding.  Errors are in units of the spread of the logits.
"""

from __future__ import annotations

import json
import subprocess
import sys
from pathlib import Path

import numpy as np
import pytest
import torch

from mini_inference_engine_b200.engine.checkpoint import save_safetensors
from mini_inference_engine_b200.engine.model_runner.continuous import ContinuousBatcher
from mini_inference_engine_b200.engine.model_runner.replay import TraceEntry, TraceSession
from mini_inference_engine_b200.engine.model_runner.ripesun import RipesunRunner
from mini_inference_engine_b200.engine.registry import load_runner
from oracle import ripesun_model as plain
from ripesun_models import CONFIGS, logit_errors, make_tokens, make_weights, oracle_weights, runner_weights

pytestmark = pytest.mark.gpu

ROOT = Path(__file__).resolve().parents[1]
# Row errors: largest, the bound that one row in fifty (or one) may pass, median.  Rounding the operands and results of
# every product to bf16 in the plain implementation gives single rows of up to 0.3 (a sublayer's result that nearly
# cancels is normed back to full size), with medians around 0.006.
LIMIT = {torch.float32: (5e-5, 5e-5, 1e-5), torch.bfloat16: (0.5, 0.1, 0.03)}
BOTH = pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16], ids=["fp32", "bf16"])
MODELS = pytest.mark.parametrize("name", list(CONFIGS))


def assert_close(got, want, dtype):
    errors = logit_errors(got, want)
    worst, over, median = float(errors.max()), int((errors > LIMIT[dtype][1]).sum()), float(errors.median())
    assert worst <= LIMIT[dtype][0] and over <= max(1, len(errors) // 50) and median <= LIMIT[dtype][2], (worst, over, median)


class Model:
    """A small model, its runner and the oracle's logits of whole sequences."""

    _cache: dict = {}

    def __init__(self, name, dtype, device, *, seed=0, page=16, num_pages=64, max_context=512, attention="auto", **kw):
        self.config, self.dtype = CONFIGS[name], dtype
        self.name, self.seed = name, seed
        tensors = make_weights(self.config, seed)
        self.weights = oracle_weights(tensors)
        self.runner = RipesunRunner(runner_weights(self.config, tensors, device, dtype, page), num_pages=num_pages,
                                    max_batch=kw.pop("max_batch", 8), max_context=max_context, attention=attention,
                                    **kw)
        self.session = TraceSession(self.runner)

    def expected(self, tokens):
        key = (self.name, self.seed, tuple(tokens))
        if key not in self._cache:
            self._cache[key] = plain.forward(self.config, self.weights, list(tokens))[0]
        return self._cache[key]

    def tokens(self, count, seed=0):
        return make_tokens(self.config, count, seed)

    def feed(self, rid, tokens, cuts):
        """Logits of every token of one request, fed in pieces of the given sizes."""

        out, at = [], 0
        for count in cuts:
            out.append(self.session.step([TraceEntry(rid, tokens[at:at + count], list(range(count)))]))
            at += count
        assert at == len(tokens)
        return torch.cat(out)

    def check(self, got, tokens):
        assert_close(got, self.expected(tokens), self.dtype)


def pieces(total, sizes):
    """Cut ``total`` into the given sizes, repeated."""

    out = []
    while sum(out) < total:
        out.append(min(sizes[len(out) % len(sizes)], total - sum(out)))
    return out


@BOTH
@MODELS
def test_whole_prompts(name, dtype, device):
    model = Model(name, dtype, device)
    for index, count in enumerate((1, 2, 6, 48, 150, 330)):
        tokens = model.tokens(count, index)
        model.check(model.feed(index, tokens, [count]), tokens)


@MODELS
def test_residual_stream_after_every_layer(name, device):
    """fp32: the residual rows themselves, layer by layer (truncated models share their leading layers)."""

    config = CONFIGS[name]
    tensors, tokens = make_weights(config), make_tokens(config, 70, 9)
    streams = plain.forward(config, oracle_weights(tensors), tokens)[1]
    for depth in range(1, len(config["layers"]) + 1):
        cut = {**config, "layers": config["layers"][:depth]}
        mine = {**tensors, "side.embed": tensors["side.embed"][:, :depth * config["token_side"]["dim"]].contiguous()}
        runner = RipesunRunner(runner_weights(cut, mine, device, torch.float32), num_pages=8, max_batch=1,
                               max_context=128)
        positions = torch.arange(70, dtype=torch.int32, device=device)
        x32 = runner._layers(torch.tensor(tokens, device=device), positions, torch.zeros_like(positions),
                             torch.arange(8, dtype=torch.int32, device=device).unsqueeze(0),
                             state_slots=torch.zeros(1, dtype=torch.int32, device=device), decode_rows=0,
                             decode_lengths=None, cu_seqlens=torch.tensor([0, 70], dtype=torch.int32, device=device),
                             kv_lens=torch.tensor([70], dtype=torch.int32, device=device), max_query_len=70)
        runner.check_status()
        difference = (x32.cpu().double() - streams[depth - 1]).abs().max()
        assert float(difference) <= 1e-4, (depth, float(difference))


@BOTH
@MODELS
def test_token_by_token_from_the_first(name, dtype, device):
    """Decoding from the first token on crosses every window and page border with cached rows, and starts every
    recurrence from nothing."""

    model = Model(name, dtype, device)
    tokens = model.tokens(75, 1)
    model.check(model.feed("a", tokens, [1] * 75), tokens)


@BOTH
@MODELS
@pytest.mark.parametrize("sizes", [(2,), (3, 1, 2), (16,), (17, 15), (64, 1, 1, 5)], ids=str)
def test_portions(name, dtype, sizes, device):
    model = Model(name, dtype, device)
    tokens = model.tokens(110, 2)
    model.check(model.feed("a", tokens, pieces(110, sizes)), tokens)


@BOTH
@MODELS
def test_long_decoding_after_a_prompt(name, dtype, device):
    model = Model(name, dtype, device, max_context=320, num_pages=20)
    tokens = model.tokens(300, 3)
    model.check(model.feed("a", tokens, [41] + [1] * 259), tokens)


@BOTH
@MODELS
def test_unequal_requests_in_one_batch(name, dtype, device):
    """Requests of different lengths advance together, by single tokens, pairs and long portions in the same
    step; each gets the logits it gets alone."""

    model = Model(name, dtype, device)
    lengths = {"a": 120, "b": 17, "c": 64, "d": 3, "e": 90}
    tokens = {rid: model.tokens(n, 10 + i) for i, (rid, n) in enumerate(lengths.items())}
    steps = {"a": [50, 1, 1, 2, 33, 33], "b": [1] * 17, "c": [16, 16, 1, 31], "d": [1, 2],
             "e": [3, 1, 1, 1, 40, 1, 43]}
    logits, at, turn = {rid: [] for rid in lengths}, dict.fromkeys(lengths, 0), 0
    while any(at[rid] < lengths[rid] for rid in lengths):
        entries = []
        for rid in lengths:
            if turn < len(steps[rid]):
                count = steps[rid][turn]
                entries.append(TraceEntry(rid, tokens[rid][at[rid]:at[rid] + count], list(range(count))))
                at[rid] += count
        rows = model.session.step(entries)
        for entry in entries:
            logits[entry.rid].append(rows[:len(entry.tokens)])
            rows = rows[len(entry.tokens):]
        turn += 1
    for rid in lengths:
        model.check(torch.cat(logits[rid]), tokens[rid])


@BOTH
@MODELS
def test_freed_pages_and_slots_are_used_again(name, dtype, device):
    """A pool that holds two requests at a time serves seven: later ones run on pages and state slots others have
    left their rows and states in."""

    model = Model(name, dtype, device, num_pages=12, max_context=96, max_batch=2)
    model.runner.state.rows.fill_(float("nan"))
    live = []
    for index in range(7):
        count = (80, 33, 95, 2, 64, 17, 90)[index]
        tokens = model.tokens(count, 20 + index)
        model.check(model.feed(index, tokens, [count - 2, 1, 1] if count > 4 else [1] * count), tokens)
        live.append(index)
        if len(live) == 2:
            model.session.end([live.pop(0 if index % 2 else 1)])
    model.session.end(live)
    assert model.session.pool.free_pages == 12 and model.session.slots.free_slots == 2 and not model.session.sequences


def stretched(config, tensors, layer, factor):
    """The weights with one latent layer's queries scaled, so that its attention is close to picking one key."""

    return {**tensors, f"l{layer}.mix.dq.norm": (tensors[f"l{layer}.mix.dq.norm"].float() * factor).to(torch.bfloat16)}


@pytest.mark.parametrize("layer", [1, 3, 4, 5])
def test_single_keys_at_the_window_edge(layer, device):
    """fp32 with one layer's scores stretched until single keys dominate: a key wrongly inside or outside the window
    then changes many logits outright, in prompts, portions and decoding."""

    config = CONFIGS["mixed"]
    tensors = stretched(config, make_weights(config, 5), layer, 4.0)
    tokens = make_tokens(config, 130, 6)
    want = plain.forward(config, oracle_weights(tensors), tokens)[0]
    for change in (-1, 1):
        near = json.loads(json.dumps(config))
        near["layers"][layer]["mixer"]["mask"]["size"] += change
        moved = logit_errors(plain.forward(near, oracle_weights(tensors), tokens)[0], want)
        assert float(moved.max()) > 0.1
    runner = RipesunRunner(runner_weights(config, tensors, device, torch.float32), num_pages=40, max_batch=4, max_context=256)
    for cuts in ([130], [1] * 130, [2] * 65, [19, 1, 20, 21, 7, 8, 54]):
        session, got, at = TraceSession(runner), [], 0
        for count in cuts:
            got.append(session.step([TraceEntry("a", tokens[at:at + count], list(range(count)))]))
            at += count
        errors = logit_errors(torch.cat(got), want)
        assert float(errors.max()) <= 2e-4, float(errors.max())


@BOTH
def test_other_page_sizes_and_the_row_kernel(dtype, device):
    for page, attention in ((32, "auto"), (5, "auto"), (16, "rows")):
        model = Model("mixed", dtype, device, page=page, attention=attention)
        bf16 = dtype == torch.bfloat16 and attention == "auto"
        streams = [s[1:] for s in model.runner._streams if s is not None]
        assert all(s == (bf16 and page % 16 == 0, bf16) for s in streams)
        tokens = model.tokens(100, 4)
        model.check(model.feed("a", tokens, [30, 1, 1, 2, 1, 40] + [1] * 25), tokens)


# Seeds for which the oracle's top-2 logit gap is decisive at every step (re-checked below).
GREEDY_SEEDS = {"mixed": 45, "wide": 32, "deep_latent": 263, "odd": 78}
GREEDY_PLAN = [(37, 4), (5, 6), (50, 3), (18, 5)]
MARGIN = {torch.float32: 5e-4, torch.bfloat16: 0.09}


def greedy_requests(model):
    out = []
    for index, (count, new) in enumerate(GREEDY_PLAN):
        prompt = model.tokens(count, 100 * GREEDY_SEEDS[model.name] + index)
        tokens, margin = plain.greedy(model.config, model.weights, prompt, new)
        assert margin >= MARGIN[model.dtype], f"the oracle is not decisive: {margin:.4f}"
        out.append((index, prompt, new, tokens))
    return out


@BOTH
@MODELS
@pytest.mark.parametrize("mixed", [False, True], ids=["graphs", "mixed"])
def test_greedy_generation_through_the_scheduler(name, dtype, mixed, device):
    """Bucketed decode graphs with padding rows, prompts in chunks, requests that arrive late and finish at
    different times, captured mixed steps."""

    model = Model(name, dtype, device, seed=GREEDY_SEEDS[name], num_pages=30, chunk_buckets=(32,), max_batch=4)
    requests = greedy_requests(model)
    batcher = ContinuousBatcher(model.runner, max_prefill_tokens=32, mixed=mixed)
    batcher.submit(*requests[0][:3])
    batcher.submit(*requests[1][:3])
    for _ in range(3):
        batcher.step()
    for request in requests[2:]:
        batcher.submit(*request[:3])
    results = batcher.run()
    assert {rid: results[rid] for rid, *_ in requests} == {rid: tokens for rid, _, _, tokens in requests}
    assert batcher.pool.free_pages == 30 and batcher.slots.free_slots == 4
    assert any(key[0] == ("mixed" if mixed else "decode") for key in model.runner._graphs)
    model.runner.release_graphs()


@BOTH
@MODELS
def test_greedy_generation_of_requests_that_arrive_together(name, dtype, device):
    model = Model(name, dtype, device, seed=GREEDY_SEEDS[name], max_batch=6)
    requests = greedy_requests(model)
    new = min(n for _, _, n, _ in requests)
    for use_graph in (True, False):
        got = model.runner.generate([prompt for _, prompt, _, _ in requests], new, use_graph=use_graph)
        assert got == [tokens[:new] for *_, tokens in requests]
    model.runner.release_graphs()


@BOTH
@MODELS
def test_shared_prefix_pages_and_states(name, dtype, device):
    """A request that borrows the pages of another's prompt starts in the middle of its sequence: it needs cached rows
    it never wrote and the recurrent state at the border.  Without spare slots nothing is shared."""

    model = Model(name, dtype, device, seed=GREEDY_SEEDS[name], max_batch=4, chunk_buckets=(32,), state_slots=6)
    requests = greedy_requests(model)
    (_, prompt, new, tokens), (_, other, _, _) = requests[0], requests[2]
    batcher = ContinuousBatcher(model.runner, prefix_cache=True)
    for rid, ids in (("first", prompt), ("other", other), ("second", prompt)):
        batcher.submit(rid, ids, new)
        batcher.run()
    results = batcher.results
    assert batcher.prefix_hits == 32 and results["first"] == results["second"] == tokens
    assert len(batcher._prefix_states) == 2 and batcher.slots.free_slots == 4
    batcher.submit("third", other[:48] + prompt[:9], 1)
    batcher.run()
    assert batcher.prefix_hits == 80 and len(batcher._prefix_states) == 2
    for rid, ids in (("fourth", prompt[::-1]), ("fifth", prompt)):  # the fourth's state pushes out the first's
        batcher.submit(rid, ids, 1)
        batcher.run()
    assert batcher.prefix_hits == 80 and len(batcher._prefix_states) == 2
    batcher.drop_prefix_cache()
    assert batcher.slots.free_slots == 6 and batcher.pool.free_pages == 64
    model.runner.release_graphs()
    model = Model(name, dtype, device, seed=GREEDY_SEEDS[name], max_batch=4, chunk_buckets=(32,))
    batcher = ContinuousBatcher(model.runner, prefix_cache=True)
    for rid in ("first", "second"):
        batcher.submit(rid, prompt, new)
        batcher.run()
    assert batcher.prefix_hits == 0 and batcher.results["first"] == batcher.results["second"] == tokens
    model.runner.release_graphs()


@pytest.fixture()
def model_folder(tmp_path):
    config = CONFIGS["mixed"]
    (tmp_path / "config.json").write_text(json.dumps(config))
    save_safetensors(tmp_path / "model.safetensors", make_weights(config, GREEDY_SEEDS["mixed"]))
    return tmp_path


@BOTH
def test_folder_loads_through_the_registry(model_folder, dtype, device):
    runner = load_runner(model_folder, dtype=dtype, num_pages=20, max_batch=2, max_context=128, state_slots=3)
    assert runner.num_slots == 3
    tokens = make_tokens(CONFIGS["mixed"], 60, 6)
    got = TraceSession(runner).step([TraceEntry("a", tokens, list(range(60)))])
    want = plain.forward(CONFIGS["mixed"], oracle_weights(make_weights(CONFIGS["mixed"], GREEDY_SEEDS["mixed"])), tokens)[0]
    assert_close(got, want, dtype)


def test_command_line_replays_and_generates(model_folder, device):
    model = Model("mixed", torch.float32, device, seed=GREEDY_SEEDS["mixed"])
    tokens = model.tokens(40, 8)
    steps = [{"step": 3, "entries": [{"id": "q", "tokens": tokens[:30], "want": [29, 0]}], "end": []},
             {"step": 4, "entries": [{"id": "q", "tokens": tokens[30:31], "want": []}], "end": []},
             {"step": 5, "entries": [{"id": "q", "tokens": tokens[31:], "want": [8]}], "end": ["q"]}]
    done = subprocess.run([str(ROOT / "bin" / "trace_run"), "--model", str(model_folder), "--dtype", "float32", "--out",
                           str(model_folder), "--max-tokens", "40"], input="\n".join(map(json.dumps, steps)) + "\n",
                          capture_output=True, text=True, timeout=300)
    assert done.returncode == 0, done.stderr[-2000:]
    assert [line for line in done.stdout.splitlines() if line.startswith("done")] == ["done 3", "done 4", "done 5"]
    assert not (model_folder / "4.f32").exists()
    want = model.expected(tokens)
    for step, places in ((3, [29, 0]), (5, [39])):
        got = np.fromfile(model_folder / f"{step}.f32", dtype="<f4").reshape(len(places), -1)
        assert_close(torch.from_numpy(got), want[places], torch.float32)
    requests = greedy_requests(model)
    new = min(n for _, _, n, _ in requests)
    command = [sys.executable, "-m", "mini_inference_engine_b200", "generate", "--model", str(model_folder), "--dtype",
               "float32", "--max-new-tokens", str(new), "--mixed", "--prefix-cache"]
    for _, prompt, _, _ in requests:
        command += ["--prompt", ",".join(map(str, prompt))]
    done = subprocess.run(command, cwd=ROOT, capture_output=True, text=True, timeout=300)
    assert done.returncode == 0, done.stderr[-2000:]
    lines = [json.loads(line) for line in done.stdout.splitlines() if line.startswith("{")]
    assert [line["tokens"] for line in lines] == [tokens[:new] for *_, tokens in requests]
