"""Tidelorn models on the GPU against the plain implementation (``oracle.tidelorn_model``, float64).

In fp32 the two agree to fp32 rounding, so every mechanism, cache path and schedule is pinned sharply there; the
bf16 runs pin the serving kernels within bf16 rounding.  Errors are in units of the spread of the logits.
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
from mini_inference_engine_b200.engine.model_runner.tidelorn import TidelornRunner
from mini_inference_engine_b200.engine.registry import load_runner
from oracle import tidelorn_model as plain
from tidelorn_models import CONFIGS, logit_errors, make_tokens, make_weights, oracle_weights, runner_weights

pytestmark = pytest.mark.gpu

ROOT = Path(__file__).resolve().parents[1]
# Largest and median row error.  Rounding activations to bf16 where the kernels do, in the plain implementation,
# gives up to 0.06 and 0.02 on these models.
LIMIT = {torch.float32: (3e-5, 1e-5), torch.bfloat16: (0.1, 0.03)}
BOTH = pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16], ids=["fp32", "bf16"])
MODELS = pytest.mark.parametrize("name", list(CONFIGS))


def assert_close(got, want, dtype):
    errors = logit_errors(got, want)
    worst, median = float(errors.max()), float(errors.median())
    assert worst <= LIMIT[dtype][0] and median <= LIMIT[dtype][1], (worst, median)


class Model:
    """A small model, its runner and the oracle's logits of whole sequences."""

    _cache: dict = {}

    def __init__(self, name, dtype, device, *, seed=0, page=16, num_pages=64, max_context=512, attention="auto", **kw):
        self.config, self.dtype = CONFIGS[name], dtype
        self.name, self.seed = name, seed
        tensors = make_weights(self.config, seed)
        self.weights = oracle_weights(tensors)
        self.runner = TidelornRunner(runner_weights(self.config, tensors, device, dtype, page), num_pages=num_pages,
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
    for index, count in enumerate((1, 2, 6, 48, 150)):
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
        runner = TidelornRunner(runner_weights(cut, tensors, device, torch.float32), num_pages=8, max_batch=1,
                                max_context=128)
        positions = torch.arange(70, dtype=torch.int32, device=device)
        x32 = runner._layers(torch.tensor(tokens, device=device), positions, torch.zeros_like(positions),
                             torch.arange(8, dtype=torch.int32, device=device).unsqueeze(0), decode_rows=0,
                             decode_lengths=None, cu_seqlens=torch.tensor([0, 70], dtype=torch.int32, device=device),
                             kv_lens=torch.tensor([70], dtype=torch.int32, device=device), max_query_len=70)
        runner.check_status()
        difference = (x32.cpu().double() - streams[depth - 1]).abs().max()
        assert float(difference) <= 5e-5, (depth, float(difference))


@BOTH
@MODELS
def test_token_by_token_from_the_first(name, dtype, device):
    """Decoding from the first token on crosses every window and page border with cached keys."""

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
def test_freed_pages_are_used_again(name, dtype, device):
    """A pool that holds two requests at a time serves seven: later ones run on pages others have left their keys,
    values and token ids in."""

    model = Model(name, dtype, device, num_pages=12, max_context=96)
    live = []
    for index in range(7):
        count = (80, 33, 95, 2, 64, 17, 90)[index]
        tokens = model.tokens(count, 20 + index)
        model.check(model.feed(index, tokens, [count - 2, 1, 1] if count > 4 else [1] * count), tokens)
        live.append(index)
        if len(live) == 2:
            model.session.end([live.pop(0 if index % 2 else 1)])
    model.session.end(live)
    assert model.session.pool.free_pages == 12 and not model.session.sequences


@BOTH
def test_other_page_sizes_and_the_row_kernel(dtype, device):
    for page, attention in ((32, "auto"), (5, "auto"), (16, "rows")):
        model = Model("grouped", dtype, device, page=page, attention=attention)
        streams = [(decode, chunks) for _, decode, chunks in model.runner._attention]
        assert all(s == ((dtype == torch.bfloat16 and page % 16 == 0 and attention == "auto",) * 2) for s in streams)
        tokens = model.tokens(100, 4)
        model.check(model.feed("a", tokens, [30, 1, 1, 2, 1, 40] + [1] * 25), tokens)


# Seeds for which the oracle's top-2 logit gap is decisive at every step (re-checked below).
GREEDY_SEEDS = {"grouped": 292, "single_kv": 36, "separate": 37, "odd": 242}
GREEDY_PLAN = [(37, 6), (5, 9), (70, 4), (18, 12)]
MARGIN = {torch.float32: 5e-4, torch.bfloat16: 0.06}


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
    assert batcher.pool.free_pages == 30
    assert any(key[0] == ("mixed" if mixed else "decode") for key in model.runner._graphs)
    model.runner.release_graphs()


@BOTH
@MODELS
def test_greedy_generation_of_requests_that_arrive_together(name, dtype, device):
    model = Model(name, dtype, device, seed=GREEDY_SEEDS[name], max_batch=4)
    requests = greedy_requests(model)
    new = min(n for _, _, n, _ in requests)
    for use_graph in (True, False):
        got = model.runner.generate([prompt for _, prompt, _, _ in requests], new, use_graph=use_graph)
        assert got == [tokens[:new] for *_, tokens in requests]
    model.runner.release_graphs()


@BOTH
@MODELS
def test_shared_prefix_pages(name, dtype, device):
    """A request that borrows the pages of another's prompt starts in the middle of its sequence: its first own
    token needs the previous token, keys and values of pages it never wrote."""

    model = Model(name, dtype, device, seed=GREEDY_SEEDS[name], max_batch=4, chunk_buckets=(32,))
    requests = greedy_requests(model)
    rid, prompt, new, tokens = requests[0]
    batcher = ContinuousBatcher(model.runner, prefix_cache=True)
    batcher.submit("first", prompt, new)
    batcher.run()
    batcher.submit("second", prompt, new)
    results = batcher.run()
    assert batcher.prefix_hits == 32 and results["first"] == results["second"] == tokens
    model.runner.release_graphs()


@pytest.fixture()
def model_folder(tmp_path):
    config = CONFIGS["single_kv"]
    (tmp_path / "config.json").write_text(json.dumps(config))
    save_safetensors(tmp_path / "model.safetensors", make_weights(config, GREEDY_SEEDS["single_kv"]))
    return tmp_path


@BOTH
def test_folder_loads_through_the_registry(model_folder, dtype, device):
    runner = load_runner(model_folder, dtype=dtype, num_pages=20, max_batch=2, max_context=128)
    tokens = make_tokens(CONFIGS["single_kv"], 60, 6)
    got = TraceSession(runner).step([TraceEntry("a", tokens, list(range(60)))])
    want = plain.forward(CONFIGS["single_kv"],
                         oracle_weights(make_weights(CONFIGS["single_kv"], GREEDY_SEEDS["single_kv"])), tokens)[0]
    assert_close(got, want, dtype)


def test_command_line_replays_and_generates(model_folder, device):
    model = Model("single_kv", torch.float32, device, seed=GREEDY_SEEDS["single_kv"])
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
    command = [sys.executable, "-m", "mini_inference_engine_b200", "generate", "--model", str(model_folder), "--dtype",
               "float32", "--max-new-tokens", "4", "--mixed"]
    for _, prompt, _, _ in requests:
        command += ["--prompt", ",".join(map(str, prompt))]
    done = subprocess.run(command, cwd=ROOT, capture_output=True, text=True, timeout=300)
    assert done.returncode == 0, done.stderr[-2000:]
    lines = [json.loads(line) for line in done.stdout.splitlines() if line.startswith("{")]
    assert [line["tokens"] for line in lines] == [tokens[:4] for *_, tokens in requests]


def test_the_registry_serves_the_other_design_too(tmp_path, device):
    """A Qwen3 configuration through the same registry, batcher and runner interface (seeded weights): scheduled
    generation gives the tokens of its own ``generate``."""

    (tmp_path / "config.json").write_text(json.dumps({
        "architectures": ["Qwen3ForCausalLM"], "num_hidden_layers": 2, "hidden_size": 512, "num_attention_heads": 4,
        "num_key_value_heads": 2, "head_dim": 128, "intermediate_size": 1024, "vocab_size": 2048,
        "rms_norm_eps": 1e-6, "rope_theta": 5e6}))
    runner = load_runner(tmp_path, random_seed=36, num_pages=32, max_batch=2, max_context=128)
    prompt = torch.randint(0, 2048, (37,), generator=torch.Generator().manual_seed(1)).tolist()
    batcher = ContinuousBatcher(runner)
    batcher.submit("a", prompt, 3)
    assert batcher.run()["a"] == runner.generate([prompt], 3)[0]
    runner.release_graphs()
