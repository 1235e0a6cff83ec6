"""Host side of the Tidelorn design, and what the plain implementation says about the test models, on the CPU."""

from __future__ import annotations

import copy
import io
import json
import math

import pytest
import torch

from mini_inference_engine_b200 import cli
from mini_inference_engine_b200.engine import registry
from mini_inference_engine_b200.engine.checkpoint import Checkpoint, CheckpointError, load_config, save_safetensors
from mini_inference_engine_b200.engine.model_runner.continuous import PagePoolExhausted
from mini_inference_engine_b200.engine.model_runner.replay import TraceEntry, TraceSession
from mini_inference_engine_b200.engine.model_runner.tidelorn import TidelornShape, TidelornWeights
from oracle import tidelorn_model as plain
from tidelorn_models import CONFIGS, logit_error, make_tokens, make_weights, oracle_weights, runner_weights

CPU = torch.device("cpu")


# -- configuration, registry, checkpoints -----------------------------------------------------------

def test_configuration_decides_sizes_and_branches():
    shape = TidelornShape.from_config(CONFIGS["grouped"])
    window, full, bare, last = shape.layers
    assert (window.window, window.temperature, window.bias, window.learned_sink, window.v_mix) == (5, None, False, False,
                                                                                                  False)
    assert (full.window, full.temperature, full.bias, full.learned_sink) == (None, (0.4, 7), True, True)
    assert bare.ff is None and last.limit == 0.5 and shape.first_v_mix == 1 and shape.alpha == 1.7
    names = shape.tensor_shapes()
    assert names["l1.mix.sink"] == (6,) and names["l1.mix.vmix"] == () and names["bigram"] == (62, 64)
    assert "l0.mix.q.b" not in names and "l0.mix.vmix" not in names and "l2.norm2" not in names
    assert TidelornShape.from_config(CONFIGS["separate"]).first_v_mix is None


@pytest.mark.parametrize("change, message", [
    (lambda c: c["layers"][0].update(type="recurrent"), "unknown type"),
    (lambda c: c["layers"][1]["mlp"].update(kind="experts"), "unknown feed-forward"),
    (lambda c: c["layers"][1]["mixer"].update(kv_heads=4), "multiple"),
    (lambda c: c["layers"][0]["mixer"]["mask"].update(size=0), "window"),
    (lambda c: c["layers"][2]["mixer"].update(vdim=8), "agree"),
])
def test_unusable_configurations_are_refused(change, message):
    config = copy.deepcopy(CONFIGS["grouped"])
    change(config)
    with pytest.raises(ValueError, match=message):
        TidelornShape.from_config(config)


def test_registry_chooses_the_design_by_config():
    assert registry.design_for({"architecture": "Tidelorn"}).name == "Tidelorn"
    qwen = registry.design_for({"architectures": ["Qwen3ForCausalLM"]})
    shape = qwen.shape({"num_hidden_layers": 2, "hidden_size": 512, "num_attention_heads": 4,
                        "num_key_value_heads": 2, "intermediate_size": 1024, "vocab_size": 2048, "rope_theta": 1e4})
    assert (shape.layers, shape.hidden, shape.head_dim, shape.rope_theta) == (2, 512, 128, 1e4)
    assert torch.float32 not in qwen.dtypes
    with pytest.raises(CheckpointError, match="no registered design"):
        registry.design_for({"architecture": "Unheard"})
    with pytest.raises(ValueError, match="registered already"):
        registry.register(qwen)


def test_checkpoint_round_trip_and_shape_checks(tmp_path):
    config, tensors = CONFIGS["odd"], make_weights(CONFIGS["odd"])
    (tmp_path / "config.json").write_text(json.dumps(config))
    save_safetensors(tmp_path / "model.safetensors", {**tensors, "extra": torch.arange(6, dtype=torch.int32)})
    assert load_config(tmp_path) == config
    checkpoint = Checkpoint(tmp_path)
    weights = TidelornWeights(TidelornShape.from_config(config), checkpoint.take, CPU, torch.float32)
    assert checkpoint.unused() == ["extra"]
    layer, shape = weights.layers[0], TidelornShape.from_config(config).layers[0]
    parts = layer.qkv.split([shape.heads * shape.dim, shape.kv_heads * shape.dim, shape.kv_heads * shape.vdim])
    for part, name in zip(parts, "qkv"):
        assert torch.equal(part, tensors[f"l0.mix.{name}"].float())
    assert layer.lam == 0.0 and weights.layers[1].lam == float(tensors["l1.mix.vmix"])  # the first one is not blended
    assert torch.equal(layer.sinks, tensors["l0.mix.sink"].float()) and not weights.layers[1].sinks.any()
    assert torch.equal(checkpoint.take("extra"), torch.arange(6, dtype=torch.int32))
    with pytest.raises(CheckpointError, match="no tensor"):
        checkpoint.take("missing")
    with pytest.raises(CheckpointError, match="expected"):
        checkpoint.take("embed", (1, 2))
    (tmp_path / "model.safetensors").write_bytes(b"\xff" * 16)
    with pytest.raises(CheckpointError, match="shorter"):
        Checkpoint(tmp_path)
    with pytest.raises(CheckpointError, match="no \\*.safetensors"):
        Checkpoint(tmp_path / "nowhere")


def test_random_weights_have_the_checkpoint_form():
    shape = TidelornShape.from_config(CONFIGS["grouped"])
    a, b = (TidelornWeights.random(shape, CPU, seed=3) for _ in range(2))
    assert torch.equal(a.layers[1].qkv, b.layers[1].qkv) and a.layers[1].qkv.shape == (shape.layers[1].qkv_rows, 64)
    assert a.weight_bytes() == 2 * (a.head.numel() + sum(
        t.numel() for w in a.layers for t in (w.qkv, w.o, w.gate_up, w.down) if t is not None))


def test_command_line_refuses_a_number_format_the_design_lacks(tmp_path, monkeypatch, capsys):
    (tmp_path / "config.json").write_text(json.dumps({
        "architectures": ["Qwen3ForCausalLM"], "num_hidden_layers": 1, "hidden_size": 512, "num_attention_heads": 4,
        "num_key_value_heads": 2, "intermediate_size": 1024, "vocab_size": 256}))
    monkeypatch.setattr("sys.stdin", io.StringIO(""))
    arguments = ["trace", "--model", str(tmp_path), "--dtype", "float32", "--out", str(tmp_path), "--max-tokens", "64"]
    assert cli.main(arguments) == cli.EXIT_UNSUPPORTED_DTYPE
    assert "does not run in" in capsys.readouterr().err
    assert cli.main(["models"]) == 0 and "Tidelorn bfloat16 float32" in capsys.readouterr().out


# -- trace sessions ---------------------------------------------------------------------------------

class _Recorder:
    """A runner that returns a row per wanted place: [token, position, table row's first page]."""

    class shape:
        page = 4

    device, num_pages, max_batch, max_context, table_width = CPU, 6, 2, 20, 5

    def decode_forward(self, ids, lengths, tables, return_logits=False):
        return None, torch.stack([ids.float(), lengths.float() - 1, tables[:, 0].float()], dim=1)

    def mixed_forward(self, ids, tok2seq, positions, tables, *, decode_rows, decode_lengths, cu_seqlens, kv_lens,
                      max_query_len, logit_rows, return_logits=False):
        assert int(cu_seqlens[-1]) == ids.shape[0] - decode_rows
        rows = torch.stack([ids.float(), positions.float(), tables[tok2seq.long(), 0].float()], dim=1)
        return None, rows[logit_rows]

    def check_status(self):
        pass


def test_trace_session_orders_rows_and_accounts_for_pages():
    session = TraceSession(_Recorder())
    assert session.step([TraceEntry("a", [11, 12, 13], [])]) is None
    # a decode row, a chunk and a second decode row in one step: results follow the entries, not the stream
    session.step([TraceEntry("c", [31], [0])])
    got = session.step([TraceEntry("b", [21, 22], [1, 0]), TraceEntry("a", [14], [0]), TraceEntry("c", [32], [0])])
    assert [row[:2] for row in got.tolist()] == [[22.0, 1.0], [21.0, 0.0], [14.0, 3.0], [32.0, 1.0]]
    assert len({page for _, _, page in got[1:].tolist()}) == 3 and session.pool.free_pages == 3
    got = session.step([TraceEntry("a", [15], [0]), TraceEntry("c", [33], [])])
    assert got.tolist()[0][:2] == [15.0, 4.0] and session.pool.free_pages == 2
    session.end(["a", "nobody"])
    assert session.pool.free_pages == 4
    with pytest.raises(ValueError, match="outside"):
        session.step([TraceEntry("b", [1], [1])])
    with pytest.raises(ValueError, match="once per step"):
        session.step([TraceEntry("b", [1], []), TraceEntry("b", [1], [])])
    with pytest.raises(ValueError, match="max_context"):
        session.step([TraceEntry("b", [1] * 30, [])])
    with pytest.raises(PagePoolExhausted):
        session.step([TraceEntry("d", [1] * 20, [])])


# -- the plain implementation: known values, and whether the test models would show a fault -----------

def test_mechanisms_have_their_known_values():
    assert plain.bigram_rows([3, 5, 2], 7, 2, 3) == [7, (6 + 15) % 7, (10 + 6) % 7]
    assert [plain.visible(9, k, 3) for k in (5, 6, 7, 9, 10)] == [False, False, True, True, False]
    positions = torch.tensor([0, 2, 3, 6, 7])
    assert plain.query_temperature(positions, 1.0, 4).tolist() == pytest.approx(
        [1.0, 1.0, 1 + math.log(2), 1 + math.log(2), 1 + math.log(3)])
    row = plain.sinusoid(torch.tensor([2]), 3)[0].tolist()
    assert row == pytest.approx([math.sin(2), math.cos(2), math.sin(2 * 10000 ** (-2 / 3))])
    weights = plain.sink_softmax(torch.tensor([[0.0, math.log(2), -math.inf]]), torch.tensor(math.log(5)))
    assert weights.tolist()[0] == pytest.approx([1 / 8, 2 / 8, 0.0])
    gate = plain.clamped_gate(torch.tensor([9.0, -9.0]), torch.tensor([-9.0, 9.0]), 2.0)
    assert gate.tolist() == pytest.approx([2 / (1 + math.exp(-3.404)) * -1.0, -9 / (1 + math.exp(15.318)) * 3.0])
    x = torch.tensor([[3.0, 4.0]])
    assert plain.rms_norm(x, torch.tensor([0.0, 1.0]), 0.5)[0].tolist() == pytest.approx(
        [3 / math.sqrt(13), 8 / math.sqrt(13)])


def _mistake(name):
    """A function that puts one mistake into a copy of (config, weights), or replaces a mechanism."""

    def sizes(key, delta):
        def change(config, weights, patch):
            for layer in config["layers"]:
                if key in layer["mixer"]:
                    layer["mixer"][key]["size"] += delta
        return change

    def scaled(suffix, factor):
        def change(config, weights, patch):
            for key in weights:
                if key.endswith(suffix):
                    weights[key] = weights[key] * factor
        return change

    def config_value(path, value):
        def change(config, weights, patch):
            for layer in config["layers"]:
                if layer["type"] == "attention":
                    layer["mixer"][path[0]][path[1]] = value(layer["mixer"][path[0]][path[1]])
        return change

    def replaced(function, make):
        return lambda config, weights, patch: patch.setattr(plain, function, make(getattr(plain, function)))

    return {
        "window one wider": sizes("mask", 1),
        "window two wider": sizes("mask", 2),
        "no learned sink": lambda c, w, p: [w.update({k: w[k] - 50}) for k in w if k.endswith("sink")],
        "no sink anywhere": replaced("sink_softmax", lambda f: lambda s, sink: torch.softmax(s, dim=-1)),
        "no biases": scaled(".b", 0.0),
        "no value mixing": scaled("vmix", 0.0),
        "temperature one position late": replaced("query_temperature", lambda f: lambda p, *a: f(p - 1, *a)),
        "previous token forgotten": replaced("bigram_rows", lambda f: lambda t, b, mp, mc: [b] * len(t)),
        "positions shifted": replaced("sinusoid", lambda f: lambda p, *a: f(p + 1, *a)),
        "gate not clamped": replaced("clamped_gate", lambda f: lambda g, u, limit: f(g, u, 1e9)),
        "norm weight not around one": replaced("rms_norm", lambda f: lambda x, w, e: f(x, w - 1.0, e)),
    }[name]


@pytest.mark.parametrize("mistake", [
    "window one wider", "window two wider", "no learned sink", "no sink anywhere", "no biases", "no value mixing",
    "temperature one position late", "previous token forgotten", "positions shifted", "gate not clamped",
    "norm weight not around one"])
def test_the_test_models_would_show_a_mistake(mistake, monkeypatch):
    """A mistake planted in the plain implementation moves the logits of a test model by several times the bf16
    tolerance of the GPU tests, so those tests cannot pass with it.  (A temperature that steps one position late
    touches few positions and by little: a thousand times the fp32 tolerance.)"""

    config = copy.deepcopy(CONFIGS["grouped"])
    weights, tokens = oracle_weights(make_weights(config)), make_tokens(config, 60, 1)
    want = plain.forward(config, weights, tokens)[0]
    _mistake(mistake)(config, weights, monkeypatch)
    assert logit_error(plain.forward(config, weights, tokens)[0], want) > (0.03 if "temperature" in mistake else 0.2)


def test_runner_weights_follow_the_requested_page_size():
    tensors = make_weights(CONFIGS["grouped"])
    assert runner_weights(CONFIGS["grouped"], tensors, CPU, torch.float32, page=32).shape.page == 32
