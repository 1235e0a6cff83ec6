"""Host side of the Ripesun design, state slots in the step machinery, and what the plain implementation says about the
test models, on the CPU."""

from __future__ import annotations

import copy
import json
import math

import pytest
import torch

from mini_inference_engine_b200.engine import registry
from mini_inference_engine_b200.engine.checkpoint import Checkpoint, save_safetensors
from mini_inference_engine_b200.engine.kernels.recurrence import StateBuffer, segment_tokens
from mini_inference_engine_b200.engine.model_runner.continuous import ContinuousBatcher, PagePoolExhausted, SlotPool
from mini_inference_engine_b200.engine.model_runner.replay import TraceEntry, TraceSession
from mini_inference_engine_b200.engine.model_runner.ripesun import RipesunShape, RipesunWeights
from mini_inference_engine_b200.engine.model_runner.step_runner import DecodeBuffers, MixedBuffers, PagedStepRunner
from oracle import ripesun_model as plain
from ripesun_models import CONFIGS, logit_error, make_tokens, make_weights, oracle_weights, runner_weights

CPU = torch.device("cpu")


# -- configuration, registry, checkpoints -----------------------------------------------------------

def test_configuration_decides_sizes_and_branches():
    shape = RipesunShape.from_config(CONFIGS["mixed"])
    first, own, average, bare, reader, _ = (layer.mixer for layer in shape.layers)
    assert (first.heads, first.dim, first.vdim, first.decay) == (3, 24, 40, (0.5, 0.97, 0.8))
    assert (own.row, own.qk_dim, own.window, own.kv_from) == (48, 24, 20, None) and average.width == 48
    assert bare.rot_base == 500.0 and shape.layers[3].ff is None
    assert (reader.kv_from, reader.kv_rank, reader.window) == (1, 40, 45)
    names = shape.tensor_shapes()
    assert names["l1.mix.dkv"] == (48, 72) and "l4.mix.dkv" not in names and "l4.mix.dkv.norm" not in names
    assert names["l4.mix.uk"] == (24, 40) and "l3.norm2" not in names and names["l3.norm1b"] == (72,)
    assert names["side.embed"] == (97, 48) and names["l0.mix.norm"] == (120,) and names["l2.mix.z.b"] == (48,)
    wide = RipesunShape.from_config(CONFIGS["wide"])
    assert (wide.layers[0].mixer.rotated, wide.layers[0].mixer.rot_dim, wide.residual_mult) == (16, 24, 1.0)


@pytest.mark.parametrize("change, message", [
    (lambda c: c["layers"][0].update(type="attention"), "unknown type"),
    (lambda c: c["layers"][1]["mlp"].update(kind="experts"), "unknown feed-forward"),
    (lambda c: c["layers"][1]["mixer"]["mask"].update(size=0), "window"),
    (lambda c: c["layers"][1]["mixer"]["rot"].update(dims=10), "rotated"),
    (lambda c: c["layers"][4]["mixer"].update(kv_from=2), "earlier layer"),
    (lambda c: c["layers"][4]["mixer"].update(kv_from=5), "earlier layer"),
    (lambda c: c["layers"][5]["mixer"].update(kv_from=4), "earlier layer"),
    (lambda c: c["layers"][4]["mixer"].update(kv_rank=48), "equal"),
    (lambda c: c["layers"][4]["mixer"]["rot"].update(base=2.0), "equal"),
    (lambda c: c["layers"][0]["mixer"].update(decay=[0.5]), "decay"),
])
def test_unusable_configurations_are_refused(change, message):
    config = copy.deepcopy(CONFIGS["mixed"])
    change(config)
    with pytest.raises(ValueError, match=message):
        RipesunShape.from_config(config)


def test_registry_and_checkpoint(tmp_path):
    design = registry.design_for({"architecture": "Ripesun"})
    assert design.recurrent and torch.float32 in design.dtypes
    assert not registry.design_for({"architecture": "Tidelorn"}).recurrent
    config, tensors = CONFIGS["mixed"], make_weights(CONFIGS["mixed"])
    (tmp_path / "config.json").write_text(json.dumps(config))
    save_safetensors(tmp_path / "model.safetensors", tensors)
    checkpoint = Checkpoint(tmp_path)
    weights = design.checkpoint_weights(design.shape(config), checkpoint, CPU, torch.float32)
    assert checkpoint.unused() == []
    assert torch.equal(weights.layers[0].inputs, torch.cat([tensors[f"l0.mix.{n}"] for n in "qkvg"]).float())
    assert torch.equal(weights.layers[1].down, torch.cat([tensors["l1.mix.dq"], tensors["l1.mix.dkv"]]).float())
    assert torch.equal(weights.layers[4].down, tensors["l4.mix.dq"].float()) and weights.layers[4].kv_norm is None
    assert torch.equal(weights.layers[2].side_table, tensors["side.embed"][:, 16:24].float())


def test_expansion_makes_whole_keys_and_values():
    tensors = make_weights(CONFIGS["mixed"])
    w = runner_weights(CONFIGS["mixed"], tensors, CPU, torch.float32).layers[3]
    row = torch.randn(72, generator=torch.Generator().manual_seed(0))
    both = w.expand @ row
    keys, values = both[:6 * 40].view(6, 40), both[6 * 40:].view(6, 16)
    latent = row[:56]
    assert torch.allclose(keys[:, :24], (tensors["l3.mix.uk"].float() @ latent).view(6, 24), atol=1e-5)
    assert torch.equal(keys[:, 24:], row[56:].expand(6, 16))
    assert torch.allclose(values, (tensors["l3.mix.uv"].float() @ latent).view(6, 16), atol=1e-5)


def test_random_weights_have_the_checkpoint_form():
    shape = RipesunShape.from_config(CONFIGS["mixed"])
    a, b = (RipesunWeights.random(shape, CPU, seed=3) for _ in range(2))
    assert torch.equal(a.layers[1].expand, b.layers[1].expand) and a.layers[2].inputs.shape == (144, 72)
    assert a.weight_bytes() > 2 * a.head.numel()


def test_segments_are_cut_only_when_lanes_are_few():
    assert segment_tokens(200, 1) == 0 and segment_tokens(5000, 75) == 0
    assert segment_tokens(300, 4) == 256 and segment_tokens(8192, 16) == 960
    assert segment_tokens(1 << 20, 64, sm_count=148) % 64 == 0


# -- state slots in the step machinery ----------------------------------------------------------------

def test_slot_pool():
    slots = SlotPool(2)
    assert (slots.take(), slots.take(), slots.free_slots) == (0, 1, 0)
    with pytest.raises(PagePoolExhausted):
        slots.take()
    slots.give_back(1)
    assert slots.take() == 1


def test_state_buffer_layout():
    state = StateBuffer([6, 8], 3, CPU)
    assert state.offsets == [0, 8] and state.layer(1).shape == (3, 8) and state.layer(1).stride(0) == 16
    state.rows[1] = 4.0
    state.copy(1, 2)
    assert state.rows.sum() == 2 * 16 * 4.0


def test_decode_rows_carry_slots_and_padding_rows_scratch_slots():
    buffers = DecodeBuffers(3, 4, CPU, (20, 21, 22), page=4, scratch_slots=(8, 9, 10))
    assert buffers.state_slots.tolist() == [8, 9, 10]
    buffers.pack_rows(["a", "b"], [1, 2], [3, 4], [[0], [1]], slots=[5, 0])
    assert buffers.state_slots.tolist() == [5, 0, 10]
    buffers.pack_rows(["b"], [2], [5], [[1, 2]], slots=[0])
    assert buffers.state_slots.tolist() == [0, 9, 10]
    with pytest.raises(ValueError, match="state slot"):
        buffers.pack_rows(["b"], [2], [5], [[1, 2]])
    assert DecodeBuffers(3, 4, CPU, (20, 21, 22), page=4).state_slots is None


def test_mixed_rows_carry_slots_in_table_row_order():
    buffers = MixedBuffers(2, 8, 2, 4, CPU, (20, 21), (22, 23), 4, decode_slots=(8, 9), chunk_slot=10)
    assert buffers.state_slots.tolist() == [8, 9, 10, 10, 10]
    buffers.pack([1], [3], [[0]], [([1, 2], 0, [1]), ([3], 4, [2, 3])], slots=[6, 2, 4])
    assert buffers.state_slots.tolist() == [6, 9, 2, 4, 10]
    with pytest.raises(ValueError, match="state slot"):
        buffers.pack([1], [3], [[0]], [([1, 2], 0, [1])], slots=[6])


class _Summing(PagedStepRunner):
    """A recurrent stand-in without a GPU: a request's state is the sum of its tokens, the next token state mod 50."""

    wants_chunk_starts = True

    class _Shape:
        page = 4

    def __init__(self, **kw):
        super().__init__(self._Shape, CPU, num_pages=40, max_context=64, chunk_buckets=(8,), **kw)
        self.state = torch.full((self.total_slots,), -1000)
        self.starts = []

    def copy_state(self, source, target):
        self.state[target] = self.state[source]

    def _advance(self, slot, tokens, start):
        before = 0 if start == 0 else int(self.state[slot])
        self.state[slot] = before + sum(tokens)
        return int(self.state[slot]) % 50

    def decode_forward(self, ids, lengths, tables, return_logits=False, *, state_slots):
        out = [self._advance(s, [t], n - 1) for s, t, n in zip(state_slots.tolist(), ids.tolist(), lengths.tolist())]
        return torch.tensor(out)

    def mixed_forward(self, ids, tok2seq, positions, tables, *, decode_rows, decode_lengths, cu_seqlens, kv_lens,
                      max_query_len, logit_rows, return_logits=False, state_slots, chunk_starts):
        assert len(state_slots) == decode_rows + len(chunk_starts)
        slots, ids, cu, pos = state_slots.tolist(), ids.tolist(), cu_seqlens.tolist(), positions.tolist()
        out = [self._advance(slots[r], [ids[r]], pos[r]) for r in range(decode_rows)]
        for r, start in enumerate(chunk_starts):
            begin, end = decode_rows + cu[r], decode_rows + cu[r + 1]
            assert pos[begin] == start
            out.append(self._advance(slots[decode_rows + r], ids[begin:end], start))
        return torch.tensor(out)

    def check_status(self):
        pass


def _summed(prompt, new):
    total, out = sum(prompt), []
    for _ in range(new):
        out.append(total % 50)
        total += out[-1]
    return out


@pytest.mark.parametrize("mixed", [False, True])
@pytest.mark.parametrize("prefix", [False, True])
def test_batcher_moves_slots_with_requests(mixed, prefix):
    runner = _Summing(max_batch=3, state_slots=5)
    batcher = ContinuousBatcher(runner, max_prefill_tokens=6, mixed=mixed, use_graphs=False, prefix_cache=prefix)
    generator = torch.Generator().manual_seed(0)
    common = torch.randint(0, 50, (12,), generator=generator).tolist()
    requests = {}
    for rid in range(9):
        tail = torch.randint(0, 50, (int(torch.randint(1, 12, (), generator=generator)),), generator=generator).tolist()
        requests[rid] = ((common if rid % 2 else common[:8]) + tail, 1 + rid % 5)
        batcher.submit(rid, *requests[rid])
    results = batcher.run()
    assert results == {rid: _summed(*request) for rid, request in requests.items()}
    assert batcher.slots.free_slots == 5 - len(batcher._prefix_states) and len(batcher._prefix_states) <= 2
    assert (batcher.prefix_hits > 0) == prefix
    batcher.drop_prefix_cache()
    assert batcher.slots.free_slots == 5 and batcher.pool.free_pages == 40


def test_batcher_needs_a_slot_per_row():
    with pytest.raises(ValueError, match="state slot"):
        ContinuousBatcher(_Summing(max_batch=3, state_slots=2))


def test_trace_session_gives_slots_back():
    class Logits(_Summing):
        def _both(self, out):
            return out, out.unsqueeze(1).float()

        def decode_forward(self, *a, return_logits=False, **kw):
            return self._both(super().decode_forward(*a, **kw))

        def mixed_forward(self, *a, return_logits=False, logit_rows, **kw):
            return self._both(super().mixed_forward(*a, logit_rows=logit_rows, **kw))

    session = TraceSession(Logits(max_batch=2, state_slots=2))
    session.step([TraceEntry("a", [1, 2, 3], [2]), TraceEntry("b", [4, 5], [])])
    got = session.step([TraceEntry("b", [6], [0]), TraceEntry("a", [7], [0])])
    assert got.flatten().tolist() == [15.0, 13.0]
    with pytest.raises(PagePoolExhausted):
        session.step([TraceEntry("c", [1], [])])
    assert "c" not in session.sequences
    session.end(["a"])
    assert session.step([TraceEntry("c", [9], [0])]).flatten().tolist() == [9.0]
    session.end(["b", "c"])
    assert session.slots.free_slots == 2 and session.pool.free_pages == 40


# -- the plain implementation: known values, and whether the test models would show a fault -----------

def test_mechanisms_have_their_known_values():
    x = torch.tensor([[1.0, 2.0, 3.0, 4.0, 5.0]], dtype=torch.float64)
    turned = plain.rotate(x, torch.tensor([3]), 4, 100.0)[0].tolist()
    a, b = 3.0, 3.0 / 10.0
    assert turned == pytest.approx([math.cos(a) - 2 * math.sin(a), 2 * math.cos(a) + math.sin(a),
                                    3 * math.cos(b) - 4 * math.sin(b), 4 * math.cos(b) + 3 * math.sin(b), 5.0])
    assert plain.visibility(4, 2).tolist() == [[True, False, False, False], [True, True, False, False],
                                               [False, True, True, False], [False, False, True, True]]
    weights = plain.sink_softmax(torch.tensor([[0.0, math.log(2), -math.inf]]), torch.tensor(math.log(5)))
    assert weights.tolist()[0] == pytest.approx([1 / 8, 2 / 8, 0.0])
    q = torch.tensor([[[1.0]], [[2.0]], [[1.0]]])
    out = plain.decayed_outer_products(q, torch.tensor([[[3.0]], [[1.0]], [[0.0]]]), torch.tensor([[[2.0]], [[5.0]], [[9.0]]]),
                                       [0.5])
    assert out.flatten().tolist() == [6.0, 16.0, 4.0]
    assert plain.gru_candidate(torch.tensor([0.0, 2.0, -math.log(3)])).tolist() == pytest.approx([0.5, 2.5, 0.25])
    steps = plain.gated_average(torch.tensor([[0.5], [0.25]]), torch.tensor([[4.0], [8.0]]))
    assert steps.flatten().tolist() == [2.0, 3.5]
    assert plain.softcap(torch.tensor(1e9), 7.0).item() == 7.0
    assert plain.gelu_tanh(torch.tensor(1.0)).item() == pytest.approx(0.841192, abs=1e-6)


def _mixers(kind, change):
    def apply(config, weights, patch):
        for layer in config["layers"]:
            if layer["type"] == kind:
                change(layer["mixer"])
    return apply


def _scaled(suffix, factor):
    def apply(config, weights, patch):
        for key in weights:
            if key.endswith(suffix):
                weights[key] = weights[key] * factor
    return apply


def _replaced(function, make):
    return lambda config, weights, patch: patch.setattr(plain, function, make(getattr(plain, function)))


def _half_rotation(x, positions, dims, base):
    """Entry i paired with entry i + dims / 2."""

    order = [i // 2 + (i % 2) * (dims // 2) for i in range(dims)] + list(range(dims, x.shape[-1]))
    back = [order.index(i) for i in range(x.shape[-1])]
    return _rotate(x[..., order], positions, dims, base)[..., back]


_rotate = plain.rotate


def _restart(f, at):
    def run(*tensors):
        *streams, last = tensors
        parts = [f(*(s[:at] for s in streams), last), f(*(s[at:] for s in streams), last)]
        return torch.cat(parts)
    return run


MISTAKES = {
    "window one wider": _mixers("latent_attention", lambda m: m["mask"].update(size=m["mask"]["size"] + 1)),
    "window one narrower": _mixers("latent_attention", lambda m: m["mask"].update(size=m["mask"]["size"] - 1)),
    "no sink": lambda c, w, p: [w.update({k: w[k] - 50}) for k in w if k.endswith("sink")],
    "sink scaled": _scaled("sink", 0.4),
    "no rotation": _replaced("rotate", lambda f: lambda x, p, d, b: x),
    "halves rotated": _replaced("rotate", lambda f: _half_rotation),
    "another base": _mixers("latent_attention", lambda m: m["rot"].update(base=m["rot"]["base"] * 3)),
    "decay twice": _mixers("lightning", lambda m: m.update(decay=[d * d for d in m["decay"]])),
    "decay before the token": _replaced("decayed_outer_products", lambda f: lambda q, k, v, d: f(
        q, k * torch.tensor(d, dtype=k.dtype).view(1, -1, 1), v, d)),
    "outer state lost": _replaced("decayed_outer_products", lambda f: _restart(f, 40)),
    "average state lost": _replaced("gated_average", lambda f: lambda z, c: torch.cat([f(z[:40], c[:40]), f(z[40:], c[40:])])),
    "gates swapped": _replaced("gated_average", lambda f: lambda z, c: f(1 - z, c)),
    "candidate without its half": _replaced("gru_candidate", lambda f: lambda u: torch.where(u >= 0, u, f(u))),
    "no gate biases": _scaled(".b", 0.0),
    "no silu": _replaced("silu", lambda f: lambda z: z),
    "no norm after a sublayer": _scaled("norm1b", 0.3),
    "no token input": _scaled("side.norm", 0.0),
    "token input of another layer": lambda c, w, p: w.update({"side.embed": w["side.embed"].roll(8, dims=1)}),
    "no residual multiplier": lambda c, w, p: c.update(residual_mult=1.0),
    "no embedding scale": lambda c, w, p: c["embedding"].update(scale=1.0),
    "no soft cap": lambda c, w, p: c.update(logit_softcap=1e9),
}
# These move few rows or move them little: hundreds of times the fp32 tolerance.
SUBTLE = {"sink scaled", "no soft cap", "average state lost", "window one wider", "window one narrower"}


@pytest.mark.parametrize("mistake", list(MISTAKES))
def test_the_test_models_would_show_a_mistake(mistake, monkeypatch):
    """A mistake planted in the plain implementation moves the logits of a test model by more than the bf16 tolerance of
    the GPU tests (subtle ones by hundreds of times the fp32 tolerance), so those tests cannot pass with it."""

    config = copy.deepcopy(CONFIGS["mixed"])
    weights, tokens = oracle_weights(make_weights(config)), make_tokens(config, 60, 1)
    want = plain.forward(config, weights, tokens)[0]
    MISTAKES[mistake](config, weights, monkeypatch)
    assert logit_error(plain.forward(config, weights, tokens)[0], want) > (0.02 if mistake in SUBTLE else 0.1)


def test_a_reader_without_its_source_layer_shows(monkeypatch):
    """A layer that reads another's cached rows differs clearly from one that projects its own."""

    config = copy.deepcopy(CONFIGS["wide"])
    weights, tokens = oracle_weights(make_weights(config)), make_tokens(config, 60, 1)
    want = plain.forward(config, weights, tokens)[0]
    del config["layers"][2]["mixer"]["kv_from"]
    for name in ("dkv", "dkv.norm"):
        weights[f"l2.mix.{name}"] = weights[f"l0.mix.{name}"]
    assert logit_error(plain.forward(config, weights, tokens)[0], want) > 0.2
