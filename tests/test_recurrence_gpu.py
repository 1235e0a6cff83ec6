"""Recurrent mixers over state slots against the token-after-token recurrences in float64: chunks, single tokens,
portions through the slots, parallel segments, and slots that others have used."""

from __future__ import annotations

import pytest
import torch

from mini_inference_engine_b200.engine.kernels import recurrence
from mini_inference_engine_b200.engine.kernels.recurrence import StateBuffer, gated_average, outer_recurrence
from oracle import ripesun_model as plain

pytestmark = pytest.mark.gpu

DTYPES = pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16], ids=["fp32", "bf16"])
TOLERANCE = {torch.float32: 2e-5, torch.bfloat16: 2.0 ** -7}
MIXED_FORMS = {torch.float32: 1, torch.bfloat16: 4}  # chunks round silu(q), silu(k), silu(v) to bf16, single tokens do not


def close(got, want, dtype, factor=1):
    """Relative to the spread of each column of the result."""

    want = want.double()
    scale = want.square().mean(dim=0, keepdim=True).sqrt() + 1e-3
    error = ((got.cpu().double() - want).abs() / (scale + want.abs())).max()
    assert float(error) <= factor * TOLERANCE[dtype], float(error)


class Outer:
    def __init__(self, dim, vdim, decay, dtype, device, slots=6, seed=0):
        self.dim, self.vdim, self.decay, self.dtype, self.device = dim, vdim, list(decay), dtype, device
        self.heads = len(self.decay)
        self.generator = torch.Generator().manual_seed(seed)
        self.state = StateBuffer([5, self.heads * dim * vdim], slots, device)
        self.state.rows.fill_(float("nan"))  # a sequence that starts must not read what the slot holds
        self.status = torch.zeros(1, dtype=torch.int32, device=device)

    def rows(self, count):
        return torch.randn(count, self.heads * (2 * self.dim + self.vdim), generator=self.generator).to(self.dtype)

    def want(self, rows, single=False):
        """``single``: of the form that takes single tokens.  The tensor-core form of chunks has bf16 q, k and v."""

        keys = self.heads * self.dim
        q, k, v = (plain.silu(part.double()) for part in rows.split([keys, keys, self.heads * self.vdim], dim=1))
        if not single and recurrence._lib.load().mie_outer_recurrence_chunked(
                self.dim, self.vdim, recurrence._lib.DTYPE_CODES[self.dtype]):
            q, k, v = (part.to(torch.bfloat16).double() for part in (q, k, v))
        out = plain.decayed_outer_products(q.view(-1, self.heads, self.dim), k.view(-1, self.heads, self.dim),
                                           v.view(-1, self.heads, self.vdim), self.decay)
        return out.reshape(rows.shape[0], -1)

    def __call__(self, parts, slots, starts, decode=False):
        rows = torch.cat(parts).to(self.device)
        positions = torch.cat([torch.arange(s, s + len(p), dtype=torch.int32) for s, p in zip(starts, parts)])
        cu = torch.tensor([0, *map(len, parts)], dtype=torch.int32).cumsum(0).to(torch.int32).to(self.device)
        out = torch.full((rows.shape[0], self.heads * self.vdim), float("nan"), dtype=self.dtype, device=self.device)
        outer_recurrence(rows, out, torch.tensor(self.decay, device=self.device), self.state.layer(1),
                         torch.tensor(slots, device=self.device), positions.to(self.device), heads=self.heads,
                         dim=self.dim, value_dim=self.vdim, cu_seqlens=None if decode else cu,
                         max_query_len=max(map(len, parts)), status=self.status)
        assert int(self.status.item()) == 0
        return out.split([len(p) for p in parts])


class Average:
    def __init__(self, width, dtype, device, slots=6, seed=0):
        self.width, self.dtype, self.device = width, dtype, device
        self.generator = torch.Generator().manual_seed(seed)
        self.biases = [torch.randn(width, generator=self.generator).to(dtype) for _ in range(2)]
        self.state = StateBuffer([3, width], slots, device)
        self.state.rows.fill_(float("nan"))
        self.status = torch.zeros(1, dtype=torch.int32, device=device)

    def rows(self, count):
        return (torch.randn(count, 3 * self.width, generator=self.generator) * 2).to(self.dtype)

    def want(self, rows, single=False):
        z, u, g = rows.double().chunk(3, dim=1)
        z, u = torch.sigmoid(z + self.biases[0].double()), u + self.biases[1].double()
        return plain.gated_average(z, plain.gru_candidate(u)) * plain.silu(g)

    def __call__(self, parts, slots, starts, decode=False):
        rows = torch.cat(parts).to(self.device)
        positions = torch.cat([torch.arange(s, s + len(p), dtype=torch.int32) for s, p in zip(starts, parts)])
        cu = torch.tensor([0, *map(len, parts)], dtype=torch.int32).cumsum(0).to(torch.int32).to(self.device)
        out = torch.full((rows.shape[0], self.width), float("nan"), dtype=self.dtype, device=self.device)
        gated_average(rows, out, *(b.to(self.device) for b in self.biases), self.state.layer(1),
                      torch.tensor(slots, device=self.device), positions.to(self.device), width=self.width,
                      cu_seqlens=None if decode else cu, max_query_len=max(map(len, parts)), status=self.status)
        assert int(self.status.item()) == 0
        return out.split([len(p) for p in parts])


OUTER = [(24, 40, (0.5, 0.97)), (128, 128, (0.999,)), (64, 64, (0.9, 1.0, 0.0)), (72, 8, (0.8,)), (8, 136, (0.99, 0.3)),
         (5, 7, (0.95, 0.6)), (160, 24, (0.9,)), (16, 36, (0.99,))]


def mixers(dtype, device):
    for index, (dim, vdim, decay) in enumerate(OUTER):
        yield Outer(dim, vdim, decay, dtype, device, seed=index)
    for width in (48, 13, 1000):
        yield Average(width, dtype, device, seed=width)


@DTYPES
def test_whole_sequences(dtype, device):
    for mixer in mixers(dtype, device):
        parts = [mixer.rows(n) for n in (1, 63, 64, 65, 200, 2)]
        for got, part in zip(mixer(parts, [4, 2, 0, 1, 5, 3], [0] * 6), parts):
            close(got, mixer.want(part), dtype)


@DTYPES
def test_token_by_token_equals_whole(dtype, device):
    for mixer in mixers(dtype, device):
        parts = [mixer.rows(40), mixer.rows(40)]
        got = [[], []]
        for t in range(40):
            for mine, row in zip(got, mixer([p[t:t + 1] for p in parts], [3, 1], [t, t], decode=True)):
                mine.append(row)
        for mine, part in zip(got, parts):
            close(torch.cat(mine), mixer.want(part, single=True), dtype)


@DTYPES
def test_portions_of_unequal_requests(dtype, device):
    """Two requests advance by different portions, down to single tokens in either form; a third joins on a slot
    that a finished one has used."""

    for mixer in mixers(dtype, device):
        parts = [mixer.rows(150), mixer.rows(90), mixer.rows(70)]
        cuts = {0: [2, 61, 1, 64, 22], 1: [64, 1, 25], 2: [0, 0, 0, 3, 67]}
        slots, at, got = {0: 5, 1: 0, 2: 0}, [0, 0, 0], [[], [], []]
        for turn in range(5):
            live = [r for r in cuts if turn < len(cuts[r]) and cuts[r][turn]]
            pieces = [parts[r][at[r]:at[r] + cuts[r][turn]] for r in live]
            decode = all(len(p) == 1 for p in pieces)
            for r, rows in zip(live, mixer(pieces, [slots[r] for r in live], [at[r] for r in live], decode)):
                got[r].append(rows)
                at[r] += len(rows)
        for mine, part in zip(got, parts):
            close(torch.cat(mine), mixer.want(part), dtype, MIXED_FORMS[dtype])


@DTYPES
def test_parallel_segments(dtype, device):
    """Long portions run as parallel segments; they start from what earlier portions left, and leave the same state."""

    for mixer in (Outer(64, 128, (0.999, 0.9), dtype, device), Outer(128, 72, (0.97,), dtype, device), Average(96, dtype, device)):
        parts = [mixer.rows(700), mixer.rows(330), mixer.rows(1)]
        if isinstance(mixer, Outer):
            assert recurrence.segment_tokens(700, 3 * mixer.heads * 2) == 256
        first = mixer([parts[0][:30], parts[1]], [1, 2], [0, 0])
        second = mixer([parts[0][30:620], parts[2]], [1, 4], [30, 0])
        third = mixer([parts[0][620:]], [1], [620])
        for got, part in ((torch.cat([first[0], second[0], third[0]]), parts[0]), (first[1], parts[1]),
                          (second[1], parts[2])):
            close(got, mixer.want(part), dtype)


@DTYPES
def test_an_old_token_is_remembered(dtype, device):
    """One early key and value far larger than the rest: with a slow decay the last outputs are mostly that token."""

    mixer = Outer(32, 24, (0.999,), dtype, device)
    rows = mixer.rows(400) * 0.05
    rows[3, 32:88] = 6.0
    rows[390:, :32] = 2.0
    want = mixer.want(rows)
    forgotten = mixer.want(torch.cat([rows[:3], rows[4:]]))[-1]
    assert float((want[-1] - forgotten).abs().min()) > 0.5 * float(want[-1].abs().max())
    for cuts in ([400], [5, 395], [200, 200]):
        mixer.state.rows.fill_(float("nan"))
        got, at = [], 0
        for n in cuts:
            got += mixer([rows[at:at + n]], [2], [at])
            at += n
        close(torch.cat(got)[-10:], want[-10:], dtype)


def test_only_the_named_slots_change_and_bad_slots_are_reported(device):
    mixer = Outer(24, 40, (0.5, 0.97), torch.bfloat16, device)
    mixer.state.rows.fill_(7.0)
    mixer([mixer.rows(70), mixer.rows(3)], [1, 4], [0, 0])
    mixer([mixer.rows(1)], [2], [0], decode=True)
    changed = [bool((row != 7.0).any()) for row in mixer.state.rows]
    assert changed == [False, True, True, False, True, False]
    assert bool((mixer.state.rows[:, :8] == 7.0).all())  # the other layer's part of the row
    for run, name in ((mixer, "outer"), (Average(48, torch.bfloat16, device), "average")):
        for decode in (False, True):
            with pytest.raises(AssertionError):
                run([run.rows(1)], [6], [0], decode=decode)
            assert int(run.status.item()) == 512, name
            run.status.zero_()


def test_states_are_copied_whole(device):
    state = StateBuffer([5, 12, 1], 4, device)
    assert state.offsets == [0, 8, 20] and state.rows.shape == (4, 24)
    state.rows.copy_(torch.arange(96, dtype=torch.float32).view(4, 24))
    state.copy(2, 0)
    assert torch.equal(state.rows[0], state.rows[2]) and float(state.layer(1)[3, 0]) == 72 + 8
