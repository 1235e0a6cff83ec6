"""Paged attention with sinks, windows and free head sizes: the three kernels against dense float64 attention.

Queries and keys are random, but for every query one key far back, one just inside and one just outside its
window (and, for whole-prefix rows, the first key) are planted along the query, so that a key that is missed or
wrongly seen changes the output by far more than rounding does.
"""

from __future__ import annotations

import math

import pytest
import torch

from mini_inference_engine_b200.engine.kv_cache.sink_attention import (
    attention_rows,
    sink_decode_attention,
    sink_decode_supported,
    sink_prefill_attention,
    sink_prefill_supported,
)
from mini_inference_engine_b200.engine.kv_cache.triton_paged_attention import decode_scratch
from oracle import tidelorn_model as plain

pytestmark = pytest.mark.gpu

# heads, kv_heads, dim, vdim, window
STREAMED = [
    (4, 4, 72, 32, None), (8, 2, 128, 128, None), (12, 4, 64, 64, 37), (6, 2, 40, 24, 16), (16, 1, 192, 128, None),
    (4, 4, 256, 256, 50), (5, 1, 72, 200, 1), (20, 1, 16, 64, 129), (3, 3, 8, 8, 128), (9, 3, 200, 136, 15),
]
ODD = [(3, 1, 20, 7, None, 5), (6, 2, 33, 65, 11, 3), (2, 2, 1, 1, 4, 1)]


class Case:
    """Random paged K/V of several sequences, and for each of them query rows at given positions."""

    def __init__(self, lengths, query_counts, heads, kv_heads, dim, vdim, window, page, dtype, seed=0, sinks="random"):
        generator = torch.Generator().manual_seed(seed)
        self.heads, self.kv_heads, self.dim, self.vdim, self.window, self.page = heads, kv_heads, dim, vdim, window, page
        self.scale = 1.3 / math.sqrt(dim)
        self.lengths, self.counts = list(lengths), list(query_counts)
        needed = [-(-n // page) for n in self.lengths]
        self.pages = sum(needed) + 5
        order = torch.randperm(self.pages, generator=generator).tolist()
        self.tables = torch.full((len(lengths), max(needed) + 2), -1, dtype=torch.int32)
        # Slots no token owns hold NaN: touching one with any weight, even zero, shows.
        self.keys = torch.full((self.pages, kv_heads, page, dim), math.nan, dtype=dtype)
        self.values = torch.full((self.pages, kv_heads, page, vdim), math.nan, dtype=dtype)
        self.sinks = {"random": torch.randn(heads, generator=generator) * 2, "zeros": torch.zeros(heads),
                      "large": torch.full((heads,), 9.0), "none": None}[sinks]
        self.queries, self.dense = [], []
        for row, (length, count) in enumerate(zip(self.lengths, self.counts)):
            k = torch.randn(length, kv_heads, dim, generator=generator)
            v = torch.randn(length, kv_heads, vdim, generator=generator)
            q = torch.randn(count, heads, dim, generator=generator)
            for i in range(count):
                pos = length - count + i
                marks = [0, pos // 2]
                if window is not None:
                    marks += [pos - window, pos - window + 1]
                for mark in marks[-2:] if i % 2 else marks[:2] + marks[-1:]:
                    if 0 <= mark <= pos and torch.rand((), generator=generator) < 8 / count:
                        for g in range(kv_heads):
                            lead = q[i, g * (heads // kv_heads)]
                            k[mark, g] = lead * (6.0 / (self.scale * float(lead.square().sum()) + 1e-9))
                            v[mark, g] = v[mark, g] + 3.0
            k, v, q = k.to(dtype), v.to(dtype), q.to(dtype)
            pages = [order.pop() for _ in range(needed[row])]
            self.tables[row, :len(pages)] = torch.tensor(pages, dtype=torch.int32)
            for t in range(length):
                self.keys[pages[t // page], :, t % page] = k[t]
                self.values[pages[t // page], :, t % page] = v[t]
            self.queries.append(q)
            self.dense.append((k.double(), v.double()))

    def expected(self) -> torch.Tensor:
        outs = []
        for (k, v), q, length, count in zip(self.dense, self.queries, self.lengths, self.counts):
            seen = plain.visibility(length, self.window)[length - count:]
            out = torch.empty(count, self.heads, self.vdim, dtype=torch.float64)
            for head in range(self.heads):
                g = head // (self.heads // self.kv_heads)
                scores = (q[:, head].double() @ k[:, g].t() * self.scale).masked_fill(~seen, -math.inf)
                sink = torch.tensor(-math.inf) if self.sinks is None else self.sinks[head].double()
                out[:, head] = plain.sink_softmax(scores, sink) @ v[:, g]
            outs.append(out)
        return torch.cat(outs)

    def on(self, device):
        self.status = torch.zeros(1, dtype=torch.int32, device=device)
        self.q = torch.cat(self.queries).to(device)
        self.out = torch.full((self.q.shape[0], self.heads, self.vdim), math.nan, dtype=self.q.dtype, device=device)
        self.common = dict(scale=self.scale, window=self.window, status=self.status,
                           sinks=None if self.sinks is None else self.sinks.to(device))
        return self.keys.to(device), self.values.to(device), self.tables.to(device)

    def rows(self, device):
        keys, values, tables = self.on(device)
        positions = torch.cat([torch.arange(n - c, n, dtype=torch.int32) for n, c in zip(self.lengths, self.counts)])
        owners = torch.cat([torch.full((c,), i, dtype=torch.int32) for i, c in enumerate(self.counts)])
        attention_rows(self.q, self.out, keys, values, positions.to(device), owners.to(device), tables, **self.common)

    def decode(self, device, split_policy=1):
        keys, values, tables = self.on(device)
        batch = len(self.lengths)
        scratch = decode_scratch(batch, self.heads, self.kv_heads, self.vdim, sum(self.lengths), device)
        lengths = torch.tensor(self.lengths, dtype=torch.int32, device=device)
        for slot in range(2):  # the second call reuses the first one's work plan
            self.out.fill_(math.nan)
            sink_decode_attention(self.q, self.out, keys, values, tables, lengths, scratch=scratch, use_plan=slot > 0,
                                  plan_slot=slot, split_policy=split_policy, **self.common)

    def prefill(self, device):
        keys, values, tables = self.on(device)
        cu = torch.tensor([0, *self.counts], dtype=torch.int32).cumsum(0).to(torch.int32).to(device)
        kv = torch.tensor(self.lengths, dtype=torch.int32, device=device)
        sink_prefill_attention(self.q, self.out, keys, values, tables, cu, kv, max_query_len=max(self.counts),
                               **self.common)

    def check(self):
        want = self.expected()
        assert int(self.status.item()) == 0
        bound = (3e-6, 3e-6) if self.q.dtype == torch.float32 else (2.0 ** -8, 2e-3)
        error = (self.out.cpu().double() - want).abs() - bound[0] * want.abs()
        assert float(error.max()) <= bound[1], float(error.max())  # NaN fails as well


RAGGED = [1, 2, 15, 16, 17, 130, 700, 2100]
CHUNKS = [(1, 1), (130, 130), (39, 2), (577, 77), (131, 128), (1300, 300)]  # (length, new tokens)


@pytest.mark.parametrize("sizes", STREAMED, ids=str)
def test_decode_kernel(sizes, device):
    assert sink_decode_supported(sizes[2], sizes[3], 16, torch.bfloat16)
    case = Case(RAGGED, [1] * len(RAGGED), *sizes, 16, torch.bfloat16)
    for policy in (1, 0, 64):
        case.decode(device, policy)
        case.check()


@pytest.mark.parametrize("sizes", STREAMED, ids=str)
def test_prefill_kernel(sizes, device):
    assert sink_prefill_supported(sizes[0], sizes[1], sizes[2], sizes[3], 16, torch.bfloat16, 0.1)
    case = Case([n for n, _ in CHUNKS], [c for _, c in CHUNKS], *sizes, 16, torch.bfloat16)
    case.prefill(device)
    case.check()


@pytest.mark.parametrize("sinks", ["none", "zeros", "large"])
@pytest.mark.parametrize("window", [None, 1, 40])
def test_sink_forms(sinks, window, device):
    """No sink, a sink score of zero and a sink above every score, with and without a window (whole tiles of a
    windowed row are hidden before its first visible key)."""

    chunks = Case([300, 150], [290, 5], 4, 2, 64, 64, window, 16, torch.bfloat16, seed=3, sinks=sinks)
    chunks.prefill(device)
    chunks.check()
    rows = Case([300, 150], [290, 5], 4, 2, 64, 64, window, 16, torch.bfloat16, seed=3, sinks=sinks)
    rows.rows(device)
    rows.check()
    decode = Case([300, 150, 3], [1, 1, 1], 4, 2, 64, 64, window, 16, torch.bfloat16, seed=4, sinks=sinks)
    decode.decode(device, 32)
    decode.check()


@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("sizes", STREAMED[:4] + [s[:5] for s in ODD], ids=str)
def test_row_kernel(sizes, dtype, device):
    page = next((s[5] for s in ODD if s[:5] == sizes), 16)
    case = Case([1, 40, 131, 517], [1, 17, 2, 60], *sizes, page, dtype, seed=1)
    case.rows(device)
    case.check()


def test_pages_of_several_tiles(device):
    for page in (32, 48):
        case = Case(RAGGED, [1] * len(RAGGED), 4, 2, 96, 40, 70, page, torch.bfloat16, seed=5)
        case.decode(device)
        case.check()
        case = Case([n for n, _ in CHUNKS], [c for _, c in CHUNKS], 4, 2, 96, 64, 70, page, torch.bfloat16, seed=6)
        case.prefill(device)
        case.check()


def test_long_context_past_the_shared_page_ids(device):
    """A chunk at the end of 66k tokens: more pages than the prefill kernel keeps in shared memory, and a split
    decode of the same context."""

    length = 66_000
    sizes = (2, 1, 16, 16, None)
    case = Case([length], [3], *sizes, 16, torch.bfloat16, seed=7)
    case.prefill(device)
    case.check()
    case = Case([length, 5], [1, 1], *sizes, 16, torch.bfloat16, seed=8)
    case.decode(device)
    case.check()


def test_unsupported_sizes_are_refused_on_the_host(device):
    assert not sink_decode_supported(20, 32, 16, torch.bfloat16)
    assert not sink_decode_supported(64, 264, 16, torch.bfloat16)
    assert not sink_decode_supported(64, 64, 8, torch.bfloat16)
    assert not sink_decode_supported(64, 64, 16, torch.float32)
    assert not sink_prefill_supported(4, 2, 264, 64, 16, torch.bfloat16, 0.1)
    assert not sink_prefill_supported(4, 2, 64, 64, 16, torch.bfloat16, -0.1)
    case = Case([20], [1], 2, 1, 20, 8, None, 16, torch.bfloat16)
    with pytest.raises(ValueError, match="multiples of 8"):
        case.decode(device)


def test_bad_metadata_sets_the_status_word(device):
    case = Case([20], [1], 2, 1, 16, 16, None, 16, torch.float32)
    keys, values, tables = case.on(device)
    word = lambda t: torch.tensor([t], dtype=torch.int32, device=device)  # noqa: E731
    attention_rows(case.q, case.out, keys, values, word(19), word(7), tables, **case.common)
    assert int(case.status.item()) == 8 and not case.out.any()
    case.status.zero_()
    attention_rows(case.q, case.out, keys, values, word(10_000), word(0), tables, **case.common)
    assert int(case.status.item()) == 2 and not case.out.any()
