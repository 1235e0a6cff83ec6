"""Latent attention's kernels: the cached row, rotation, the streaming decode kernel and the row kernel over a latent
cache, and the gathered spans of packed chunks, each against dense float64.

As in the other attention tests, keys just inside and just outside a query's window (and far back) are planted along
the query, and slots nobody owns hold NaN."""

from __future__ import annotations

import math

import pytest
import torch

from mini_inference_engine_b200.engine.kernels.decoder_glue import sinusoid_turns
from mini_inference_engine_b200.engine.kv_cache.latent_attention import (
    VisibleSpans,
    latent_decode_attention,
    latent_decode_scratch,
    latent_decode_supported,
    latent_norm_write,
    rotate_heads,
)
from mini_inference_engine_b200.engine.kv_cache.sink_attention import attention_rows, sink_prefill_attention
from oracle import ripesun_model as plain

pytestmark = pytest.mark.gpu

DTYPES = pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16], ids=["fp32", "bf16"])


def close(got, want):
    unit = {torch.float32: 4e-6, torch.bfloat16: 2.0 ** -8}[got.dtype]
    error = (got.cpu().double() - want.double()).abs()
    assert bool((error <= unit * want.double().abs() + unit * 2.0).all()), float(error.max())


class Case:
    """A latent cache of several sequences and one query row (all heads) at the end of each."""

    def __init__(self, lengths, heads, rank, rot, window, *, page=16, dtype=torch.bfloat16, seed=0, sinks="random"):
        generator = torch.Generator().manual_seed(seed)
        self.lengths, self.heads, self.rank, self.window = list(lengths), heads, rank, window
        dim = rank + rot
        self.scale = 1.3 / math.sqrt(dim)
        needed = [-(-n // page) for n in lengths]
        pages = sum(needed) + 4
        order = torch.randperm(pages, generator=generator).tolist()
        self.tables = torch.full((len(lengths), max(needed) + 3), -1, dtype=torch.int32)
        self.pages = torch.full((pages, 1, page, dim), math.nan, dtype=dtype)
        self.sinks = {"random": torch.randn(heads, generator=generator) * 2, "none": None,
                      "large": torch.full((heads,), 8.0)}[sinks]
        self.query = torch.randn(len(lengths), heads, dim, generator=generator).to(dtype)
        rows = []
        for row, length in enumerate(lengths):
            keys = torch.randn(length, dim, generator=generator)
            pos = length - 1
            marks = [0, pos // 2] + ([pos - window, pos - window + 1] if window else [])
            for i, mark in enumerate(marks):  # each planted along another head's query
                if 0 <= mark <= pos:
                    lead = self.query[row, i % heads].float()
                    keys[mark] = lead * (6.0 / (self.scale * float(lead.square().sum())))
            keys = keys.to(dtype)
            mine = [order.pop() for _ in range(needed[row])]
            self.tables[row, :len(mine)] = torch.tensor(mine, dtype=torch.int32)
            for t in range(length):
                self.pages[mine[t // page], 0, t % page] = keys[t]
            rows.append(keys.double())
        self.want = torch.empty(len(lengths), heads, rank, dtype=torch.float64)
        for row, (length, keys) in enumerate(zip(lengths, rows)):
            seen = plain.visibility(length, window or length)[-1]
            scores = (self.query[row].double() @ keys.t() * self.scale).masked_fill(~seen, -math.inf)
            sink = torch.full((heads, 1), -math.inf) if self.sinks is None else self.sinks.double().unsqueeze(1)
            self.want[row] = plain.sink_softmax(scores, sink) @ keys[:, :rank]

    def run(self, device, kind, split_policy=1):
        status = torch.zeros(1, dtype=torch.int32, device=device)
        pages, tables, query = self.pages.to(device), self.tables.to(device), self.query.to(device)
        out = torch.full((*query.shape[:2], self.rank), math.nan, dtype=query.dtype, device=device)
        common = dict(scale=self.scale, window=self.window, status=status,
                      sinks=None if self.sinks is None else self.sinks.to(device))
        lengths = torch.tensor(self.lengths, dtype=torch.int32, device=device)
        if kind == "rows":
            attention_rows(query, out, pages, pages[..., :self.rank], lengths - 1, None, tables, **common)
        else:
            scratch = latent_decode_scratch(len(self.lengths), self.heads, self.rank, sum(self.lengths), device)
            for reuse in (False, True):
                out.fill_(math.nan)
                latent_decode_attention(query, out, pages, tables, lengths, scratch=scratch, use_plan=reuse,
                                        split_policy=split_policy, **common)
        assert int(status.item()) == 0
        close(out, self.want)


# heads, rank, rotated part, window, page
SIZES = [(5, 40, 8, 20, 16), (16, 512, 64, 100, 16), (20, 136, 24, 33, 32), (40, 512, 64, None, 16), (33, 64, 0, 16, 16),
         (1, 8, 8, 1, 16), (12, 200, 40, 129, 48), (64, 256, 64, 64, 16), (17, 320, 8, 500, 16), (7, 480, 160, 48, 16)]


@pytest.mark.parametrize("heads, rank, rot, window, page", SIZES)
@pytest.mark.parametrize("split_policy", [0, 1, 64, 80])
def test_streaming_decode(heads, rank, rot, window, page, split_policy, device):
    assert latent_decode_supported(rank + rot, rank, page, torch.bfloat16)
    lengths = [1, 2, 15, 16, 17, 63, 64, 65, 130, 401, 640]
    for sinks in ("random", "none", "large"):
        Case(lengths, heads, rank, rot, window, page=page, sinks=sinks).run(device, "stream", split_policy)


def test_streaming_decode_many_requests(device):
    """More work items than the GPU has SMs: every CTA walks several, with stages in flight across items."""

    generator = torch.Generator().manual_seed(3)
    lengths = torch.randint(1, 300, (230,), generator=generator).tolist()
    for heads in (16, 48):
        Case(lengths, heads, 128, 64, 90, seed=4).run(device, "stream")
        Case(lengths, heads, 96, 32, 77, seed=5).run(device, "stream", 64)


@DTYPES
@pytest.mark.parametrize("heads, rank, rot, window, page", [(5, 40, 8, 20, 16), (3, 11, 6, 9, 5), (2, 512, 64, None, 16)])
def test_row_kernel_over_a_latent_cache(dtype, heads, rank, rot, window, page, device):
    Case([1, 9, 17, 100, 203], heads, rank, rot, window, page=page, dtype=dtype).run(device, "rows")


def test_decode_support_is_decided_by_sizes():
    assert not latent_decode_supported(576, 512, 16, torch.float32)
    assert not latent_decode_supported(577, 512, 16, torch.bfloat16)
    assert not latent_decode_supported(648, 512, 16, torch.bfloat16)
    assert not latent_decode_supported(600, 520, 16, torch.bfloat16)
    assert not latent_decode_supported(576, 512, 5, torch.bfloat16)


@DTYPES
@pytest.mark.parametrize("q_rank, rank, rot, rotated", [(32, 40, 8, 8), (9, 11, 6, 4), (1536, 512, 64, 64), (24, 16, 0, 0)])
def test_norms_rotation_and_page_write(dtype, q_rank, rank, rot, rotated, device):
    generator = torch.Generator().manual_seed(0)
    page, positions = 16, [0, 1, 15, 16, 77, 31]
    rows = torch.randn(6, q_rank + rank + rot, generator=generator).to(dtype)
    q_weight, weight = (torch.randn(n, generator=generator).to(dtype) for n in (q_rank, rank))
    owners = [0, 0, 1, 1, 1, 0]
    tables = torch.tensor([[4, 2, -1, -1, -1], [0, 3, 5, 6, 1]], dtype=torch.int32)
    pages = torch.full((7, 1, page, rank + rot), math.nan, dtype=dtype, device=device)
    status = torch.zeros(1, dtype=torch.int32, device=device)
    turns = sinusoid_turns(rotated, 700.0, device) if rotated else None
    arguments = (torch.tensor(positions, device=device), torch.tensor(owners, device=device), tables.to(device))
    sizes = dict(q_rank=q_rank, rank=rank, rot_dim=rot, rotated=rotated, eps=1e-3, status=status)
    got = latent_norm_write(rows.to(device), q_weight.to(device), weight.to(device), turns, pages, *arguments, **sizes)
    close(got, plain.rms_norm(rows[:, :q_rank].double(), q_weight.double(), 1e-3))
    latent = plain.rms_norm(rows[:, q_rank:q_rank + rank].double(), weight.double(), 1e-3)
    shared = plain.rotate(rows[:, q_rank + rank:].double(), torch.tensor(positions), rotated, 700.0)
    written = pages.cpu()
    for i, (pos, owner) in enumerate(zip(positions, owners)):
        close(written[tables[owner, pos // page], 0, pos % page], torch.cat([latent[i], shared[i]]))
    assert int(written.isnan().all(dim=-1).sum()) == 7 * page - 6
    # without pages only the queries come out; a position past the table is reported and skipped
    again = latent_norm_write(rows[:, :q_rank].contiguous().to(device), q_weight.to(device), None, None, None,
                              *arguments, **{**sizes, "rot_dim": 0, "rotated": 0})
    assert torch.equal(again, got) and int(status.item()) == 0
    arguments[0][0] = 80
    latent_norm_write(rows.to(device), q_weight.to(device), weight.to(device), turns, pages, *arguments, **sizes)
    assert int(status.item()) != 0


@DTYPES
def test_rotation_of_heads(dtype, device):
    """Far positions have the angle of the exact product; entries past the rotated ones pass; in place and into rows of
    another stride."""

    generator = torch.Generator().manual_seed(1)
    x = torch.randn(5, 3, 22, generator=generator).to(dtype)
    positions = torch.tensor([0, 1, 3, 1000, 100000])
    turns = sinusoid_turns(10, 1e4, device)
    want = x.double().clone()
    want[..., 8:] = plain.rotate(x[..., 8:].double(), positions, 10, 1e4)
    source, target = x.to(device), torch.zeros(5, 3, 20, dtype=dtype, device=device)
    rotate_heads(source[..., 8:], target[..., 6:], positions.to(device), turns, 10)
    close(target[..., 6:], want[..., 8:])
    assert not target[..., :6].any()
    rotate_heads(source[..., 8:], source[..., 8:], positions.to(device), turns, 10)
    close(source, want)


@pytest.mark.parametrize("dtype, cols", [(torch.float32, 11), (torch.bfloat16, 11), (torch.bfloat16, 48)])
@pytest.mark.parametrize("window", [1, 16, 37, 1000])
@pytest.mark.parametrize("exact", [True, False], ids=["starts", "bound"])
def test_spans_hold_what_the_chunks_see(dtype, cols, window, exact, device):
    generator = torch.Generator().manual_seed(2)
    starts, counts, page = [0, 40, 0, 119, 15], [33, 2, 0, 70, 1], 16
    lengths = [s + c for s, c in zip(starts, counts)]
    tables = torch.randperm(60, generator=generator)[:5 * 12].view(5, 12).to(torch.int32)
    pages = torch.randn(60, 1, page, cols, generator=generator).to(dtype)
    status = torch.zeros(1, dtype=torch.int32, device=device)
    cu = torch.tensor([0, *counts], dtype=torch.int32).cumsum(0).to(torch.int32).to(device)
    spans = VisibleSpans(cu, torch.tensor(lengths, dtype=torch.int32, device=device), window=window, tokens=sum(counts),
                         max_query_len=max(counts), max_context=192, chunk_starts=starts if exact else None, status=status)
    rows = spans.gather(pages.to(device), tables.to(device)).cpu()
    table, lens = spans.table.cpu(), spans.lens.tolist()
    assert int(status.item()) == 0
    for r, (start, length) in enumerate(zip(starts, lengths)):
        if counts[r] == 0:
            assert lens[r] == 0 and bool((table[r] == -1).all())
            continue
        first = max(0, start - window + 1) // 16 * 16
        assert lens[r] == length - first
        for i in range(-(-lens[r] // 16) * 16):
            token, row = first + i, int(table[r, i // 16]) * 16 + i % 16
            want = pages[tables[r, token // page], 0, token % page] if token < length else torch.zeros(cols).to(dtype)
            assert torch.equal(rows[row], want)
    if not exact:  # a span that does not fit is reported, not written past its buffer
        long = torch.tensor([1 << 20] * 5, dtype=torch.int32, device=device)
        VisibleSpans(cu, long, window=10 ** 7, tokens=104, max_query_len=70, max_context=192, status=status)
        assert int(status.item()) != 0


def test_chunks_over_gathered_keys(device):
    """Spans, a projection to heads and the prefill kernel against dense attention over the whole sequences."""

    generator = torch.Generator().manual_seed(5)
    heads, dim, vdim, cols, window, page = 6, 24, 40, 32, 21, 16
    starts, counts = [0, 50, 7, 200], [61, 2, 9, 37]
    lengths = [s + c for s, c in zip(starts, counts)]
    tables = torch.randperm(64, generator=generator).view(4, 16).to(torch.int32)
    pages = torch.randn(64, 1, page, cols, generator=generator).to(torch.bfloat16)
    expand = (torch.randn(heads * (dim + vdim), cols, generator=generator) / 4).to(torch.bfloat16)
    q = torch.randn(sum(counts), heads, dim, generator=generator).to(torch.bfloat16)
    sinks = torch.randn(heads, generator=generator)
    status = torch.zeros(1, dtype=torch.int32, device=device)
    cu = torch.tensor([0, *counts], dtype=torch.int32).cumsum(0).to(torch.int32).to(device)
    for exact in (True, False):
        spans = VisibleSpans(cu, torch.tensor(lengths, dtype=torch.int32, device=device), window=window,
                             tokens=sum(counts), max_query_len=61, max_context=256,
                             chunk_starts=starts if exact else None, status=status)
        both = spans.gather(pages.to(device), tables.to(device)) @ expand.to(device).t()
        out = torch.empty(sum(counts), heads, vdim, dtype=torch.bfloat16, device=device)
        sink_prefill_attention(q.to(device), out, spans.pages(both, 0, heads, dim),
                               spans.pages(both, heads * dim, heads, vdim), spans.table, cu, spans.lens,
                               max_query_len=61, scale=0.3, window=window, sinks=sinks.to(device), status=status)
        assert int(status.item()) == 0
        at = 0
        for r, (start, count) in enumerate(zip(starts, counts)):
            cached = torch.stack([pages[tables[r, t // page], 0, t % page] for t in range(start + count)])
            kv = (cached.to(device) @ expand.to(device).t()).cpu().double()
            k, v = kv[:, :heads * dim].view(-1, heads, dim), kv[:, heads * dim:].view(-1, heads, vdim)
            seen = plain.visibility(start + count, window)[start:]
            for h in range(heads):
                scores = (q[at:at + count, h].double() @ k[:, h].t() * 0.3).masked_fill(~seen, -math.inf)
                close(out[at:at + count, h], plain.sink_softmax(scores, sinks[h].double()) @ v[:, h])
            at += count
