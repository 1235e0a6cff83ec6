"""Glue kernels of decoders with a 32-bit residual stream, each against the plain equation in float64."""

from __future__ import annotations

import pytest
import torch

from mini_inference_engine_b200.engine.kernels.decoder_glue import (
    clamped_glu,
    embed_tokens,
    qkv_norm_mix_write,
    sinusoid_turns,
    sum_rms_norm,
)
from oracle import tidelorn_model as plain

pytestmark = pytest.mark.gpu

DTYPES = [torch.float32, torch.bfloat16]


def close(got, want, dtype=None):
    """Within rounding of the result's own number format (or ``dtype``'s), relative to each element."""

    unit = {torch.float32: 4e-6, torch.bfloat16: 2.0 ** -8}[dtype or got.dtype]
    error = (got.cpu().double() - want.double()).abs()
    assert bool((error <= unit * want.double().abs() + unit * 2.0).all()), float(error.max())


def status(device):
    return torch.zeros(1, dtype=torch.int32, device=device)


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("width", [64, 37, 1000])
def test_embedding_parts_and_previous_token(dtype, width, device):
    """Two sequences arrive in pieces (pieces of one token, pieces that start inside a page and on a page border);
    the bigram row of a piece's first token comes from the paged token history."""

    vocab, buckets, page = 50, 23, 4
    generator = torch.Generator().manual_seed(0)
    table = torch.randn(vocab, width, generator=generator).to(dtype)
    bigram = torch.randn(buckets + 1, width, generator=generator).to(dtype)
    tokens = {0: torch.randint(0, vocab, (19,), generator=generator).tolist(),
              1: torch.randint(0, vocab, (9,), generator=generator).tolist()}
    tables = torch.tensor([[3, 7, 1, 9, 5], [2, 8, 0, -1, -1]], dtype=torch.int32)
    history = torch.full((10, page), -1, dtype=torch.int32, device=device)
    turns = sinusoid_turns(width, 10000.0, device)
    want = {}
    for row, ids in tokens.items():
        rows = plain.bigram_rows(ids, buckets, 29, 11)
        want[row] = (table[ids].double() * 1.75 + bigram[rows].double()
                     + plain.sinusoid(torch.arange(len(ids)), width))
    word = status(device)
    at = {0: 0, 1: 0}
    for counts in ({0: 3, 1: 1}, {0: 1, 1: 3}, {0: 4}, {0: 1, 1: 1}, {1: 4, 0: 10}):
        ids, positions, owners, expected = [], [], [], []
        for row, count in counts.items():
            span = range(at[row], at[row] + count)
            ids += [tokens[row][p] for p in span]
            positions += list(span)
            owners += [row] * count
            expected.append(want[row][at[row]:at[row] + count])
            at[row] += count
        x32, x = embed_tokens(torch.tensor(ids, device=device), table.to(device),
                              torch.tensor(positions, dtype=torch.int32, device=device),
                              torch.tensor(owners, dtype=torch.int32, device=device), tables.to(device), scale=1.75,
                              page=page, num_pages=10, bigram=bigram.to(device), mul_prev=29, mul_cur=11,
                              history=history, turns=turns, status=word)
        close(x32, torch.cat(expected))
        close(x, torch.cat(expected))
    assert int(word.item()) == 0 and at == {0: 19, 1: 9}


def test_embedding_far_positions_large_ids_and_bare_table(device):
    vocab, width = 140_000, 48
    table = torch.randn(vocab, width, generator=torch.Generator().manual_seed(1))
    bigram = torch.randn(1_000_004, width, generator=torch.Generator().manual_seed(2))
    turns = sinusoid_turns(width, 10000.0, device)
    word, position = status(device), 131_071
    tables = torch.arange(8192, dtype=torch.int32, device=device).unsqueeze(0)
    history = torch.zeros(8192, 16, dtype=torch.int32, device=device)
    history.view(-1)[position - 1] = 139_998
    ids = torch.tensor([139_999], device=device)
    place = torch.tensor([position], dtype=torch.int32, device=device)
    multipliers = (2_000_003, 1_999_993)  # products beyond 32 bits
    x32, _ = embed_tokens(ids, table.to(device), place, None, tables, scale=0.5, page=16, num_pages=8192,
                          bigram=bigram.to(device), mul_prev=multipliers[0], mul_cur=multipliers[1], history=history,
                          turns=turns, status=word)
    row = (139_998 * multipliers[0] + 139_999 * multipliers[1]) % 1_000_003
    want = table[139_999].double() * 0.5 + bigram[row].double() + plain.sinusoid(torch.tensor([position]), width)[0]
    close(x32[0], want)
    x32, _ = embed_tokens(ids, table.to(device), place, None, tables, scale=3.0, page=16, num_pages=8192, status=word)
    close(x32[0], table[139_999].double() * 3.0)
    assert int(word.item()) == 0
    embed_tokens(torch.tensor([vocab], device=device), table.to(device), place, None, tables, scale=3.0, page=16,
                 num_pages=8192, status=word)
    assert int(word.item()) == 256


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("cols", [8, 37, 192, 4096, 20_000, 9_001])
def test_sum_and_norm(dtype, cols, device):
    generator = torch.Generator().manual_seed(cols)
    x = torch.randn(5, cols, generator=generator) * 3
    y = torch.randn(5, cols, generator=generator).to(dtype)
    weight = (torch.randn(cols, generator=generator) * 0.3).to(dtype)
    out32, out = sum_rms_norm(x.to(device), y.to(device), weight.to(device), eps=0.02, alpha=2.25, weight_offset=1.0)
    want = plain.rms_norm(2.25 * x.double() + y.double(), weight.double(), 0.02)
    close(out32, want)
    close(out, want)
    none32, out = sum_rms_norm(x.to(device), None, weight.to(device), eps=1e-6, keep32=False)
    close(out, plain.unit_rms(x.double(), 1e-6) * weight.double())
    assert none32 is None or dtype == torch.float32
    tiny, _ = sum_rms_norm((x * 1e-4).to(device), None, weight.to(device), eps=1e-2, weight_offset=1.0)
    close(tiny, plain.rms_norm(x.double() * 1e-4, weight.double(), 1e-2))  # eps under the root decides the scale


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("sizes", [(4, 2, 64, 32), (3, 1, 10, 7), (2, 2, 136, 264)], ids=str)
def test_between_projection_and_attention(dtype, sizes, device):
    """Unit norms, the query temperature around its steps, value mixing, and the page slots that are written."""

    heads, kv_heads, dim, vdim = sizes
    page, pages = 4, 12
    generator = torch.Generator().manual_seed(0)
    positions = torch.tensor([0, 5, 6, 7, 12, 13, 14, 20], dtype=torch.int32)
    owners = torch.tensor([0, 1, 1, 1, 0, 0, 0, 2], dtype=torch.int32)
    tables = torch.tensor([[4, 0, 2, 9, -1, -1], [1, 3, -1, -1, -1, -1], [5, 6, 7, 8, 10, 11]], dtype=torch.int32)
    tokens, width = len(positions), (heads + kv_heads) * dim + kv_heads * vdim
    qkv = (torch.randn(tokens, width, generator=generator) * 2).to(dtype)
    first = torch.randn(tokens, 3 + kv_heads * vdim, generator=generator).to(dtype)
    queries = torch.empty(tokens, heads, dim, dtype=dtype, device=device)
    keys = torch.full((pages, kv_heads, page, dim), 77.0, dtype=dtype, device=device)
    values = torch.full((pages, kv_heads, page, vdim), 77.0, dtype=dtype, device=device)
    word = status(device)
    args = (positions.to(device), owners.to(device), tables.to(device))
    common = dict(q_heads=heads, kv_heads=kv_heads, dim=dim, value_dim=vdim, status=word)
    qkv_norm_mix_write(qkv.to(device), queries, keys, values, *args, unit_norm=True, eps=0.01, temperature=(0.7, 7),
                       v_first=first.to(device)[:, 3:], lam=0.375, **common)
    q, k, v = (t.double() for t in qkv.split([heads * dim, kv_heads * dim, kv_heads * vdim], dim=1))
    q, k, v = q.view(tokens, heads, dim), k.view(tokens, kv_heads, dim), v.view(tokens, kv_heads, vdim)
    temperature = plain.query_temperature(positions, 0.7, 7).view(-1, 1, 1)
    assert len(set(temperature.flatten().tolist())) == 4  # positions 0-5, 6-12, 13-19 and 20
    close(queries, plain.unit_rms(q, 0.01) * temperature)
    mixed = plain.mix_values(v, first[:, 3:].double().view(tokens, kv_heads, vdim), torch.tensor(0.375).double())
    untouched = torch.ones(pages, page, dtype=torch.bool)
    for t in range(tokens):
        where = int(tables[owners[t], positions[t] // page]), int(positions[t] % page)
        close(keys[where[0], :, where[1]], plain.unit_rms(k[t], 0.01))
        close(values[where[0], :, where[1]], mixed[t])
        untouched[where] = False
    assert bool((keys.cpu().transpose(1, 2)[untouched] == 77.0).all())
    assert bool((values.cpu().transpose(1, 2)[untouched] == 77.0).all())
    qkv_norm_mix_write(qkv.to(device), queries, keys, values, *args, **common)  # every optional part off
    close(queries, q)
    close(values[4, :, 0], v[0])
    assert int(word.item()) == 0


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("cols", [8, 11, 328])
def test_clamped_gate(dtype, cols, device):
    gate_up = (torch.randn(6, 2 * cols, generator=torch.Generator().manual_seed(3)) * 3).to(dtype)
    gate_up[0, :2] = torch.tensor([9.0, -9.0])
    gate_up[0, cols:cols + 2] = torch.tensor([-9.0, 9.0])
    out = clamped_glu(gate_up.to(device), limit=1.25, slope=1.702, up_offset=1.0)
    close(out, plain.clamped_gate(gate_up[:, :cols].double(), gate_up[:, cols:].double(), 1.25))
