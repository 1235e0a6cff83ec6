"""Row kernels around normed sublayers, each against the plain equation in float64."""

from __future__ import annotations

import pytest
import torch

from mini_inference_engine_b200.engine.kernels.decoder_glue import gated_rms_norm, gelu, residual_norm_, softcap_
from oracle import ripesun_model as plain

pytestmark = pytest.mark.gpu

DTYPES = pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16], ids=["fp32", "bf16"])
WIDTHS = pytest.mark.parametrize("width", [64, 37, 1000, 9000])


def close(got, want):
    unit = {torch.float32: 4e-6, torch.bfloat16: 2.0 ** -8}[got.dtype]
    error = (got.cpu().double() - want.double()).abs()
    assert bool((error <= unit * want.double().abs() + unit * 2.0).all()), float(error.max())


def draw(seed, *shapes):
    generator = torch.Generator().manual_seed(seed)
    return [torch.randn(shape, generator=generator) for shape in shapes]


@DTYPES
@WIDTHS
def test_normed_result_joins_the_stream(dtype, width, device):
    x, y, w, n = draw(0, (5, width), (5, width), (width,), (width,))
    y, w, n = (t.to(dtype) for t in (y * 3, w, n))
    want = x.double() + 0.4 * plain.rms_norm(y.double(), w.double(), 1e-3)
    for following in (n, None):
        stream = x.to(device)
        out = residual_norm_(stream, y.to(device), w.to(device), None if following is None else following.to(device),
                             alpha=0.4, eps=1e-3)
        close(stream, want)
        close(out, want if following is None else plain.rms_norm(want, n.double(), 1e-3))
    stream = x.to(device)
    assert residual_norm_(stream, y.to(device), w.to(device), alpha=0.4, eps=1e-3, keep_rows=False) is None
    close(stream, want)


@DTYPES
@WIDTHS
def test_gelu_and_token_factor(dtype, width, device):
    x, table = draw(1, (6, width), (9, 3 * width + 1))
    x, table = (x * 3).to(dtype), table.to(dtype)
    close(gelu(x.to(device)), plain.gelu_tanh(x.double()))
    ids = torch.tensor([8, 0, 3, 3, 1, 7])
    part = table.to(device)[:, width:2 * width]
    status = torch.zeros(1, dtype=torch.int32, device=device)
    got = gelu(x.to(device), ids=ids.to(device), table=part, status=status)
    close(got, plain.gelu_tanh(x.double()) * table[ids, width:2 * width].double())
    assert int(status.item()) == 0
    gelu(x.to(device), ids=torch.tensor([8, 0, 9, 3, 1, 7], device=device), table=part, status=status)
    assert int(status.item()) == 256


@DTYPES
@WIDTHS
def test_gated_norm(dtype, width, device):
    x, wide, w = draw(2, (4, width), (4, 2 * width + 8), (width,))
    x, wide, w = x.to(dtype), (wide * 2).to(dtype), w.to(dtype)
    gate = wide.to(device)[:, width:2 * width]
    want = plain.rms_norm(x.double(), w.double(), 1e-2) * torch.sigmoid(wide[:, width:2 * width].double())
    close(gated_rms_norm(x.to(device), gate, w.to(device), eps=1e-2), want)


def test_soft_cap(device):
    logits, = draw(3, (3, 77))
    close(softcap_((logits * 40).to(device), 15.0), plain.softcap(logits.double() * 40, 15.0))
