"""Fused glue of decoders with a 32-bit residual stream, over ``csrc/decoder_glue.cu``.

Activations are bf16 or fp32 tensors, the residual stream is fp32.  Every constant is an argument, so that a
design picks the parts it has: which additive embeddings, which weight convention of a norm, whether query and
key heads are normalised, a query temperature, value mixing, the limits of a gated activation.
"""

from __future__ import annotations

import math

import torch

from ... import _lib


def sinusoid_turns(width: int, base: float, device: torch.device) -> torch.Tensor:
    """``[ceil(width / 2), 2]`` fp32: base^(-2i / width) / 2 pi, the turns of entry pair i per position, as a
    rounded number and its remainder."""

    turns = torch.tensor([base ** (-2.0 * i / width) / (2.0 * math.pi) for i in range((width + 1) // 2)],
                         dtype=torch.float64)
    high = turns.float()
    return torch.stack((high, (turns - high.double()).float()), dim=1).contiguous().to(device)


def embed_tokens(ids, table, positions, token_to_sequence, block_tables, *, scale: float, page: int, num_pages: int,
                 bigram=None, mul_prev: int = 0, mul_cur: int = 0, history=None, turns=None, keep_rows: bool = True,
                 status: torch.Tensor) -> tuple[torch.Tensor, torch.Tensor | None]:
    """``(fp32 rows, activation rows)`` of table[id] * scale (+ bigram row) (+ sinusoid); without ``keep_rows`` only
    the fp32 rows.  ``history`` (``[pages, page]`` int32) is the paged record of token ids the bigram part reads a
    predecessor from."""

    tokens, width = int(ids.shape[0]), int(table.shape[1])
    out32 = torch.empty(tokens, width, dtype=torch.float32, device=table.device)
    out = out32 if table.dtype == torch.float32 else None
    if out is None and keep_rows:
        out = torch.empty(tokens, width, dtype=table.dtype, device=table.device)
    _lib.check(_lib.load().mie_embed_tokens(
        _lib.index_arg(ids), _lib.ptr(table), int(table.shape[0]), float(scale), _lib.ptr(bigram),
        0 if bigram is None else int(bigram.shape[0]) - 1, int(mul_prev), int(mul_cur), _lib.ptr(turns),
        _lib.ptr(history), _lib.index_arg(positions), _lib.index_arg(token_to_sequence), _lib.index_arg(block_tables),
        _lib.ptr(out32), None if out is out32 else _lib.ptr(out), tokens, width, _lib.DTYPE_CODES[table.dtype], page,
        num_pages, int(block_tables.shape[0]), int(block_tables.shape[1]), _lib.ptr(status),
        _lib.stream_arg(table.device)))
    return out32, out


def sum_rms_norm(x32, y, weight, *, eps: float, alpha: float = 1.0, weight_offset: float = 0.0,
                 keep32: bool = True) -> tuple[torch.Tensor | None, torch.Tensor]:
    """RMS norm of ``alpha * x32 + y`` (``y`` may be None), weight ``weight_offset + weight``.  Returns the fp32
    rows (None unless ``keep32``) and the rows in the weight's dtype."""

    rows, cols = x32.shape
    out32 = torch.empty(rows, cols, dtype=torch.float32, device=x32.device) if keep32 else None
    if weight.dtype == torch.float32:
        out32 = torch.empty(rows, cols, dtype=torch.float32, device=x32.device) if out32 is None else out32
        out = out32
    else:
        out = torch.empty(rows, cols, dtype=weight.dtype, device=x32.device)
    _lib.check(_lib.load().mie_sum_rms_norm(
        _lib.ptr(x32), x32.stride(0), _lib.ptr(y), 0 if y is None else y.stride(0), float(alpha), _lib.ptr(weight),
        float(weight_offset), _lib.ptr(out32), cols, None if out is out32 else _lib.ptr(out), cols, rows, cols,
        _lib.DTYPE_CODES[weight.dtype], float(eps), _lib.stream_arg(x32.device)))
    return out32, out


def qkv_norm_mix_write(qkv, q_out, key_blocks, value_blocks, positions, token_to_sequence, block_tables, *,
                       q_heads: int, kv_heads: int, dim: int, value_dim: int, unit_norm: bool = False,
                       eps: float = 0.0, temperature: tuple[float, int] | None = None, v_first=None,
                       lam: float = 0.0, status: torch.Tensor) -> None:
    """Merged projection rows -> normalised, tempered queries in ``q_out`` and normalised keys / mixed values in
    their page slots.  ``temperature`` is (coefficient, period in positions); ``v_first`` the rows whose values
    are blended in with weight ``lam``."""

    coef, every = temperature if temperature is not None else (0.0, 0)
    _lib.check(_lib.load().mie_qkv_norm_mix_write(
        _lib.ptr(qkv), qkv.stride(0), _lib.ptr(v_first), 0 if v_first is None else v_first.stride(0), float(lam),
        int(unit_norm), float(eps), float(coef), int(every), _lib.index_arg(positions),
        _lib.index_arg(token_to_sequence), _lib.index_arg(block_tables), _lib.ptr(q_out),
        _lib.view4_arg(key_blocks), _lib.view4_arg(value_blocks), int(qkv.shape[0]), q_heads, kv_heads, dim, value_dim,
        _lib.DTYPE_CODES[qkv.dtype], int(key_blocks.shape[2]), int(key_blocks.shape[0]), int(block_tables.shape[0]),
        int(block_tables.shape[1]), _lib.ptr(status), _lib.stream_arg(qkv.device)))


def clamped_glu(gate_up, *, limit: float, slope: float, up_offset: float) -> torch.Tensor:
    """g sigmoid(slope g) (u + up_offset) over the two halves of a merged gate / up projection, g clamped from
    above and u from both sides at ``limit``."""

    rows, cols = int(gate_up.shape[0]), int(gate_up.shape[1]) // 2
    out = torch.empty(rows, cols, dtype=gate_up.dtype, device=gate_up.device)
    _lib.check(_lib.load().mie_clamped_glu(
        _lib.ptr(gate_up), _lib.ptr(gate_up[:, cols:]), gate_up.stride(0), _lib.ptr(out), cols, rows, cols,
        _lib.DTYPE_CODES[gate_up.dtype], float(limit), float(slope), float(up_offset),
        _lib.stream_arg(gate_up.device)))
    return out


def residual_norm_(x32, y, y_weight, next_weight=None, *, alpha: float, eps: float, keep_rows: bool = True):
    """``x32 += alpha * rms_norm(y) * y_weight`` in place, then the rows the next product reads, in the weights' dtype:
    ``rms_norm(x32) * next_weight``, or ``x32`` itself without a next weight.  ``keep_rows=False``: only ``x32``."""

    rows, cols = x32.shape
    if next_weight is None and y_weight.dtype == torch.float32:
        out = x32 if keep_rows else None
        target = None
    else:
        out = target = torch.empty(rows, cols, dtype=y_weight.dtype, device=x32.device) if keep_rows else None
    _lib.check(_lib.load().mie_residual_norm(
        _lib.ptr(x32), x32.stride(0), _lib.ptr(y), y.stride(0), _lib.ptr(y_weight), float(alpha),
        _lib.ptr(next_weight), _lib.ptr(target), cols, rows, cols, _lib.DTYPE_CODES[y_weight.dtype], float(eps),
        _lib.stream_arg(x32.device)))
    return out


def gelu(x, *, ids=None, table=None, status: torch.Tensor | None = None) -> torch.Tensor:
    """tanh-form gelu of rows, times the rows ``table[ids]`` (a column slice of a wider table) when given."""

    rows, cols = x.shape
    out = torch.empty(rows, cols, dtype=x.dtype, device=x.device)
    _lib.check(_lib.load().mie_gelu(
        _lib.ptr(x), x.stride(0), _lib.index_arg(ids), _lib.ptr(table), 0 if table is None else table.stride(0),
        0 if table is None else int(table.shape[0]), _lib.ptr(out), cols, rows, cols, _lib.DTYPE_CODES[x.dtype],
        _lib.ptr(status), _lib.stream_arg(x.device)))
    return out


def gated_rms_norm(x, gate, weight, *, eps: float) -> torch.Tensor:
    """rms_norm(x) * weight * sigmoid(gate) over whole rows."""

    rows, cols = x.shape
    out = torch.empty(rows, cols, dtype=x.dtype, device=x.device)
    _lib.check(_lib.load().mie_gated_norm(
        _lib.ptr(x), x.stride(0), _lib.ptr(gate), gate.stride(0), _lib.ptr(weight), _lib.ptr(out), cols, rows, cols,
        _lib.DTYPE_CODES[x.dtype], float(eps), _lib.stream_arg(x.device)))
    return out


def softcap_(logits, cap: float) -> torch.Tensor:
    """cap * tanh(logits / cap) in place on contiguous fp32 logits."""

    _lib.check(_lib.load().mie_softcap(_lib.ptr(logits), logits.numel(), float(cap), _lib.stream_arg(logits.device)))
    return logits


__all__ = ["clamped_glu", "embed_tokens", "gated_rms_norm", "gelu", "qkv_norm_mix_write", "residual_norm_",
           "sinusoid_turns", "softcap_", "sum_rms_norm"]
