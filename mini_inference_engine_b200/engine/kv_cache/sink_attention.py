"""Paged attention with a sink in the softmax denominator, an optional sliding window and separate key / value
head sizes.

    out = sum_j exp(s_j) v_j / (exp(sink_h) + sum_j exp(s_j)),   s_j = (q . k_j) * scale

over the cached keys j <= position, or only the last ``window`` of them.  ``sinks`` is one fp32 score per query
head (zeros for "one added to the denominator"), or None for a plain softmax.

Three kernels compute it.  ``sink_decode_attention`` (one row per request) and ``sink_prefill_attention`` (packed
chunks) are the streaming bf16 kernels; ``attention_rows`` takes any sizes and fp32 as well.
"""

from __future__ import annotations

import torch

from ... import _lib


def attention_rows(query, out, key_blocks, value_blocks, positions, token_to_sequence, block_tables, *,
                   scale: float, window: int | None = None, sinks=None, status: torch.Tensor) -> None:
    """Independent rows ``[tokens, heads, dim]`` through the one-warp-per-row kernel: any sizes, bf16 or fp32."""

    tokens, heads, dim = (int(n) for n in query.shape)
    if tokens == 0:
        return
    _lib.check(_lib.load().mie_paged_attention_rows(
        _lib.ptr(query), query.stride(0), query.stride(1), _lib.ptr(out), out.stride(0), out.stride(1),
        _lib.view4_arg(key_blocks), _lib.view4_arg(value_blocks), _lib.index_arg(positions),
        _lib.index_arg(token_to_sequence), _lib.index_arg(block_tables), tokens, heads, int(key_blocks.shape[1]), dim,
        int(value_blocks.shape[3]), int(key_blocks.shape[2]), int(key_blocks.shape[0]), int(block_tables.shape[0]),
        int(block_tables.shape[1]), _lib.DTYPE_CODES[query.dtype], float(scale), int(window or 0), _lib.ptr(sinks),
        _lib.ptr(status), _lib.stream_arg(query.device)))


def sink_decode_supported(dim: int, value_dim: int, page: int, dtype: torch.dtype) -> bool:
    return bool(_lib.load().mie_sink_decode_supported(dim, value_dim, page, _lib.DTYPE_CODES[dtype]))


def sink_prefill_supported(heads: int, kv_heads: int, dim: int, value_dim: int, page: int, dtype: torch.dtype,
                           scale: float) -> bool:
    return bool(_lib.load().mie_sink_prefill_supported(heads, kv_heads, dim, value_dim, page, _lib.DTYPE_CODES[dtype],
                                                       float(scale)))


def sink_decode_attention(query, out, key_blocks, value_blocks, block_tables, sequence_lengths, *, scale: float,
                          window: int | None = None, sinks=None, scratch: torch.Tensor, use_plan: bool = False,
                          plan_slot: int = 0, split_policy: int = 1, status: torch.Tensor) -> None:
    """One query row per request (``[batch, heads, dim]``) through the persistent streaming kernel."""

    batch, heads, dim = (int(n) for n in query.shape)
    _lib.check(_lib.load().mie_sink_decode_attention(
        _lib.ptr(query), query.stride(0), query.stride(1), _lib.ptr(out), out.stride(0), out.stride(1),
        _lib.view4_arg(key_blocks), _lib.view4_arg(value_blocks), _lib.index_arg(block_tables),
        _lib.index_arg(sequence_lengths), batch, heads, int(key_blocks.shape[1]), dim, int(value_blocks.shape[3]),
        int(key_blocks.shape[2]), int(key_blocks.shape[0]), int(block_tables.shape[1]),
        _lib.DTYPE_CODES[query.dtype], float(scale), int(window or 0), _lib.ptr(sinks), split_policy,
        _lib.ptr(scratch), scratch.numel() * scratch.element_size(), int(use_plan), plan_slot, _lib.ptr(status),
        _lib.stream_arg(query.device)))


def sink_prefill_attention(query, out, key_blocks, value_blocks, block_tables, cu_seqlens, kv_lens, *,
                           max_query_len: int, scale: float, window: int | None = None, sinks=None,
                           status: torch.Tensor) -> None:
    """Packed prompt chunks (``[tokens, heads, dim]``) through the tcgen05 kernel."""

    tokens, heads, dim = (int(n) for n in query.shape)
    requests = int(cu_seqlens.shape[0]) - 1
    if tokens == 0 or requests <= 0:
        return
    _lib.check(_lib.load().mie_sink_prefill_attention(
        _lib.ptr(query), query.stride(0), query.stride(1), _lib.ptr(out), out.stride(0), out.stride(1),
        _lib.view4_arg(key_blocks), _lib.view4_arg(value_blocks), _lib.index_arg(block_tables),
        _lib.index_arg(cu_seqlens), _lib.index_arg(kv_lens), requests, int(max_query_len), heads,
        int(key_blocks.shape[1]), dim, int(value_blocks.shape[3]), int(key_blocks.shape[2]),
        int(key_blocks.shape[0]), int(block_tables.shape[1]), _lib.DTYPE_CODES[query.dtype], float(scale),
        int(window or 0), _lib.ptr(sinks), _lib.ptr(status), _lib.stream_arg(query.device)))


__all__ = ["attention_rows", "sink_decode_attention", "sink_decode_supported", "sink_prefill_attention",
           "sink_prefill_supported"]
