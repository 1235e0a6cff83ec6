"""Paged attention with a sink in the softmax denominator, an optional sliding window and separate key / value
head sizes.

    out = sum_j exp(s_j) v_j / (exp(sink_h) + sum_j exp(s_j)),   s_j = (q . k_j) * scale

over the cached keys j <= position, or only the last ``window`` of them.  ``sinks`` is one fp32 score per query
head (zeros for "one added to the denominator"), or None for a plain softmax.
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


__all__ = ["attention_rows"]
