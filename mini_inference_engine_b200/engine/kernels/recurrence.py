"""Recurrent mixers over per-request state slots (``csrc/linear_recurrence.cu``), and the buffer that holds the slots.

A step hands a mixer its rows in two forms: single tokens (one per request) and packed chunks with ``cu_seqlens``.
``slots`` names each request's state row; a sequence that starts at position 0 starts from zero whatever its slot holds.
"""

from __future__ import annotations

import torch

from ... import _lib

TILE = 64  # tokens the chunked forms advance at a time


class StateBuffer:
    """fp32 state of a model's recurrent layers: one row per slot, a layer's part at a fixed offset of the row, so
    that a request's whole state is one contiguous row."""

    def __init__(self, sizes: list[int], slots: int, device: torch.device) -> None:
        """``sizes``: state floats per slot of every recurrent layer."""

        self.offsets, total = [], 0
        for size in sizes:
            self.offsets.append(total)
            total += -(-size // 4) * 4
        self.rows = torch.zeros(slots, max(total, 4), dtype=torch.float32, device=device)

    def layer(self, index: int) -> torch.Tensor:
        """View of all slots that starts at layer ``index``'s part."""

        return self.rows[:, self.offsets[index]:]

    def copy(self, source: int, target: int) -> None:
        self.rows[target].copy_(self.rows[source])


def segment_tokens(max_query_len: int, lanes: int, sm_count: int = 148) -> int:
    """Tokens per parallel segment of a packed chunk, 0 for one segment per request.  ``lanes`` is how many CTAs run
    without cutting; requests are cut until the GPU has about one CTA per SM to run, in pieces of at least 256 (the
    pieces but the last are gone over twice)."""

    if max_query_len <= 256 or 2 * lanes > sm_count:
        return 0
    pieces = sm_count // max(lanes, 1)
    length = -(-max_query_len // pieces)
    return max(256, -(-length // TILE) * TILE)


def outer_recurrence(rows, out, decay, state, slots, positions, *, heads: int, dim: int, value_dim: int,
                     cu_seqlens=None, max_query_len: int = 1, status: torch.Tensor) -> None:
    """Per head S <- decay S + k v^T, o = S^T q with q, k, v = silu of a merged row [q | k | v]; o to ``out``."""

    tokens, requests = int(rows.shape[0]), 0 if cu_seqlens is None else int(cu_seqlens.shape[0]) - 1
    length, carry = 0, None
    if cu_seqlens is not None and _lib.load().mie_outer_recurrence_chunked(dim, value_dim, _lib.DTYPE_CODES[rows.dtype]):
        length = segment_tokens(max_query_len, requests * heads * -(-value_dim // 128))
        if length and max_query_len > length:
            carry = torch.empty((tokens // length + requests) * heads * dim * value_dim, dtype=torch.float32,
                                device=rows.device)
    _lib.check(_lib.load().mie_outer_recurrence(
        _lib.ptr(rows), rows.stride(0), _lib.ptr(decay), _lib.ptr(out), out.stride(0), _lib.ptr(state), state.stride(0),
        int(state.shape[0]), _lib.index_arg(slots), _lib.index_arg(positions), _lib.index_arg(cu_seqlens), requests,
        length if carry is not None else 0, _lib.ptr(carry), 0 if carry is None else carry.numel(), tokens, heads, dim,
        value_dim, _lib.DTYPE_CODES[rows.dtype], _lib.ptr(status), _lib.stream_arg(rows.device)))


def gated_average(rows, out, z_bias, u_bias, state, slots, positions, *, width: int, cu_seqlens=None,
                  max_query_len: int = 1, status: torch.Tensor) -> None:
    """S <- (1 - z) S + z c element by element, z and c from a merged row [z | u | gate]; S silu(gate) to ``out``."""

    tokens, requests = int(rows.shape[0]), 0 if cu_seqlens is None else int(cu_seqlens.shape[0]) - 1
    length, carry = 0, None
    if cu_seqlens is not None and max_query_len > TILE:
        length = TILE if tokens * width >= 64 * 512 * 296 else TILE // 2  # shorter pieces when they are few
        carry = torch.empty((tokens // length + requests) * 2 * width, dtype=torch.float32, device=rows.device)
    _lib.check(_lib.load().mie_gated_average(
        _lib.ptr(rows), rows.stride(0), _lib.ptr(z_bias), _lib.ptr(u_bias), _lib.ptr(out), out.stride(0),
        _lib.ptr(state), state.stride(0), int(state.shape[0]), _lib.index_arg(slots), _lib.index_arg(positions),
        _lib.index_arg(cu_seqlens), requests, length, _lib.ptr(carry), 0 if carry is None else carry.numel(), tokens,
        width, _lib.DTYPE_CODES[rows.dtype], _lib.ptr(status), _lib.stream_arg(rows.device)))


__all__ = ["StateBuffer", "gated_average", "outer_recurrence", "segment_tokens"]
