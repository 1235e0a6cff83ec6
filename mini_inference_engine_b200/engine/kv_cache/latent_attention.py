"""Attention over a latent cache: a layer caches one row per token, [latent (rank) | rotated key part (rot_dim)], in
pages ``[pages, 1, page, rank + rot_dim]`` that all heads read.

Two ways to attend.  Absorbed: queries are carried into the latent space (q^T W_uk per head), every head attends the
cached rows themselves and the result leaves the latent space through W_uv - ``latent_decode_attention`` (streaming,
bf16) or the row kernel of ``sink_attention`` (any sizes, fp32).  Expanded: the cached rows a packed chunk can see are
gathered (``VisibleSpans``), projected to per-head keys and values, and attended by the tcgen05 prefill kernel.
"""

from __future__ import annotations

import torch

from ... import _lib


def latent_norm_write(rows, q_weight, weight, turns, pages, positions, token_to_sequence, block_tables, *, q_rank: int,
                      rank: int, rot_dim: int, rotated: int, eps: float, status: torch.Tensor) -> torch.Tensor:
    """Merged projection rows [query latent | latent | key part] -> normed query latents (returned) and, unless
    ``pages`` is None, cached rows in their page slots."""

    tokens = int(rows.shape[0])
    out = torch.empty(tokens, q_rank, dtype=rows.dtype, device=rows.device)
    page = (0, 0, 16, 1) if pages is None else (pages.stride(0), pages.stride(2), int(pages.shape[2]), int(pages.shape[0]))
    _lib.check(_lib.load().mie_latent_norm_write(
        _lib.ptr(rows), rows.stride(0), q_rank, rank, rot_dim, rotated, _lib.ptr(q_weight), _lib.ptr(weight),
        _lib.ptr(turns), _lib.ptr(out), q_rank, _lib.ptr(pages), page[0], page[1], _lib.index_arg(positions),
        _lib.index_arg(token_to_sequence), _lib.index_arg(block_tables), tokens, _lib.DTYPE_CODES[rows.dtype], page[2],
        page[3], int(block_tables.shape[0]), int(block_tables.shape[1]), float(eps), _lib.ptr(status),
        _lib.stream_arg(rows.device)))
    return out


def rotate_heads(source, target, positions, turns, rotated: int) -> None:
    """Rotate ``[tokens, heads, rot_dim]`` rows (the first ``rotated`` entries, pairs 2i / 2i + 1) into ``target``, which
    may be ``source``."""

    tokens, heads, rot_dim = (int(n) for n in source.shape)
    _lib.check(_lib.load().mie_rotate_heads(
        _lib.ptr(source), source.stride(0), source.stride(1), _lib.ptr(target), target.stride(0), target.stride(1),
        _lib.index_arg(positions), _lib.ptr(turns), tokens, heads, rot_dim, rotated, _lib.DTYPE_CODES[source.dtype],
        _lib.stream_arg(source.device)))


class VisibleSpans:
    """The cached tokens that the packed chunks of a step see through a window, laid end to end in 16-token pages.

    ``chunk_starts`` (host numbers) sizes the buffer exactly; without them - a captured step - it is sized for chunks
    anywhere in sequences of up to ``max_context`` tokens."""

    def __init__(self, cu_seqlens, kv_lens, *, window: int, tokens: int, max_query_len: int, max_context: int,
                 chunk_starts=None, status: torch.Tensor) -> None:
        requests, device = int(cu_seqlens.shape[0]) - 1, cu_seqlens.device
        behind = min(window - 1, max_context)
        before = [behind] * requests if chunk_starts is None else [min(start, behind) for start in chunk_starts]
        self.rows = -(-(tokens + sum(before) + 30 * requests) // 16) * 16
        self.width = -(-(max_query_len + max(before, default=0) + 30) // 16)
        self.requests, self.kv_lens, self.status = requests, kv_lens, status
        self.spans = torch.empty(2 * requests + 1, dtype=torch.int32, device=device)
        self.lens = torch.empty(requests, dtype=torch.int32, device=device)
        self.table = torch.empty(requests, self.width, dtype=torch.int32, device=device)
        _lib.check(_lib.load().mie_latent_spans(
            _lib.index_arg(cu_seqlens), _lib.index_arg(kv_lens), requests, window, self.width, self.rows,
            1 << 40, _lib.ptr(self.spans), _lib.ptr(self.lens), _lib.ptr(self.table), _lib.ptr(status),
            _lib.stream_arg(device)))

    def gather(self, pages, block_tables) -> torch.Tensor:
        """``[rows, cols]`` cached rows of the spans; rows after the last span are left unset."""

        cols = int(pages.shape[3])
        out = torch.empty(self.rows, cols, dtype=pages.dtype, device=pages.device)
        _lib.check(_lib.load().mie_latent_gather(
            _lib.ptr(pages), pages.stride(0), pages.stride(2), _lib.ptr(self.spans), _lib.index_arg(self.kv_lens),
            _lib.index_arg(block_tables), _lib.ptr(out), self.rows, cols, self.requests, _lib.DTYPE_CODES[pages.dtype],
            int(pages.shape[2]), int(pages.shape[0]), int(block_tables.shape[1]), _lib.ptr(self.status),
            _lib.stream_arg(pages.device)))
        return out

    def pages(self, rows: torch.Tensor, begin: int, heads: int, size: int) -> torch.Tensor:
        """Columns ``begin ... + heads * size`` of rows laid out like the spans, as pages [pages, heads, 16, size]."""

        paged = rows.view(self.rows // 16, 16, rows.shape[1])[..., begin:begin + heads * size]
        return paged.unflatten(-1, (heads, size)).transpose(1, 2)


def latent_decode_supported(dim: int, value_dim: int, page: int, dtype: torch.dtype) -> bool:
    return bool(_lib.load().mie_latent_decode_supported(dim, value_dim, page, _lib.DTYPE_CODES[dtype]))


def latent_decode_scratch(batch: int, heads: int, value_dim: int, max_total_tokens: int,
                          device: torch.device) -> torch.Tensor:
    size = int(_lib.load().mie_latent_decode_scratch_bytes(batch, heads, value_dim, int(max_total_tokens)))
    return torch.empty(size, dtype=torch.uint8, device=device)


def latent_decode_attention(query, out, pages, block_tables, sequence_lengths, *, scale: float,
                            window: int | None = None, sinks=None, scratch: torch.Tensor, use_plan: bool = False,
                            split_policy: int = 1, status: torch.Tensor) -> None:
    """One row per request, ``query [batch, heads, dim]`` over the cached rows, ``out [batch, heads, value_dim]``."""

    batch, heads, dim = (int(n) for n in query.shape)
    _lib.check(_lib.load().mie_latent_decode_attention(
        _lib.ptr(query), query.stride(0), query.stride(1), _lib.ptr(out), out.stride(0), out.stride(1),
        _lib.view4_arg(pages), _lib.index_arg(block_tables), _lib.index_arg(sequence_lengths), batch, heads, dim,
        int(out.shape[2]), int(pages.shape[2]), int(pages.shape[0]), int(block_tables.shape[1]),
        _lib.DTYPE_CODES[query.dtype], float(scale), int(window or 0), _lib.ptr(sinks), split_policy,
        _lib.ptr(scratch), scratch.numel(), int(use_plan), _lib.ptr(status), _lib.stream_arg(query.device)))


__all__ = ["VisibleSpans", "latent_decode_attention", "latent_decode_scratch", "latent_decode_supported",
           "latent_norm_write", "rotate_heads"]
