"""Step machinery shared by the model runners: static buffers, CUDA-graph buckets and generation loops.

A runner owns a pool of request pages followed by scratch pages, and two forwards over it - ``decode_forward``
(one token per row) and ``mixed_forward`` (decode rows and packed prompt chunks in one flat token stream).
``PagedStepRunner`` is everything around those two that does not depend on the model: bucket selection, padding
rows on private scratch pages, capture and replay, packing of host metadata, greedy generation.  A model design
subclasses it with its weights, its cache tensors and the two forwards; ``ContinuousBatcher`` drives any of them.

A design with recurrent layers also keeps a state slot per request: every row of a step then carries the slot of its
request next to its block-table row, and padding rows have private scratch slots.
"""

from __future__ import annotations

import torch

from ... import _lib


# A decode work plan carries 64 work counters, one per attention launch that reuses it; deeper models
# rebuild the plan every 64 layers.
PLAN_SLOTS = 64
LM_HEAD_MAX_ROWS = 256  # rows one mie_lm_head_argmax call takes
DEFAULT_DECODE_BUCKETS = (1, 2, 4, 8, 16, 32, 64, 128, 256)


def select_bucket(rows: int, buckets: tuple[int, ...]) -> int | None:
    """Smallest bucket that holds ``rows`` (reference: engine/serving/decode_graph.py:29-32)."""

    if rows < 1:
        return None
    return next((size for size in buckets if size >= rows), None)


class _Padding:
    """Owner of a row that carries no request."""

    def __repr__(self) -> str:  # pragma: no cover - debugging aid
        return "<padding row>"


PADDING = _Padding()


class DecodeBuffers:
    """Static buffers of one decode-graph bucket (reference: engine/serving/decode_graph.py:36-96): ids,
    lengths (including the new token), block tables and output tokens keep their addresses across replays.

    Rows ``[0, live)`` carry requests, the rest are padding rows: token 0, length 1 and a one-entry table
    pointing at the row's OWN scratch page, so a padding row writes and reads offset 0 of a page no request
    and no other padding row uses.  ``scratch_pages`` must hold ``batch`` distinct page ids.  With ``scratch_slots``
    (as many distinct state slots) the rows carry state slots too.

    Host side.  Ids and lengths (12 bytes a row) are copied whole every step.  The block tables are not:
    a pinned host mirror remembers, per row, who owns it and how many table entries the device already
    holds, and ``pack_rows`` copies only what changed - a whole row when its owner changed, the new tail
    when a request grew into another page, the scratch entry when a row became padding.  Block lists are
    append-only per owner.  The copies are asynchronous reads of the pinned mirror, so the caller must have
    synchronised with the previous step's copies before packing again (reading the step's tokens does).
    """

    def __init__(self, batch: int, table_width: int, device: torch.device, scratch_pages=None,
                 page: int = 16, scratch_slots=None) -> None:
        self.batch, self.table_width, self.page = batch, table_width, page
        self.advance = False  # True when the captured graph feeds its tokens back and bumps the lengths
        self.scratch_pages = None if scratch_pages is None else tuple(int(p) for p in scratch_pages[:batch])
        if self.scratch_pages is not None and (len(self.scratch_pages) != batch
                                               or len(set(self.scratch_pages)) != batch
                                               or min(self.scratch_pages) < 0):
            raise ValueError("each graph row requires a distinct non-negative scratch page")
        self.input_ids = torch.zeros(batch, dtype=torch.int64, device=device)
        self.sequence_lengths = torch.ones(batch, dtype=torch.int32, device=device)
        self.block_tables = torch.full((batch, table_width), -1, dtype=torch.int32, device=device)
        self.output_tokens = torch.zeros(batch, dtype=torch.int64, device=device)
        pin = device.type == "cuda"

        def host(shape, dtype, fill):
            tensor = torch.full(shape, fill, dtype=dtype)
            return tensor.pin_memory() if pin else tensor

        # Host mirrors for the end-to-end path.
        self.host_ids = host((batch,), torch.int64, 0)
        self.host_lengths = host((batch,), torch.int32, 1)
        self.host_tables = host((batch, table_width), torch.int32, -1)
        self.host_tokens = host((batch,), torch.int64, 0)
        self.state_slots = self.host_slots = None
        if scratch_slots is not None:
            self.scratch_slots = torch.tensor([int(n) for n in scratch_slots[:batch]], dtype=torch.int32)
            self.state_slots = self.scratch_slots.clone().to(device)
            self.host_slots = host((batch,), torch.int32, 0)
        self._owners: list[object] = [None] * batch  # None: the device row is in an unknown state
        self._held: list[int] = [0] * batch          # table entries of the row that the device holds
        self.table_bytes_copied = 0                  # running total, for the measurement of the host step
        if self.scratch_pages is not None:
            self.pack_rows((), (), (), ())           # a valid all-padding batch for warm-up and capture

    def pack(self, ids, lengths, tables=None) -> int:
        """Copy one step's host metadata to the device whole (async, pinned). Returns the bytes copied."""

        self.host_ids.copy_(torch.as_tensor(ids, dtype=torch.int64))
        self.host_lengths.copy_(torch.as_tensor(lengths, dtype=torch.int32))
        self.input_ids.copy_(self.host_ids, non_blocking=True)
        self.sequence_lengths.copy_(self.host_lengths, non_blocking=True)
        copied = self.host_ids.numel() * 8 + self.host_lengths.numel() * 4
        if tables is not None:
            self.host_tables.copy_(torch.as_tensor(tables, dtype=torch.int32))
            self.block_tables.copy_(self.host_tables, non_blocking=True)
            copied += self.host_tables.numel() * 4
            self._owners = [None] * self.batch
        return copied

    def pack_rows(self, owners, ids, lengths, block_rows, slots=None) -> int:
        """One step's rows: ``owners[i]`` (any hashable identity of the request in row i), its input token,
        its length INCLUDING the new token, its page ids and (``slots``) its state slot.  Rows beyond
        ``len(owners)`` become padding.  Only table entries that changed since the previous call are copied.  Returns the bytes copied."""

        live = len(owners)
        if not (len(ids) == len(lengths) == len(block_rows) == live) or live > self.batch:
            raise ValueError("real row counts must agree and fit the graph bucket")
        if self.host_slots is not None and live and (slots is None or len(slots) != live):
            raise ValueError("every row of a recurrent model needs a state slot")
        if self.scratch_pages is None and live < self.batch:
            raise ValueError("padding rows need scratch pages")
        page, width = self.page, self.table_width
        # Ids and lengths: two vectorised writes into the pinned mirrors.
        if live:
            self.host_ids[:live] = torch.as_tensor(ids, dtype=torch.int64)
            self.host_lengths[:live] = torch.as_tensor(lengths, dtype=torch.int32)
        if live < self.batch:
            self.host_ids[live:] = 0
            self.host_lengths[live:] = 1
        # Tables: plain Python comparisons per row, tensor writes only for what changed.
        scratch = None
        dirty: list[tuple[int, int, int]] = []  # (row, first entry, end entry)
        owners_now, held = self._owners, self._held
        for row in range(live):
            blocks, length = block_rows[row], int(lengths[row])
            count = len(blocks)
            if length < 1 or count > width or count * page < length:
                raise ValueError("decode position/block row exceeds the fixed graph table capacity")
            previous = owners_now[row]
            same_owner = previous is not None and previous is not PADDING and previous == owners[row]
            first = held[row] if same_owner else 0
            if count == first:
                continue
            if count < first:
                raise ValueError("a request's block list may only grow")
            fresh = [int(b) for b in blocks[first:]]
            if scratch is None:
                scratch = set(self.scratch_pages or ())
            if min(fresh) < 0 or not scratch.isdisjoint(fresh):
                raise ValueError("real rows must use valid blocks disjoint from scratch pages")
            self.host_tables[row, first:count] = torch.tensor(fresh, dtype=torch.int32)
            dirty.append((row, first, count))
            owners_now[row], held[row] = owners[row], count
        for row in range(live, self.batch):
            if owners_now[row] is not PADDING:
                self.host_tables[row, 0] = self.scratch_pages[row]
                dirty.append((row, 0, 1))
                owners_now[row], held[row] = PADDING, 1
        self.input_ids.copy_(self.host_ids, non_blocking=True)
        self.sequence_lengths.copy_(self.host_lengths, non_blocking=True)
        copied = self.batch * 12
        if self.host_slots is not None:
            if live:
                self.host_slots[:live] = torch.as_tensor(slots, dtype=torch.int32)
            self.host_slots[live:] = self.scratch_slots[live:]
            self.state_slots.copy_(self.host_slots, non_blocking=True)
            copied += self.batch * 4
        entries = sum(end - first for _, first, end in dirty)
        if len(dirty) > 32 or entries * 4 > self.host_tables.numel():
            self.block_tables.copy_(self.host_tables, non_blocking=True)
            table_bytes = self.host_tables.numel() * 4
        else:
            for row, first, end in dirty:
                self.block_tables[row, first:end].copy_(self.host_tables[row, first:end], non_blocking=True)
            table_bytes = entries * 4
        self.table_bytes_copied += table_bytes
        return copied + table_bytes


class MixedBuffers:
    """Static buffers of one captured mixed step: ``decode`` decode rows followed by ``chunk`` prompt-chunk
    tokens in one flat stream (reference: engine/kv_cache/mixed.py:44 ``MixedBatchMetadata``, built per step by
    engine/model_runner/qwen3_mixed.py:41-122; here the tensors are fixed so that the step can be replayed).

    Table rows ``[0, decode)`` belong to the decode rows, rows ``[decode, decode + chunks)`` to the prompt
    chunks, the last row to the padding "request" that owns every unused chunk token (its pages are scratch).
    With ``decode_slots`` and ``chunk_slot`` (scratch) every row carries a state slot.
    """

    def __init__(self, decode: int, chunk: int, chunks: int, table_width: int, device: torch.device,
                 decode_scratch: tuple[int, ...], chunk_scratch: tuple[int, ...], page: int,
                 decode_slots: tuple[int, ...] | None = None, chunk_slot: int = 0) -> None:
        self.decode, self.chunk, self.chunks, self.table_width, self.page = decode, chunk, chunks, table_width, page
        pad_pages = -(-chunk // page)  # pages the padding tokens of this bucket can spread over
        if len(decode_scratch) < decode or len(chunk_scratch) < pad_pages:
            raise ValueError("not enough scratch pages for this mixed bucket")
        if pad_pages > table_width:
            raise ValueError(f"a chunk bucket of {chunk} tokens needs block tables at least {pad_pages} pages wide")
        self.decode_scratch, self.chunk_scratch = decode_scratch[:decode], tuple(chunk_scratch[:pad_pages])
        tokens, rows = decode + chunk, decode + chunks + 1
        self.tokens, self.rows = tokens, rows
        pin = device.type == "cuda"

        def pair(shape, dtype):
            host = torch.zeros(shape, dtype=dtype)
            return torch.zeros(shape, dtype=dtype, device=device), (host.pin_memory() if pin else host)

        self.input_ids, self.host_ids = pair((tokens,), torch.int64)
        self.token_to_sequence, self.host_tok2seq = pair((tokens,), torch.int32)
        self.token_positions, self.host_tokpos = pair((tokens,), torch.int32)
        self.block_tables, self.host_tables = pair((rows, table_width), torch.int32)
        self.decode_lengths, self.host_lengths = pair((max(decode, 1),), torch.int32)
        self.cu_seqlens, self.host_cu = pair((chunks + 2,), torch.int32)
        self.kv_lens, self.host_kv = pair((chunks + 1,), torch.int32)
        self.logit_rows, self.host_logit_rows = pair((decode + chunks,), torch.int64)
        self.state_slots = self.host_slots = None
        if decode_slots is not None:
            self.scratch_slots = torch.tensor([*decode_slots[:decode], *[chunk_slot] * (chunks + 1)], dtype=torch.int32)
            self.state_slots, self.host_slots = pair((rows,), torch.int32)
        self.output_tokens = torch.zeros(decode + chunks, dtype=torch.int64, device=device)
        self.host_tokens = torch.zeros(decode + chunks, dtype=torch.int64)
        if pin:
            self.host_tokens = self.host_tokens.pin_memory()
        self.pack([], [], [], [])

    def pack(self, decode_ids, decode_lengths, decode_blocks, chunks, slots=()) -> int:
        """``decode_*``: the live decode rows (token, length including it, page ids).  ``chunks``: a list of
        ``(token ids, start position, page ids)`` with at most ``self.chunks`` entries and ``self.chunk``
        tokens in total.  ``slots``: state slots of the decode rows and then the chunks.  Everything else becomes
        padding.  Returns the bytes copied to the device."""

        live, page = len(decode_ids), self.page
        total = sum(len(c[0]) for c in chunks)
        if live > self.decode or len(chunks) > self.chunks or total > self.chunk:
            raise ValueError("the step does not fit this mixed bucket")
        if self.host_slots is not None and len(slots) != live + len(chunks):
            raise ValueError("every row of a recurrent model needs a state slot")
        ids, seq, pos = self.host_ids, self.host_tok2seq, self.host_tokpos
        tables, lengths = self.host_tables, self.host_lengths
        tables.fill_(-1)
        for row in range(self.decode):
            if row < live:
                blocks, length = decode_blocks[row], int(decode_lengths[row])
                if length < 1 or len(blocks) > self.table_width or len(blocks) * page < length:
                    raise ValueError("decode position/block row exceeds the fixed table capacity")
                ids[row], seq[row], pos[row], lengths[row] = int(decode_ids[row]), row, length - 1, length
                tables[row, :len(blocks)] = torch.tensor([int(b) for b in blocks], dtype=torch.int32)
            else:
                ids[row], seq[row], pos[row], lengths[row] = 0, row, 0, 1
                tables[row, 0] = self.decode_scratch[row]
        cursor = self.decode
        self.host_cu[0] = 0
        for index in range(self.chunks):
            if index < len(chunks):
                tokens, start, blocks = chunks[index]
                count = len(tokens)
                if count < 1 or len(blocks) > self.table_width or len(blocks) * page < start + count:
                    raise ValueError("chunk position/block row exceeds the fixed table capacity")
                ids[cursor:cursor + count] = torch.tensor([int(t) for t in tokens], dtype=torch.int64)
                seq[cursor:cursor + count] = self.decode + index
                pos[cursor:cursor + count] = torch.arange(start, start + count, dtype=torch.int32)
                tables[self.decode + index, :len(blocks)] = torch.tensor([int(b) for b in blocks], dtype=torch.int32)
                self.host_kv[index] = start + count
                cursor += count
                self.host_logit_rows[self.decode + index] = cursor - 1
            else:
                self.host_kv[index] = 0
                self.host_logit_rows[self.decode + index] = 0
            self.host_cu[index + 1] = cursor - self.decode
        padding = self.tokens - cursor
        pad_row = self.decode + self.chunks
        ids[cursor:] = 0
        seq[cursor:] = pad_row
        pos[cursor:] = torch.arange(padding, dtype=torch.int32)
        tables[pad_row, :len(self.chunk_scratch)] = torch.tensor(self.chunk_scratch, dtype=torch.int32)
        self.host_kv[self.chunks] = padding
        self.host_cu[self.chunks + 1] = self.tokens - self.decode
        self.host_logit_rows[:self.decode] = torch.arange(self.decode, dtype=torch.int64)
        copied = 0
        if self.host_slots is not None:
            self.host_slots.copy_(self.scratch_slots)
            for row, slot in enumerate(slots):
                self.host_slots[row if row < live else self.decode + row - live] = int(slot)
            self.state_slots.copy_(self.host_slots, non_blocking=True)
            copied += self.host_slots.numel() * 4
        for device_tensor, host_tensor in ((self.input_ids, ids), (self.token_to_sequence, seq),
                                           (self.token_positions, pos), (self.block_tables, tables),
                                           (self.decode_lengths, lengths), (self.cu_seqlens, self.host_cu),
                                           (self.kv_lens, self.host_kv), (self.logit_rows, self.host_logit_rows)):
            device_tensor.copy_(host_tensor, non_blocking=True)
            copied += host_tensor.numel() * host_tensor.element_size()
        return copied


def eager_step(runner, decode_ids, decode_lengths, decode_blocks, chunks, *, slots=(), logit_rows=None,
               return_logits: bool = False):
    """One step of a runner from host data without a graph.  ``decode_*``: one token per row (id, length
    including it, page ids); ``chunks``: ``(token ids, start position, page ids)``; ``slots``: state slots of the
    decode rows and then the chunks (recurrent runners).  The flat stream is the decode rows followed by the
    chunks; ``logit_rows`` picks rows of it (default: every decode row and each chunk's last row).  Returns what
    the forward returns for those rows."""

    device, live = runner.device, len(decode_ids)
    extra = {"return_logits": True} if return_logits else {}
    if getattr(runner, "recurrent", False):
        if len(slots) != live + len(chunks):
            raise ValueError("every row of a recurrent model needs a state slot")
        extra["state_slots"] = torch.tensor(list(slots), dtype=torch.int32).to(device)
    counts = [len(tokens) for tokens, _, _ in chunks]
    tables = torch.full((live + len(chunks), runner.table_width), -1, dtype=torch.int32)
    for row, pages in enumerate([*decode_blocks, *(pages for _, _, pages in chunks)]):
        tables[row, :len(pages)] = torch.tensor(pages, dtype=torch.int32)
    tables = tables.to(device)
    lengths = torch.tensor(decode_lengths, dtype=torch.int32)
    if not chunks and (logit_rows is None or list(logit_rows) == list(range(live))):
        return runner.decode_forward(torch.tensor(decode_ids, dtype=torch.int64, device=device), lengths.to(device),
                                     tables, **extra)
    flat = torch.tensor([*decode_ids, *(t for tokens, _, _ in chunks for t in tokens)], dtype=torch.int64).to(device)
    tok2seq = torch.cat([torch.arange(live, dtype=torch.int32),
                         *[torch.full((n,), live + i, dtype=torch.int32) for i, n in enumerate(counts)]]).to(device)
    tokpos = torch.cat([lengths - 1, *[torch.arange(start, start + n, dtype=torch.int32)
                                       for (_, start, _), n in zip(chunks, counts)]]).to(device)
    cu = torch.zeros(len(counts) + 1, dtype=torch.int32)
    if counts:
        cu[1:] = torch.tensor(counts, dtype=torch.int32).cumsum(0)
    kv_lens = torch.tensor([start + n for (_, start, _), n in zip(chunks, counts)], dtype=torch.int32).to(device)
    longest = max(counts, default=0)
    if getattr(runner, "wants_chunk_starts", False):
        extra["chunk_starts"] = [start for _, start, _ in chunks]
    if not live and logit_rows is None:
        return runner.prefill_forward(flat, tok2seq, tokpos, tables, cu.to(device), kv_lens, longest, **extra)
    if logit_rows is None:
        rows = torch.cat([torch.arange(live, dtype=torch.int64), live + cu[1:].long() - 1])
    else:
        rows = torch.tensor(logit_rows, dtype=torch.int64)
    return runner.mixed_forward(flat, tok2seq, tokpos, tables, decode_rows=live,
                                decode_lengths=lengths.to(device) if live else None, cu_seqlens=cu.to(device),
                                kv_lens=kv_lens, max_query_len=longest, logit_rows=rows.to(device), **extra)


class PagedStepRunner:
    """Steps over paged per-request state: decode rows, packed prompt chunks or both in one flat forward, eager
    or replayed from CUDA graphs captured per bucket.

    The pool holds ``num_pages`` request pages followed by scratch pages that only padding rows of a captured
    bucket touch (reference: engine/serving/chunked_prefill.py:133-148 - the extra pages are exclusively scratch,
    the request capacity is unchanged): one page per row of the largest decode bucket and enough pages for the
    padding tokens of the largest prompt-chunk bucket.  ``state_slots`` (recurrent designs) is the number of
    requests that can hold a state slot; scratch slots for padding rows follow them in the same way.

    Subclasses provide ``shape`` (with ``page``, the tokens per page), ``decode_forward`` and ``mixed_forward``.
    """

    wants_chunk_starts = False  # whether the mixed forward takes the chunks' start positions as host numbers

    def __init__(self, shape, device: torch.device, *, num_pages: int, max_batch: int, max_context: int,
                 decode_buckets: tuple[int, ...] | None = None, chunk_buckets: tuple[int, ...] = (128, 512),
                 max_chunks: int = 4, state_slots: int = 0) -> None:
        self.shape, self.device = shape, device
        self.num_pages, self.max_batch, self.max_context = num_pages, max_batch, max_context
        if decode_buckets is None:
            decode_buckets = tuple(b for b in DEFAULT_DECODE_BUCKETS if b < max_batch) + (max_batch,)
        if not decode_buckets or tuple(sorted(set(decode_buckets))) != tuple(decode_buckets) or decode_buckets[0] < 1:
            raise ValueError("decode_buckets must be non-empty, strictly increasing positive integers")
        self.decode_buckets = tuple(int(b) for b in decode_buckets)
        self.chunk_buckets = tuple(sorted(int(c) for c in chunk_buckets))
        self.max_chunks = int(max_chunks)
        chunk_scratch = -(-max(self.chunk_buckets, default=0) // shape.page)
        self.decode_scratch_pages = tuple(range(num_pages, num_pages + self.decode_buckets[-1]))
        self.chunk_scratch_pages = tuple(range(num_pages + self.decode_buckets[-1],
                                               num_pages + self.decode_buckets[-1] + chunk_scratch))
        self.total_pages = num_pages + self.decode_buckets[-1] + chunk_scratch
        self.table_width = -(-max_context // shape.page)
        self.num_slots = int(state_slots)
        self.recurrent = self.num_slots > 0
        self.decode_scratch_slots = tuple(range(self.num_slots, self.num_slots + self.decode_buckets[-1]))
        self.chunk_scratch_slot = self.num_slots + self.decode_buckets[-1]
        self.total_slots = self.chunk_scratch_slot + 1 if self.recurrent else 0
        self.status = torch.zeros(1, dtype=torch.int32, device=device)
        # (kind, bucket...) -> (graph, buffers): ("decode", rows, advance) or ("mixed", rows, chunk tokens)
        self._graphs: dict[tuple, tuple[torch.cuda.CUDAGraph, object]] = {}
        self._generation = 0  # distinguishes the rows of successive generate() calls
        self.launches_per_step = 0
        self._lm_keys = torch.zeros(LM_HEAD_MAX_ROWS, dtype=torch.int64, device=device)  # zero between calls

    # -- greedy sampling ---------------------------------------------------------------------------

    @staticmethod
    def can_fuse_lm_head(final: torch.Tensor, head: torch.Tensor) -> bool:
        """Whether ``lm_head_argmax`` takes these rows: bf16, few enough, a width of whole 16-byte groups."""

        return bool(final.dtype == head.dtype == torch.bfloat16 and final.shape[0] <= LM_HEAD_MAX_ROWS
                    and head.shape[1] % 8 == 0 and head.stride(0) % 8 == 0 and head.data_ptr() % 16 == 0)

    def lm_head_argmax(self, final: torch.Tensor, head: torch.Tensor, vocab_start: int = 0,
                       values: torch.Tensor | None = None) -> torch.Tensor:
        """Greedy next tokens of normed hidden rows: the bf16 product with the head and its argmax in one pass
        over the vocabulary that never writes the logits (``mie_lm_head_argmax``)."""

        rows = int(final.shape[0])
        if final.stride(1) != 1 or final.stride(0) % 8 != 0 or final.data_ptr() % 16 != 0:
            final = final.contiguous()
        tokens = torch.empty(rows, dtype=torch.int64, device=self.device)
        _lib.check(_lib.load().mie_lm_head_argmax(
            _lib.ptr(final), final.stride(0), _lib.ptr(head), head.stride(0), rows, head.shape[0], head.shape[1],
            vocab_start, _lib.ptr(self._lm_keys), _lib.ptr(tokens), _lib.ptr(values), _lib.ptr(self.status),
            _lib.stream_arg(self.device)))
        return tokens

    # -- the two forwards of a model -------------------------------------------------------------

    def decode_forward(self, input_ids, sequence_lengths, block_tables, return_logits: bool = False):
        raise NotImplementedError

    def mixed_forward(self, input_ids, token_to_sequence, token_positions, block_tables, *, decode_rows: int,
                      decode_lengths, cu_seqlens, kv_lens, max_query_len: int, logit_rows,
                      return_logits: bool = False):
        raise NotImplementedError

    def prefill_forward(self, input_ids: torch.Tensor, token_to_sequence: torch.Tensor,
                        token_positions: torch.Tensor, block_tables: torch.Tensor, cu_seqlens: torch.Tensor,
                        kv_lens: torch.Tensor, max_query_len: int, return_logits: bool = False, **extra):
        """Flat ``[tokens]`` forward of packed prompt chunks only (reference: engine/model_runner/qwen3_packed.py:29):
        the mixed forward without decode rows; each request's last row is projected to logits.
        Returns the greedy next token of every request ``[requests]``."""

        last_rows = (cu_seqlens[1:].long() - 1).clamp_min(0)
        return self.mixed_forward(input_ids, token_to_sequence, token_positions, block_tables, decode_rows=0,
                                  decode_lengths=None, cu_seqlens=cu_seqlens, kv_lens=kv_lens,
                                  max_query_len=max_query_len, logit_rows=last_rows, return_logits=return_logits,
                                  **extra)

    def generate(self, prompts: list[list[int]], max_new_tokens: int, *, use_graph: bool = True) -> list[list[int]]:
        """Greedy generation for requests that arrive together: one packed
        whole-prompt prefill, then one decode step per new token (a CUDA graph of the bucket that holds the
        batch when ``use_graph``).  Pages are handed out in order from the start of the pool.  Requests that
        arrive and finish at different times go through ``ContinuousBatcher`` instead."""

        shape, device = self.shape, self.device
        batch = len(prompts)
        lengths = [len(p) for p in prompts]
        needed = [-(-(n + max_new_tokens) // shape.page) for n in lengths]
        if sum(needed) > self.num_pages:
            raise ValueError("the KV pool is too small for these requests")
        if max(n + max_new_tokens for n in lengths) > self.max_context:
            raise ValueError("a request is longer than max_context")
        if self.recurrent and batch > self.num_slots:
            raise ValueError("more requests than state slots")
        slots = torch.arange(batch, dtype=torch.int32, device=device) if self.recurrent else None
        extra = {"state_slots": slots} if self.recurrent else {}
        starts = {"chunk_starts": [0] * batch} if self.wants_chunk_starts else {}
        width = self.table_width
        tables = torch.full((batch, width), -1, dtype=torch.int32)
        cursor = 0
        for row, pages in enumerate(needed):
            tables[row, :pages] = torch.arange(cursor, cursor + pages, dtype=torch.int32)
            cursor += pages
        tables_dev = tables.to(device)
        flat = torch.tensor([t for p in prompts for t in p], dtype=torch.int64, device=device)
        tok2seq = torch.cat([torch.full((n,), r, dtype=torch.int32) for r, n in enumerate(lengths)]).to(device)
        tokpos = torch.cat([torch.arange(n, dtype=torch.int32) for n in lengths]).to(device)
        cu = torch.zeros(batch + 1, dtype=torch.int32)
        cu[1:] = torch.tensor(lengths, dtype=torch.int32).cumsum(0)
        kv_lens = torch.tensor(lengths, dtype=torch.int32, device=device)
        bucket = select_bucket(batch, self.decode_buckets) if use_graph and max_new_tokens > 1 else None
        buffers = None
        if bucket is not None:
            # A serving engine captures its buckets once at start-up; capture only touches scratch pages.
            buffers = self.capture(bucket, advance=True)
        next_ids = self.prefill_forward(flat, tok2seq, tokpos, tables_dev, cu.to(device), kv_lens, max(lengths),
                                        **extra, **starts)
        outputs = [[int(t)] for t in next_ids.tolist()]
        current = kv_lens.clone()
        if buffers is not None:
            # The graph feeds its own tokens back, so the steps are queued back to back; every step's tokens
            # are kept on the device and read in one copy at the end (no host round trip between steps).
            # Rows beyond the batch stay padding rows: their length grows with every replay but stays inside
            # their scratch page for up to `page` replays, after which they are reset.
            self._generation += 1
            buffers.pack_rows([(self._generation, row) for row in range(batch)], [0] * batch,
                              [n + 1 for n in lengths],
                              [tables[row, :needed[row]].tolist() for row in range(batch)],
                              list(range(batch)) if self.recurrent else None)
            buffers.input_ids[:batch].copy_(next_ids)
            history = torch.empty(max_new_tokens - 1, batch, dtype=torch.int64, device=device)
            for step in range(max_new_tokens - 1):
                if bucket > batch and step and step % (shape.page - 1) == 0:
                    buffers.sequence_lengths[batch:].fill_(1)
                self.replay(bucket, advance=True)
                history[step].copy_(buffers.output_tokens[:batch])
            for step_tokens in history.tolist():
                for row, token in enumerate(step_tokens):
                    outputs[row].append(int(token))
        else:
            for _ in range(max_new_tokens - 1):
                current = current + 1
                next_ids = self.decode_forward(next_ids, current, tables_dev, **extra)
                for row, token in enumerate(next_ids.tolist()):
                    outputs[row].append(int(token))
        self.check_status()
        return outputs

    # -- CUDA graphs -----------------------------------------------------------------------------

    def capture(self, batch: int, table_width: int | None = None, *, advance: bool = False) -> DecodeBuffers:
        """Capture (once) the decode step for a bucket of ``batch`` rows (reference:
        engine/serving/chunked_prefill.py:231-262).  Warm-up and capture run on an all-padding batch, so
        they only touch scratch pages.  With ``advance`` the graph also feeds the sampled tokens back as the
        next inputs and bumps the lengths, so replays need no host work."""

        key = ("decode", batch, bool(advance))
        if key in self._graphs and (table_width is None or self._graphs[key][1].table_width == table_width):
            return self._graphs[key][1]
        if batch > len(self.decode_scratch_pages):
            raise ValueError(f"bucket {batch} exceeds the largest decode bucket {len(self.decode_scratch_pages)}")
        buffers = DecodeBuffers(batch, table_width or self.table_width, self.device, self.decode_scratch_pages,
                                self.shape.page, self.decode_scratch_slots if self.recurrent else None)
        buffers.advance = advance
        extra = {"state_slots": buffers.state_slots} if self.recurrent else {}
        self._capture(key, buffers, lambda: self.decode_forward(buffers.input_ids, buffers.sequence_lengths,
                                                                buffers.block_tables, **extra), advance)
        return buffers

    def capture_mixed(self, decode: int, chunk: int) -> MixedBuffers:
        """Capture (once) the mixed step for ``decode`` decode rows plus ``chunk`` prompt-chunk tokens."""

        key = ("mixed", decode, chunk)
        if key in self._graphs:
            return self._graphs[key][1]
        buffers = MixedBuffers(decode, chunk, self.max_chunks, self.table_width, self.device,
                               self.decode_scratch_pages, self.chunk_scratch_pages, self.shape.page,
                               self.decode_scratch_slots if self.recurrent else None, self.chunk_scratch_slot)
        extra = {"state_slots": buffers.state_slots} if self.recurrent else {}

        def forward():
            return self.mixed_forward(buffers.input_ids, buffers.token_to_sequence, buffers.token_positions,
                                      buffers.block_tables, decode_rows=decode,
                                      decode_lengths=buffers.decode_lengths if decode else None,
                                      cu_seqlens=buffers.cu_seqlens, kv_lens=buffers.kv_lens, max_query_len=chunk,
                                      logit_rows=buffers.logit_rows, **extra)

        self._capture(key, buffers, forward, False)
        return buffers

    def _capture(self, key, buffers, forward, advance: bool) -> None:
        side = torch.cuda.Stream(device=self.device)
        side.wait_stream(torch.cuda.current_stream(self.device))
        with torch.cuda.stream(side):
            for _ in range(2):
                forward()
        torch.cuda.current_stream(self.device).wait_stream(side)
        torch.cuda.synchronize(self.device)
        graph = torch.cuda.CUDAGraph()
        with torch.cuda.graph(graph):
            tokens = forward()
            buffers.output_tokens.copy_(tokens)
            if advance:
                buffers.input_ids.copy_(tokens)
                buffers.sequence_lengths.add_(1)
        self._graphs[key] = (graph, buffers)

    def replay(self, batch: int, *, advance: bool = False) -> None:
        self._graphs[("decode", batch, bool(advance))][0].replay()

    def step_host(self, batch: int, ids, lengths, tables=None) -> tuple[torch.Tensor, int, int]:
        """End-to-end step from host metadata: H2D, graph replay, D2H of the sampled tokens.
        Returns ``(host tokens, h2d bytes, d2h bytes)``; synchronises the stream."""

        graph, buffers = self._graphs[("decode", batch, False)]
        h2d = buffers.pack(ids, lengths, tables)
        graph.replay()
        buffers.host_tokens.copy_(buffers.output_tokens, non_blocking=True)
        torch.cuda.current_stream(self.device).synchronize()
        return buffers.host_tokens, h2d, buffers.host_tokens.numel() * 8

    def decode_rows(self, owners, ids, lengths, block_rows, slots=None) -> tuple[list[int], int, int]:
        """One decode step for the live rows of a continuous batch: the smallest bucket that holds them is
        captured on first use, the rows are packed (padding rows reset, block tables updated incrementally),
        the bucket's graph is replayed and the live rows' tokens are read back (reference:
        engine/serving/chunked_prefill.py:264-298).  Returns ``(tokens, h2d bytes, d2h bytes)``."""

        live = len(owners)
        bucket = select_bucket(live, self.decode_buckets)
        if bucket is None:
            raise ValueError(f"{live} rows exceed the largest decode bucket {self.decode_buckets[-1]}")
        buffers = self.capture(bucket)
        h2d = buffers.pack_rows(owners, ids, lengths, block_rows, slots)
        self._graphs[("decode", bucket, False)][0].replay()
        buffers.host_tokens[:live].copy_(buffers.output_tokens[:live], non_blocking=True)
        torch.cuda.current_stream(self.device).synchronize()
        return buffers.host_tokens[:live].tolist(), h2d, live * 8

    def mixed_rows(self, decode_ids, decode_lengths, decode_blocks, chunks, slots=()) -> tuple[list[int], list[int]]:
        """One captured mixed step (see ``MixedBuffers.pack``).  Returns the decode rows' tokens and, per
        chunk, the greedy token after its last row (meaningful when the chunk completes its prompt)."""

        live, total = len(decode_ids), sum(len(c[0]) for c in chunks)
        decode = select_bucket(live, self.decode_buckets) if live else 0
        chunk = next((c for c in self.chunk_buckets if c >= total), None)
        if decode is None or chunk is None or len(chunks) > self.max_chunks:
            raise ValueError("the step exceeds the largest mixed bucket")
        buffers = self.capture_mixed(decode, chunk)
        buffers.pack(decode_ids, decode_lengths, decode_blocks, chunks, slots)
        self._graphs[("mixed", decode, chunk)][0].replay()
        buffers.host_tokens.copy_(buffers.output_tokens, non_blocking=True)
        torch.cuda.current_stream(self.device).synchronize()
        tokens = buffers.host_tokens.tolist()
        return tokens[:live], tokens[decode:decode + len(chunks)]

    def release_graphs(self) -> None:
        """Drop every captured graph (they hold pointers into the pools, the exchange and NCCL)."""

        self._graphs.clear()

    def check_status(self) -> None:
        _lib.raise_for_status(self.status)


__all__ = ["DEFAULT_DECODE_BUCKETS", "DecodeBuffers", "LM_HEAD_MAX_ROWS", "MixedBuffers", "PADDING", "PLAN_SLOTS",
           "PagedStepRunner", "eager_step", "select_bucket"]
