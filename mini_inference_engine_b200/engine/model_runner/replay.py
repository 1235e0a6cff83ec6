"""Replaying given tokens through a model's steps and reading logits, without sampling.

``TraceSession`` is the bookkeeping of ``ContinuousBatcher`` without its scheduling: the caller decides which
requests advance by which tokens in a step, and the session gives them pages of the same pool, runs the same
forwards (single tokens of a started request are decode rows, everything else prompt chunks) and takes the pages
back when a request ends.
"""

from __future__ import annotations

from dataclasses import dataclass, field

import torch

from .continuous import PagePool, SlotPool
from .step_runner import PagedStepRunner, eager_step


@dataclass
class _Sequence:
    pages: list[int] = field(default_factory=list)
    length: int = 0
    slot: int | None = None


@dataclass(frozen=True)
class TraceEntry:
    """One request's next tokens, and the places among them whose logits are wanted."""

    rid: object
    tokens: list[int]
    want: list[int]


class TraceSession:
    def __init__(self, runner: PagedStepRunner) -> None:
        self.runner = runner
        self.pool = PagePool(runner.num_pages)
        self.slots = SlotPool(getattr(runner, "num_slots", 0))
        self.sequences: dict[object, _Sequence] = {}

    def _extend(self, rid, count: int) -> _Sequence:
        sequence = self.sequences.get(rid) or _Sequence()
        if sequence.length + count > self.runner.max_context:
            raise ValueError(f"request {rid!r} grows past max_context {self.runner.max_context}")
        if self.slots.size and sequence.slot is None:
            sequence.slot = self.slots.take()
        self.sequences[rid] = sequence
        while len(sequence.pages) * self.runner.shape.page < sequence.length + count:
            self.pool.promise(1)
            sequence.pages.append(self.pool.take())
        return sequence

    def step(self, entries: list[TraceEntry]) -> torch.Tensor | None:
        """Run one step.  Returns fp32 logits ``[wanted, vocab]`` on the host, in the order of the entries and of
        their ``want``, or None when nothing is wanted."""

        if len({e.rid for e in entries}) != len(entries):
            raise ValueError("a request may appear once per step")
        for entry in entries:
            if any(not 0 <= place < len(entry.tokens) for place in entry.want):
                raise ValueError(f"request {entry.rid!r}: a wanted place is outside its tokens")
        active = [e for e in entries if e.tokens]
        if not active:
            return None
        decode, chunks = [], []
        for entry in active:
            sequence = self._extend(entry.rid, len(entry.tokens))
            single = len(entry.tokens) == 1 and sequence.length > 0 and len(decode) < self.runner.max_batch
            (decode if single else chunks).append((entry, sequence))
        starts, cursor = {}, 0
        for entry, _ in (*decode, *chunks):
            starts[entry.rid] = cursor
            cursor += len(entry.tokens)
        wanted = [starts[e.rid] + place for e in active for place in e.want]
        out = eager_step(
            self.runner, [e.tokens[0] for e, _ in decode], [s.length + 1 for _, s in decode], [s.pages for _, s in decode],
            [(e.tokens, s.length, s.pages) for e, s in chunks],
            slots=[s.slot for _, s in (*decode, *chunks)] if self.slots.size else (), logit_rows=wanted or [0],
            return_logits=True)
        for entry, sequence in (*decode, *chunks):
            sequence.length += len(entry.tokens)
        logits = out[1].float().cpu() if wanted else None
        self.runner.check_status()
        return logits

    def end(self, rids) -> None:
        for rid in rids:
            sequence = self.sequences.pop(rid, None)
            if sequence is not None:
                self.pool.give_back(sequence.pages, 0)
                if sequence.slot is not None:
                    self.slots.give_back(sequence.slot)


__all__ = ["TraceEntry", "TraceSession"]
