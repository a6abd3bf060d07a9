"""Sequences that are fed with given tokens instead of sampled ones: replaying a trace, scoring texts.

They live beside the sampled requests in the scheduler's own memory: a parent row of the block table (which is also the row
of the recurrent state), pages of the shared allocator, and the worker's batch step, the one prompts run through.  A sequence
is admitted with its first tokens, may be left out of steps, and gives everything back when it ends.
"""
from __future__ import annotations

from dataclasses import dataclass
from typing import Dict, Iterable, List, Sequence, Tuple

import torch

from .worker import ExtendItem


@dataclass
class FedSequence:
    row: int
    length: int = 0


class TokenFeeder:
    def __init__(self, sched):
        self.s = sched
        self.live: Dict[str, FedSequence] = {}
        self.held_pages = 0

    def _open(self, rid: str) -> FedSequence:
        s = self.s
        row = s.bt.alloc_parent_row()
        if row is None:
            raise RuntimeError(f"no free sequence row for {rid!r} ({len(self.live)} sequences are live)")
        for pool in (s.state_t, s.state_d):
            if pool is not None:
                pool.clear_rows(torch.tensor([row], device=s.device))
        seq = self.live[rid] = FedSequence(row)
        return seq

    def close(self, rid: str) -> None:
        s, seq = self.s, self.live.pop(rid)
        if seq.length:
            s.alloc.dec_ref_and_free(s.bt.table[seq.row, :seq.length])
        s.bt.free_parent_row(seq.row)
        self.held_pages -= seq.length
        s.reserved_pages -= seq.length

    def step(self, entries: Sequence[Tuple[str, List[int], List[int]]], end: Iterable[str] = ()) -> torch.Tensor:
        """``entries``: (id, next tokens, offsets among them whose logits are wanted), one batch; ``end``: ids whose rows
        and pages are given back after the step.  Returns fp32 logits [wanted, vocab] in the order of the entries."""
        s = self.s
        s._flush_pending()                          # the host changes allocator state here
        if len({rid for rid, _, _ in entries}) != len(entries):
            raise ValueError("a sequence may appear once per step")
        entries = [(rid, list(toks), list(want)) for rid, toks, want in entries]
        for rid, toks, want in entries:
            have = self.live[rid].length if rid in self.live else 0
            if have + len(toks) > s.context_len:
                raise ValueError(f"{rid!r} would exceed the context length ({s.context_len})")
            if any(not 0 <= w < len(toks) for w in want):
                raise ValueError(f"{rid!r}: a wanted offset is outside its tokens")
            if any(not 0 <= t < s.target.cfg.vocab_size for t in toks):
                raise ValueError(f"{rid!r}: a token is outside the vocabulary")
        need = sum(len(t) for _, t, _ in entries)
        if s.reserved_pages + need > s.alloc.size:
            raise RuntimeError(f"{need} more tokens do not fit: {s.alloc.size - s.reserved_pages} of {s.alloc.size} pages are free")
        items = []
        for rid, toks, want in entries:
            seq = self.live.get(rid) or self._open(rid)
            if not toks:
                continue
            pages = s.alloc.alloc(len(toks))
            if pages is None:
                raise RuntimeError("page reservation violated")
            s.bt.table[seq.row, seq.length:seq.length + len(toks)] = pages
            items.append(ExtendItem(seq.row, seq.length, toks, want))
            seq.length += len(toks)
            self.held_pages += len(toks)
            s.reserved_pages += len(toks)
        out = s.worker.extend(items) if items else torch.empty(0, s.target.cfg.vocab_size, device=s.device)
        if s.native_runner is not None:
            status = s.native_runner.check_status()
            if status:
                raise RuntimeError(f"device status {status} in a step of given tokens")
        for rid in end:
            self.close(rid)
        return out
