"""Step plans over sequences of unequal length: portions of prompts beside single decoded tokens.

A plan is what one launch chain runs: tokens back to back, the sequence each belongs to, and the blocks the kernels walk.
``pack_ragged`` cuts a list of portions into plans of at most ``capacity`` tokens (a portion may continue in the next plan;
cache and state carry it on) and uploads each plan in one copy.
"""
from __future__ import annotations

from dataclasses import dataclass
from typing import List, Optional, Sequence, Tuple

import torch

from . import native as K


@dataclass
class Portion:
    """The next tokens of one sequence: block-table / state row, tokens already held, token ids."""
    row: int
    prefix: int
    ids: Sequence[int]


@dataclass
class RaggedPlan:
    T: int
    single: bool                          # every sequence brings exactly one token
    longest: int                          # most tokens any sequence brings
    max_keys: int                         # longest context any token sees
    ids: torch.Tensor
    positions: torch.Tensor
    locs: torch.Tensor
    rows: torch.Tensor                    # [n_seq]
    struct: K.Ragged
    keep: tuple                           # tensors the structure points into
    tokens: List[Tuple[int, int]]         # (portion index, offset inside the portion) of every token, in plan order


def uniform_struct(rows: torch.Tensor, prefix: torch.Tensor, bs: int, E: int, block: int) -> K.Ragged:
    """The list of a uniform batch (bs sequences of E tokens): no index arrays, so it can be captured in a graph."""
    return K.Ragged(seq_row=K.ptr(rows), seq_prefix=K.ptr(prefix), n_seq=bs, n_blk=bs * ((E + block - 1) // block), E=E, B=block)


def pack_ragged(portions: Sequence[Portion], capacity: int, block: int, block_table: torch.Tensor):
    """Yields the plans of ``portions`` one by one (pages must already be in the block table)."""
    dev = block_table.device
    cursor, at = 0, 0                     # portion, offset inside it
    while cursor < len(portions):
        seqs, used = [], 0                # (portion, offset, length)
        while cursor < len(portions) and used < capacity:
            n = min(len(portions[cursor].ids) - at, capacity - used)
            if n > 0:
                seqs.append((cursor, at, n))
                used += n
                at += n
            if at >= len(portions[cursor].ids):
                cursor, at = cursor + 1, 0
        if not seqs:
            continue
        ids, pos, row_of, tokens = [], [], [], []
        seq_cols, blk_seq, blk_start = [], [], []
        off = 0
        for s, (p, o, n) in enumerate(seqs):
            q = portions[p]
            ids += list(q.ids[o:o + n])
            pos += range(q.prefix + o, q.prefix + o + n)
            row_of += [q.row] * n
            tokens += [(p, o + i) for i in range(n)]
            seq_cols.append((q.row, q.prefix + o, off, n))
            for b in range(0, n, block):
                blk_seq.append(s)
                blk_start.append(b)
            off += n
        n_seq, n_blk = len(seqs), len(blk_seq)
        cols = [list(c) for c in zip(*seq_cols)]
        host = torch.tensor(ids + pos + row_of + cols[0] + cols[1] + cols[2] + cols[3] + blk_seq + blk_start, dtype=torch.int32)
        if dev.type == "cuda":
            host = host.pin_memory()
        d = host.to(dev, non_blocking=True)
        t_ids, t_pos, t_row, rows, prefix, soff, slen, bseq, bstart = d.split([off] * 3 + [n_seq] * 4 + [n_blk] * 2)
        locs = block_table[t_row.long(), t_pos.long()].contiguous()
        st = K.Ragged(seq_row=K.ptr(rows), seq_prefix=K.ptr(prefix), seq_off=K.ptr(soff), seq_len=K.ptr(slen), blk_seq=K.ptr(bseq),
                      blk_start=K.ptr(bstart), n_seq=n_seq, n_blk=n_blk, E=0, B=block)
        yield RaggedPlan(off, all(n == 1 for _, _, n in seqs), max(c[3] for c in seq_cols), max(c[1] + c[3] for c in seq_cols), t_ids, t_pos, locs, rows, st,
                         (host, d), tokens)
