"""One step's work as the models take it: token rows of several sequences with everything the kernels read beside them.

A step mixes whole prompts, portions of prompts and single decoded tokens.  Rows of a sequence are consecutive and in position
order.  Models whose attention has a form for few rows per sequence and one for many get the few-row sequences first
(``n_rows_form`` rows), the others after them."""
from __future__ import annotations

from dataclasses import dataclass, field
from typing import List, Optional, Sequence

import numpy as np
import torch


@dataclass
class Portion:
    """The next tokens of one sequence: batch row of the cache manager, position of the first token, wanted offsets."""
    row: int
    start: int
    tokens: Sequence[int]
    want: Sequence[int] = ()


@dataclass
class StepBatch:
    T: int
    ids: torch.Tensor                      # int64 [T]
    positions: torch.Tensor                # int32 [T]
    slots: torch.Tensor                    # int64 [T] cache slot of every row
    tables: torch.Tensor                   # int32 [rows, max_blocks]
    ctx: torch.Tensor                      # int32 [T] keys visible to every row
    n_logits: int
    seq_of_row: Optional[torch.Tensor] = None      # int32 [T]; None: row i is sequence i
    logit_rows: Optional[torch.Tensor] = None      # int64 [n_logits]; None: all rows
    out_tokens: Optional[torch.Tensor] = None      # int64: greedy tokens of the logit rows (None: no sampling)
    logits_out: Optional[torch.Tensor] = None      # fp32 [n_logits, vocab]: the logits themselves
    attn_splits: int = 1
    # paged-attention query tiles (ops.prefill_tiles)
    tiles: Optional[torch.Tensor] = None
    # models with carried state: int32 [nseg, 4] (first row, rows, state slot, 0) and the segment of every row (None: identity)
    segs: Optional[torch.Tensor] = None
    seg_of_row: Optional[torch.Tensor] = None
    # the segments cut for chunked recurrences: int32 [n, 4] (first row, rows, state slot, flags: 1 = a group of the segment precedes, 2 = one
    # follows); scan_cut: some segment has several
    scan_groups: Optional[torch.Tensor] = None
    scan_cut: bool = False
    # two-form attention: rows [0, n_rows_form) take the few-row form; the context of the others is expanded
    n_rows_form: int = 0
    dense_tiles: Optional[torch.Tensor] = None     # int32 [n, 4] (first row, rows <= 64, first context row, keys of the first row)
    dense_slots: Optional[torch.Tensor] = None     # int64 [context rows] cache slots, sequence after sequence


def dense_context(first_rows, counts, starts, rows, tables_host: np.ndarray, block_size: int, window: int = 0):
    """(tiles int32 [n, 4], cache slots int64) for the sequences whose context is expanded: tiles of at most 64 query rows, the
    ones that see most keys first (they take longest).  ``window`` > 0: no row looks further back, and what lies before the first visible key's
    group of 64 positions is left out (the context row of a sequence's first token, in the tiles, then lies that far before its rows)."""
    tiles, slots, base = [], [], 0
    for first, n, start, row in zip(first_rows, counts, starts, rows):
        ctx = start + n
        skip = max(0, start + 1 - window) // 64 * 64 if window else 0
        pos = np.arange(skip, ctx, dtype=np.int64)
        slots.append(tables_host[row, pos // block_size].astype(np.int64) * block_size + pos % block_size)
        for k in range(0, n, 64):
            tiles.append((first + k, min(64, n - k), base - skip, start + k + 1))
        base += ctx - skip
    t = np.asarray(tiles, dtype=np.int32).reshape(-1, 4)
    t = t[np.argsort(-(t[:, 3] + t[:, 1]), kind="stable")]
    return t, np.concatenate(slots) if slots else np.zeros(0, dtype=np.int64)


def scan_groups(segs: np.ndarray, group_rows: int) -> np.ndarray:
    """Segments (first row, rows, slot, 0) cut into groups of at most ``group_rows`` rows (a multiple of the recurrences' chunk)."""
    out = []
    for first, n, slot, _ in segs.tolist():
        for at in range(0, n, group_rows):
            out.append((first + at, min(group_rows, n - at), slot, (1 if at else 0) | (2 if at + group_rows < n else 0)))
    return np.asarray(out, dtype=np.int32).reshape(-1, 4)


@dataclass
class HostBatch:
    """Row arrays of a step on the host; ``order`` = index of every portion in the order of the rows."""
    order: List[int]
    ids: np.ndarray
    pos: np.ndarray
    seq: np.ndarray
    slots: np.ndarray
    seg: np.ndarray
    segs: np.ndarray
    want_rows: np.ndarray                  # rows whose logits are wanted, in the order portions were GIVEN
    n_rows_form: int
    dense_tiles: np.ndarray = field(default=None)
    dense_slots: np.ndarray = field(default=None)


def lay_out(parts: Sequence[Portion], tables_host: np.ndarray, block_size: int, rows_form_max: int = 0, window: int = 0) -> HostBatch:
    """numpy throughout: a 4096-row step must not spend milliseconds in Python loops."""
    few = [i for i, p in enumerate(parts) if len(p.tokens) <= rows_form_max]
    many = [i for i, p in enumerate(parts) if len(p.tokens) > rows_form_max]
    order = few + many
    ps = [parts[i] for i in order]
    n = np.array([len(p.tokens) for p in ps], dtype=np.int64)
    total = int(n.sum())
    first = np.cumsum(n) - n
    seg = np.repeat(np.arange(len(ps), dtype=np.int64), n)
    row = np.array([p.row for p in ps], dtype=np.int64)
    start = np.array([p.start for p in ps], dtype=np.int64)
    ids = np.concatenate([np.asarray(p.tokens, dtype=np.int64) for p in ps]) if total else np.zeros(0, dtype=np.int64)
    pos = np.arange(total, dtype=np.int64) - np.repeat(first, n) + np.repeat(start, n)
    seq = row[seg] if total else np.zeros(0, dtype=np.int64)
    slots = tables_host[seq, pos // block_size].astype(np.int64) * block_size + pos % block_size
    first_of = {o: int(f) for o, f in zip(order, first)}
    want = [np.asarray(p.want, dtype=np.int64) + first_of[i] for i, p in enumerate(parts) if len(p.want)]
    segs = np.stack([first, n, row + 1, np.zeros_like(n)], axis=1).astype(np.int32) if len(ps) else np.zeros((0, 4), dtype=np.int32)
    hb = HostBatch(order, ids, pos, seq, slots, seg, segs, np.concatenate(want) if want else np.zeros(0, dtype=np.int64), int(n[: len(few)].sum()))
    k = len(few)
    hb.dense_tiles, hb.dense_slots = dense_context(first[k:].tolist(), n[k:].tolist(), start[k:].tolist(), row[k:].tolist(), tables_host, block_size, window) \
        if rows_form_max > 0 else (None, None)
    return hb
