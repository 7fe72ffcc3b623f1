"""Block allocator and block tables for the paged KV cache.

The reference's engine lists a "KV cache" without code (reports/11_custom_engine.md:10-20);
in its shipped path the cache is vLLM's.  Here: fixed-size blocks (16 tokens by default), a
free list on the host, and a device-resident block table [max_batch, max_blocks_per_seq]
that the attention kernel reads.  Block 0 is never handed out: idle batch rows and graph
warm-up point at it, so a stray write can never land in a live sequence.
"""
from __future__ import annotations

from typing import Dict, List, NamedTuple

import torch


class BlockManager:
    def __init__(self, num_blocks: int, block_size: int, max_batch: int, max_blocks_per_seq: int, device):
        self.num_blocks, self.block_size = num_blocks, block_size
        self.max_batch, self.max_blocks_per_seq = max_batch, max_blocks_per_seq
        self.free: List[int] = list(range(num_blocks - 1, 0, -1))   # block 0 reserved
        self.tables_host = torch.zeros(max_batch, max_blocks_per_seq, dtype=torch.int32).pin_memory() \
            if torch.cuda.is_available() else torch.zeros(max_batch, max_blocks_per_seq, dtype=torch.int32)
        self.tables = torch.zeros(max_batch, max_blocks_per_seq, dtype=torch.int32, device=device)
        self.owned: List[List[int]] = [[] for _ in range(max_batch)]

    def blocks_needed(self, tokens: int) -> int:
        return (tokens + self.block_size - 1) // self.block_size

    def reserve(self, row: int, tokens: int) -> None:
        """Make sure batch row ``row`` owns blocks for ``tokens`` tokens."""
        need = self.blocks_needed(tokens)
        if need > self.max_blocks_per_seq:
            raise ValueError(f"sequence of {tokens} tokens exceeds max_seq_len")
        have = self.owned[row]
        while len(have) < need:
            if not self.free:
                raise RuntimeError("KV cache is out of blocks")
            b = self.free.pop()
            self.tables_host[row, len(have)] = b
            have.append(b)

    def release(self, row: int) -> None:
        self.free.extend(reversed(self.owned[row]))
        self.owned[row] = []
        self.tables_host[row].zero_()

    def release_all(self) -> None:
        for r in range(self.max_batch):
            if self.owned[r]:
                self.release(r)

    def slot(self, row: int, pos: int) -> int:
        return int(self.tables_host[row, pos // self.block_size]) * self.block_size + pos % self.block_size

    def sync_to_device(self) -> None:
        self.tables.copy_(self.tables_host, non_blocking=True)


class Request(NamedTuple):
    row: int        # batch row: block-table row, and state slot row + 1 in models that carry state (slot 0 is nobody's)
    length: int     # tokens already in the cache / state


class RequestTable:
    """Live requests of ``Engine.step``: a batch row (with its blocks and state slot) from the first entry to the end, however many
    steps lie between.  A row that is given back goes to the end of the line; blocks are handed out as tokens arrive.  What a previous owner left
    in a state slot is never read: a sequence's first token starts from zero."""

    def __init__(self, blocks: BlockManager):
        self.blocks = blocks
        self.free_rows: List[int] = list(range(blocks.max_batch))
        self.live: Dict[object, Request] = {}

    def admit(self, key) -> Request:
        if key not in self.live:
            if not self.free_rows:
                raise RuntimeError(f"more than {self.blocks.max_batch} live requests")
            self.live[key] = Request(self.free_rows.pop(0), 0)
        return self.live[key]

    def extend(self, key, tokens: int) -> Request:
        """Admit if new, make room for ``tokens`` more and count them; returns the request as it was before them."""
        r = self.admit(key)
        self.blocks.reserve(r.row, r.length + tokens)
        self.live[key] = r._replace(length=r.length + tokens)
        return r

    def end(self, key) -> None:
        r = self.live.pop(key, None)
        if r is not None:
            self.blocks.release(r.row)
            self.free_rows.append(r.row)

    def end_all(self) -> None:
        for k in list(self.live):
            self.end(k)
