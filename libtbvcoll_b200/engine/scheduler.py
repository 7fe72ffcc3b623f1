"""Continuous batching over ``Engine.step``: every step carries the next token of each running request and, within the row
budget, portions of the prompts of admitted ones; a request that ends hands its row, blocks and state slot to the next in line.

Admission reserves by arithmetic, not by luck: a request enters only when the pool could hold its whole prompt and all of its
new tokens beside what the running ones may still need, so a running request never has to be evicted."""
from __future__ import annotations

from typing import Dict, List, Optional, Sequence


class _Running:
    __slots__ = ("index", "prompt", "done", "out", "limit")

    def __init__(self, index: int, prompt: Sequence[int], limit: int):
        self.index, self.prompt, self.done, self.out, self.limit = index, list(prompt), 0, [], limit


class Scheduler:
    def __init__(self, engine, step_rows: Optional[int] = None):
        self.engine = engine
        self.step_rows = step_rows or engine.prefill_chunk
        self.steps = 0

    def _blocks(self, r: _Running) -> int:
        return self.engine.bm.blocks_needed(len(r.prompt) + r.limit)

    def run(self, prompts: Sequence[Sequence[int]], max_new_tokens: int, eos_id: Optional[int] = None) -> List[List[int]]:
        eng = self.engine
        eng.requests.end_all()
        eng.bm.release_all()
        pool = eng.bm.num_blocks - 1
        waiting = [_Running(i, p, max_new_tokens) for i, p in enumerate(prompts)]
        for r in waiting:
            if not r.prompt or len(r.prompt) + r.limit > eng.max_seq_len or self._blocks(r) > pool:
                raise ValueError(f"prompt {r.index}: {len(r.prompt)} + {r.limit} tokens do not fit")
        outs: List[List[int]] = [[] for _ in prompts]
        running: Dict[int, _Running] = {}
        while waiting or running:
            while waiting and len(running) < eng.max_batch and sum(map(self._blocks, running.values())) + self._blocks(waiting[0]) <= pool:
                r = waiting.pop(0)
                running[r.index] = r
            entries, sampled, room = [], [], self.step_rows
            for r in running.values():                       # decoding requests first: one row each
                if r.out and room > 0:
                    entries.append((r.index, r.out[-1:], (0,)))
                    sampled.append(r)
                    room -= 1
            for r in running.values():
                if not r.out and room > 0:
                    part = r.prompt[r.done: r.done + room]
                    r.done += len(part)
                    room -= len(part)
                    last = r.done == len(r.prompt)
                    entries.append((r.index, part, (len(part) - 1,) if last else ()))
                    if last:
                        sampled.append(r)
            tokens = eng.step(entries, sample=True)
            self.steps += 1
            for r, t in zip(sampled, tokens):
                r.out.append(t)
                if len(r.out) == r.limit or t == eos_id:
                    eng.requests.end(r.index)
                    outs[r.index] = r.out
                    del running[r.index]
        return outs
