"""Greedy TP decode engine: chunked prefill, paged KV cache, decode steps under CUDA graphs.

Counterpart of the reference's undocumented-in-code engine (``engine.py`` / ``run_engine.py``
in reports/11_custom_engine.md:8-23: TP=1/2 decode, greedy, KV cache) and of the vLLM call
its bench makes (``LLM.generate`` with temperature 0 and ``ignore_eos=True``,
step3b/vllm_tp_bench.py:148-171).  The reference measured 6.3-7.8 ms of CPU dispatch per
step in its engine and 28.5 -> 7.1 us for a graph-captured segment (:61-72) but could not
capture its CPU-driven collective (:74); here the whole step, collectives included, is one
graph.

Two decode loops over the same captured step:
  * host loop  — every step copies the step's inputs (token ids, positions, cache slots,
    context lengths) host -> device from pinned memory and reads the sampled tokens back;
    this is what a serving front-end does and what ``generate`` uses by default;
  * device loop — a small kernel inside the graph feeds the sampled token back and advances
    positions/slots, so K steps replay back to back with no host round trip.
"""
from __future__ import annotations

import contextlib
import math
import os
import time
from typing import Dict, List, Optional, Sequence

import numpy as np
import torch

from .. import ops
from ..models.registry import architecture_of
from ..parallel.tp import TPGroup
from ..utils.weights import RandomSource
from .batch import Portion, StepBatch, lay_out, scan_groups
from .kv_cache import BlockManager, RequestTable


def _nvtx(name: str):
    """NVTX range around a phase when TBV_NVTX=1 (the native library marks every collective under the same knob)."""
    if os.environ.get("TBV_NVTX", "0") == "1" and torch.cuda.is_available():
        return torch.cuda.nvtx.range(name)
    return contextlib.nullcontext()


def prefill_rows(prompts: Sequence[Sequence[int]], tables: np.ndarray, block_size: int):
    """Flat per-row arrays over all prompts, rows grouped by sequence in position order:
    (total rows, sequence of row, position, token id, KV-cache slot, is-last-row-of-its-prompt)."""
    hb = lay_out([Portion(b, 0, p, (len(p) - 1,)) for b, p in enumerate(prompts)], tables, block_size)
    is_last = np.zeros(hb.ids.size, dtype=bool)
    is_last[hb.want_rows] = True
    return int(hb.ids.size), hb.seq, hb.pos, hb.ids, hb.slots, is_last


class _GraphChain:
    """Graphs that are always replayed one after the other on the current stream."""

    def __init__(self, graphs):
        self.graphs = list(graphs)

    def replay(self) -> None:
        for g in self.graphs:
            g.replay()


class Engine:
    def __init__(self, cfg, tp: Optional[TPGroup] = None, device="cuda:0", weights: Optional[Dict[str, torch.Tensor]] = None,
                 source=None, seed: int = 0, max_batch: int = 8, max_seq_len: int = 1024, block_size: int = 16,
                 prefill_chunk: int = 2048, max_attn_splits: int = 32, dtype: torch.dtype = torch.bfloat16,
                 max_cache_tokens: Optional[int] = None):
        """``cfg``: a configuration of any registered architecture.  ``max_cache_tokens``: size of the cache pool (default: ``max_batch``
        sequences of ``max_seq_len`` tokens each)."""
        arch = architecture_of(cfg)
        if str(dtype).split(".")[-1] not in arch.dtypes:
            raise ValueError(f"{arch.name} models do not run in {dtype}")
        self.cfg, self.dtype = cfg, dtype
        self.tp = tp or TPGroup()
        self.device = torch.device(device)
        self.max_batch, self.max_seq_len, self.block_size = max_batch, max_seq_len, block_size
        self.prefill_chunk = prefill_chunk
        if weights is None:
            source = source or RandomSource(cfg, seed=seed, device=self.device)
            weights = arch.model().load_weights(cfg, source, self.tp, self.device, dtype)
        max_blocks_per_seq = (max_seq_len + block_size - 1) // block_size
        pool = max_batch * max_blocks_per_seq if max_cache_tokens is None else (max_cache_tokens + block_size - 1) // block_size
        num_blocks = pool + 1          # block 0 is never handed out
        self.bm = BlockManager(num_blocks, block_size, max_batch, max_blocks_per_seq, self.device)
        self.requests = RequestTable(self.bm)
        self.model = arch.model()(cfg, self.tp, weights, self.device, max_tokens=max(prefill_chunk, max_batch), max_batch=max_batch,
                                  num_blocks=num_blocks, block_size=block_size, max_attn_splits=max_attn_splits, dtype=dtype)
        dev, B = self.device, max_batch
        # Static decode inputs (graph-captured addresses): ONE device block and ONE pinned mirror, so that a step's inputs
        # cross PCIe as a single copy:  ids int64[B] | cache slots int64[B] | positions int32[B] | context lengths int32[B]
        self.in_d = torch.zeros(24 * B, dtype=torch.uint8, device=dev)
        self.in_h = torch.zeros(24 * B, dtype=torch.uint8).pin_memory()
        carve = lambda buf: (buf[0:8 * B].view(torch.int64), buf[8 * B:16 * B].view(torch.int64),
                             buf[16 * B:20 * B].view(torch.int32), buf[20 * B:24 * B].view(torch.int32))
        self.ids, self.slots, self.positions, self.ctx = carve(self.in_d)
        self.ids_h, self.slots_h, self.pos_h, self.ctx_h = carve(self.in_h)
        self.ctx.fill_(1)
        self.ctx_h.fill_(1)
        self.out_tokens = torch.zeros(B, dtype=torch.int64, device=dev)
        self.out_h = torch.zeros(B, dtype=torch.int64).pin_memory()
        self.h2d_bytes_per_step, self.d2h_bytes_per_step = 24 * B, 8 * B
        # serving loop: layers in a short first graph of a step (0 = one graph per step, the default: measured 3.327 ms per step
        # with 0, 3.323 / 3.327 / 3.348 with 1 / 2 / 4 head layers on the 8B shape; replaying the graph costs the host 13 us); see capture()
        self.serve_head_layers = int(os.environ.get("TBV_SERVE_HEAD", "0"))
        # one-token segments of a decode step: row i is a sequence whose state slot is i + 1 (idle: the dummy slot 0)
        seg = torch.zeros(B, 4, dtype=torch.int32)
        seg[:, 0], seg[:, 1] = torch.arange(B), 1
        self.idle_segs = seg.to(dev)
        seg[:, 2] = torch.arange(B) + 1
        self.decode_segs = seg.to(dev)
        self.step_counter = torch.zeros(1, dtype=torch.int32, device=dev)
        self.history = torch.zeros(max_seq_len, B, dtype=torch.int64, device=dev)
        # Sequence-parallel prefill (GEMM->reduce-scatter, all-gather->GEMM) for chunks whose row count divides evenly.
        # Off by default: measured slower than the all-reduce path, whose GEMMs are the persistent many-token kernel
        # (8 x 512 tokens, 8B shape, TP=2: 62.7 vs 39.9 ms; 16384 tokens, 70B shape, TP=8: 1623 vs 559 ms).  TBV_SP_PREFILL=1
        # or ``engine.sp_prefill = True`` selects it; both paths produce identical tokens.
        self.sp_prefill = os.environ.get("TBV_SP_PREFILL", "0") == "1"
        self.sp_chunks = 0
        # query-tiled tensor-core attention for prompt rows (TBV_PREFILL_ATTN=rows: one CTA per query row)
        self.tiled_prefill_attention = os.environ.get("TBV_PREFILL_ATTN", "tiled") != "rows"
        self._ids_np, self._pos_np = self.ids_h.numpy(), self.pos_h.numpy()
        self._slots_np, self._ctx_np, self._out_np = self.slots_h.numpy(), self.ctx_h.numpy(), self.out_h.numpy()
        self._tables_np = self.bm.tables_host.numpy()
        self.graphs: Dict[tuple, torch.cuda.CUDAGraph] = {}
        self.launches_per_step = 0
        self.last_stats: Dict[str, float] = {}

    # ---- prefill ----------------------------------------------------------------------------
    def prefill(self, prompts: Sequence[Sequence[int]], reserve_new: int) -> List[int]:
        """Run the prompts through the model in chunks of at most ``prefill_chunk`` token rows
        (a sequence may straddle chunks: attention reads earlier chunks from the cache).
        Returns the first generated token of every sequence."""
        B = len(prompts)
        assert 0 < B <= self.max_batch
        self.requests.end_all()
        self.bm.release_all()
        for b, p in enumerate(prompts):
            if len(p) + reserve_new > self.max_seq_len:
                raise ValueError("prompt + new tokens exceed max_seq_len")
            self.bm.reserve(b, len(p) + reserve_new)
        self.bm.sync_to_device()
        first = [0] * B
        for parts in self._chunks([Portion(b, 0, p, (len(p) - 1,)) for b, p in enumerate(prompts)]):
            rows = [p.row for p in parts if len(p.want)]
            out = torch.zeros(max(len(rows), 1), dtype=torch.int64, device=self.device)
            batch = self.batch_of(parts, out_tokens=out)
            if self.sp_prefill and hasattr(self.model, "sp_ok") and self.model.sp_ok(batch.T):
                sel = batch.logit_rows if rows else torch.zeros(1, dtype=torch.int64, device=self.device)
                self.model.forward_sp(batch.T, batch.ids, batch.positions, batch.slots, self.bm.tables, batch.ctx, batch.seq_of_row, sel,
                                      max(len(rows), 1), out, prefill_tiles=batch.tiles)
                self.sp_chunks += 1
            else:
                self.model.forward_batch(batch)
            if rows:
                for b, t in zip(rows, out[: len(rows)].tolist()):
                    first[b] = t
        return first

    def _chunks(self, parts: Sequence[Portion]):
        """The portions cut into passes of at most ``prefill_chunk`` rows (a sequence may straddle passes)."""
        cur, room = [], self.prefill_chunk
        for p in parts:
            n, at = len(p.tokens), 0
            while at < n:
                k = min(room, n - at)
                cur.append(Portion(p.row, p.start + at, p.tokens[at:at + k], tuple(w - at for w in p.want if at <= w < at + k)))
                at += k
                room -= k
                if room == 0:
                    yield cur
                    cur, room = [], self.prefill_chunk
        if cur:
            yield cur

    def batch_of(self, parts: Sequence[Portion], out_tokens: Optional[torch.Tensor] = None, logits_out: Optional[torch.Tensor] = None) -> StepBatch:
        """Device arrays of one pass over ``parts`` (blocks reserved, tables on the device)."""
        m, dev = self.model, self.device
        hb = lay_out(parts, self._tables_np, self.block_size, m.rows_form_max, getattr(m, "context_window", 0))
        put = lambda a, dt: torch.from_numpy(np.ascontiguousarray(a.astype(dt, copy=False))).to(dev)
        T = int(hb.ids.size)
        b = StepBatch(T=T, ids=put(hb.ids, np.int64), positions=put(hb.pos, np.int32), slots=put(hb.slots, np.int64), tables=self.bm.tables,
                      ctx=put(hb.pos + 1, np.int32), n_logits=int(hb.want_rows.size), seq_of_row=put(hb.seq, np.int32),
                      logit_rows=put(hb.want_rows, np.int64), out_tokens=out_tokens, logits_out=logits_out, n_rows_form=hb.n_rows_form)
        if m.uses_state:
            b.segs = put(hb.segs, np.int32)
            if T > len(hb.segs):                   # otherwise one row per sequence: the models' one-token forms
                b.seg_of_row = put(hb.seg, np.int32)
                rows = m.scan_group_rows(hb.segs[:, 1])
                if rows:
                    groups = scan_groups(hb.segs, rows)
                    b.scan_groups, b.scan_cut = put(groups, np.int32), len(groups) > len(hb.segs)
        if m.rows_form_max:
            if hb.n_rows_form:
                b.attn_splits = self.attn_splits_for(hb.n_rows_form, int(hb.pos[: hb.n_rows_form].max()) + 1)
            if hb.n_rows_form < T:
                b.dense_tiles = put(hb.dense_tiles, np.int32)
                if m.expands_context:
                    b.dense_slots = put(hb.dense_slots, np.int64)
        elif self.tiled_prefill_attention:
            b.tiles = ops.prefill_tiles(torch.from_numpy(hb.seq.astype(np.int32)), m.nq // m.nkv).to(dev)
        return b

    # ---- one mixed step ---------------------------------------------------------------------------
    def step(self, entries, end=(), sample: bool = False):
        """One step over live requests: ``entries`` = (request id, next tokens, wanted offsets among them) per request — whole prompts,
        portions of prompts and single tokens side by side.  A request is admitted at its first entry and keeps its row, blocks and
        state until it is named in ``end`` (given back after this step).  Returns the fp32 logits [wanted, vocab] in the order of
        the entries and offsets, or the greedy tokens (list) with ``sample``.  ``generate`` resets the same cache: do not mix the two
        while requests are live."""
        parts, n = [], 0
        for key, tokens, want in entries:
            r = self.requests.extend(key, len(tokens))
            parts.append(Portion(r.row, r.length, list(tokens), tuple(want)))
            n += len(want)
        self.bm.sync_to_device()
        out = torch.empty(n, dtype=torch.int64, device=self.device) if sample else \
            torch.empty(n, self.cfg.vocab_size, dtype=torch.float32, device=self.device)
        at = 0
        for piece in self._chunks(parts):
            k = sum(len(p.want) for p in piece)
            self.model.forward_batch(self.batch_of(piece, **{"out_tokens" if sample else "logits_out": out[at: at + k]}))
            at += k
        for key in end:
            self.requests.end(key)
        if ops.gemm_error():
            raise RuntimeError("a GEMM barrier wait gave up on the device (see the kernel's watchdog)")
        return out.tolist() if sample else out

    # ---- decode -------------------------------------------------------------------------------
    def _decode_step(self, B: int, splits: int, advance: bool, layer_begin: int = 0, layer_end: Optional[int] = None, idle: bool = False) -> None:
        """One token per row.  ``idle``: a warm-up pass that must leave no trace — the cache rows it writes are written again
        by the real step, and carried state goes to the dummy slot."""
        self.model.forward_batch(StepBatch(T=B, ids=self.ids[:B], positions=self.positions[:B], slots=self.slots[:B], tables=self.bm.tables,
                                           ctx=self.ctx[:B], n_logits=B, out_tokens=self.out_tokens, attn_splits=splits, n_rows_form=B,
                                           segs=(self.idle_segs if idle else self.decode_segs)[:B]),
                                 layer_begin=layer_begin, layer_end=layer_end)
        if advance and (layer_end is None or layer_end == self.cfg.num_layers):
            ops.decode_advance(self.out_tokens[:B], self.ids[:B], self.positions[:B], self.ctx[:B], self.slots[:B], self.bm.tables,
                               self.block_size, self.history, self.step_counter)

    def attn_splits_for(self, B: int, max_ctx: int) -> int:
        sms = torch.cuda.get_device_properties(self.device).multi_processor_count
        # kv splits are the CTAs of one cluster: the largest power of two (<= 8) that keeps the whole
        # grid in one wave and leaves at least 64 cached tokens per CTA
        s = 1
        while s < 8 and B * self.model.attn_ctas_per_row * s * 2 <= self.model.attn_cta_slots(s * 2, sms) and max_ctx // (s * 2) >= 64:
            s *= 2
        return min(s, self.model.max_attn_splits)

    def capture(self, B: int, splits: int, advance: bool, io: bool = False):
        """Capture one decode step (all layers, both collectives per layer, sampling) as a graph.  ``io=True`` is the
        serving form: the step starts with the copy of the packed inputs from pinned memory and ends with the copy of
        the sampled tokens back to pinned memory, so that a step costs the host one graph launch.  With
        ``serve_head_layers`` > 0 it is captured as TWO graphs, a short head (copy in, embedding, the first layers) and
        the rest, so that the launch of the long tail overlaps the head's execution (the host cannot launch a step
        before it has read the previous step's tokens).  The returned object has ``replay()``."""
        key = (B, splits, advance, io)
        if key in self.graphs:
            return self.graphs[key]
        L = self.cfg.num_layers
        head = min(max(0, self.serve_head_layers), L) if io else 0
        s = torch.cuda.Stream(device=self.device)
        s.wait_stream(torch.cuda.current_stream(self.device))
        parts = []
        with torch.cuda.stream(s):
            self._decode_step(B, splits, False, idle=True)      # eager warm-up: leaves no trace (no advance)
            s.synchronize()
            n0 = ops.launch_count + self.tp.launches
            for lo, hi in ([(0, head), (head, L)] if 0 < head < L else [(0, L)]):
                g = torch.cuda.CUDAGraph()
                with torch.cuda.graph(g, stream=s):
                    if io and lo == 0:
                        ops.copy_async(self.in_d, self.in_h)
                    self._decode_step(B, splits, advance, lo, hi)
                    if io and hi == L:
                        ops.copy_async(self.out_h, self.out_tokens)
                parts.append(g)
            self.launches_per_step = ops.launch_count + self.tp.launches - n0
        torch.cuda.current_stream(self.device).wait_stream(s)
        self.graphs[key] = parts[0] if len(parts) == 1 else _GraphChain(parts)
        return self.graphs[key]

    def _load_decode_inputs(self, B: int, tokens, lens) -> None:
        """Stage one step's inputs in pinned memory (vectorised on the numpy views of the pinned
        tensors) and copy them to the device: the fed token of row b sits at position lens[b]."""
        import numpy as np
        pos = np.asarray(lens, dtype=np.int64)[:B]
        self._ids_np[:B] = np.asarray(tokens, dtype=np.int64)[:B]
        self._pos_np[:B] = pos
        self._ctx_np[:B] = pos + 1
        bs = self.block_size
        self._slots_np[:B] = self._tables_np[np.arange(B), pos // bs].astype(np.int64) * bs + pos % bs
        ops.copy_async(self.in_d, self.in_h)

    def generate(self, prompts: Sequence[Sequence[int]], max_new_tokens: int, loop: str = "host", use_graph: bool = True,
                 eos_id: Optional[int] = None) -> List[List[int]]:
        """Greedy generation.  ``loop="host"``: per-step H2D inputs + D2H tokens (serving shape);
        ``loop="device"``: steps chained on the device, tokens read back once at the end.
        EOS is ignored unless ``eos_id`` is given (the reference bench sets ignore_eos).  More prompts than ``max_batch`` go
        through the scheduler, which admits them as rows and cache blocks become free."""
        B = len(prompts)
        if B > self.max_batch:
            from .scheduler import Scheduler
            return Scheduler(self).run(prompts, max_new_tokens, eos_id)
        t0 = time.perf_counter()
        with _nvtx("tbv.prefill"):
            first = self.prefill(prompts, max_new_tokens)
            torch.cuda.synchronize(self.device)
        t1 = time.perf_counter()
        outs = [[t] for t in first]
        lens = [len(p) for p in prompts]      # tokens already in the cache per row
        steps = max_new_tokens - 1
        if steps <= 0:
            return outs
        splits = self.attn_splits_for(B, max(lens) + max_new_tokens)
        if loop == "device":
            self._load_decode_inputs(B, first, lens)
            self.step_counter.zero_()
            g = self.capture(B, splits, True) if use_graph else None
            for _ in range(steps):
                if g is not None:
                    g.replay()
                else:
                    self._decode_step(B, splits, True)
            torch.cuda.synchronize(self.device)
            hist = self.history.view(-1)[: steps * B].view(steps, B).cpu()   # the kernel logs rows of B tokens
            for b in range(B):
                outs[b].extend(hist[:, b].tolist())
        else:
            # Serving shape: every step copies its inputs from pinned memory to the device and reads the sampled tokens
            # back.  Positions, cache slots and context lengths of all steps are laid out before the loop (they do not
            # depend on what is sampled); a step then costs the host four small array writes, one graph launch (copy in,
            # the step's kernels, copy out) and one stream synchronisation.
            import numpy as np
            g = self.capture(B, splits, False, io=True) if use_graph else None
            cur = np.asarray(first, dtype=np.int64)
            bs = self.block_size
            pos_all = np.asarray(lens, dtype=np.int64)[None, :] + np.arange(steps, dtype=np.int64)[:, None]      # [steps, B]
            slots_all = self._tables_np[np.arange(B)[None, :], pos_all // bs].astype(np.int64) * bs + pos_all % bs
            pos32, ctx32 = pos_all.astype(np.int32), (pos_all + 1).astype(np.int32)
            ids_np, slots_np, pos_np, ctx_np, out_np = self._ids_np, self._slots_np, self._pos_np, self._ctx_np, self._out_np
            done = np.zeros(B, dtype=bool)
            trace = []
            sync = torch.cuda.current_stream(self.device).synchronize
            for i in range(steps):
                ids_np[:B] = cur
                slots_np[:B] = slots_all[i]
                pos_np[:B] = pos32[i]
                ctx_np[:B] = ctx32[i]
                if g is not None:
                    g.replay()
                else:
                    ops.copy_async(self.in_d, self.in_h)
                    self._decode_step(B, splits, False)
                    ops.copy_async(self.out_h, self.out_tokens)
                sync()
                cur = out_np[:B].copy()
                trace.append((cur, done.copy()))
                if eos_id is not None:
                    done |= cur == eos_id
                    if done.all():
                        break
            for tok, was_done in trace:
                for b in range(B):
                    if not was_done[b]:
                        outs[b].append(int(tok[b]))
        t2 = time.perf_counter()
        self.last_stats = {"prefill_s": t1 - t0, "decode_s": t2 - t1, "decode_steps": steps, "batch": B,
                           "decode_tok_s": B * steps / max(t2 - t1, 1e-9), "attn_splits": splits,
                           "launches_per_step": self.launches_per_step}
        if ops.gemm_error():
            raise RuntimeError("a GEMM barrier wait gave up on the device (see the kernel's watchdog)")
        return outs
