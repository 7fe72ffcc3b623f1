"""Bobarax decoder: lightning (fixed-decay matrix state), chunked and windowed attention layers, each with a norm before and behind its sublayers; dense ReLU-
gated feed-forwards or mixtures of experts that a table picks by token id; the embedding as output head.

What lies between two sublayers is ONE kernel (``ops.residual`` with ``post``: norm of the branch, residual sum, next norm, and where a mixture of experts
follows, the rows on their places).  The places of all mixtures are laid out by one launch at the start of the step, since they depend on the ids alone.

    lightning   q, k, v, gate GEMM (SiLU on q, k, v) -> recurrence with weight and gate -> out-projection GEMM (fp32); the joint norm of the heads is one factor
                per token, which the kernel behind it applies
    attention   q, k, v, gate GEMM -> norms over whole projections, rotation, cache write -> rows kernel over the cache (few rows) or tiled kernel (many), both
                with window or chunks and the gate -> out-projection GEMM (fp32)
    dense       gate / up GEMM -> down GEMM (fp32)
    experts     gate / up GEMM over each expert's rows -> down GEMM

A layer that takes its keys and values from another reads that layer's cache.  ``dtype`` float32 runs the same sequence with 32-bit weights, activations and
products (rows kernel for every row).  All buffers of a decode step are preallocated, so the step can be captured in a CUDA graph."""
from __future__ import annotations

import os
from typing import Callable, Dict, Optional

import torch

from .. import ops
from ..engine.batch import StepBatch
from ..parallel.tp import TPGroup
from .config import BobaraxConfig, GatedMlpSpec, LightningSpec, PairedAttentionSpec, TableMoeSpec
from .decoder import StreamDecoder, pad16


class Bobarax(StreamDecoder):
    SCAN_CHUNK = 32

    def __init__(self, cfg: BobaraxConfig, tp: TPGroup, weights: Dict[str, torch.Tensor], device, max_tokens: int, max_batch: int,
                 num_blocks: int, block_size: int = 16, max_attn_splits: int = 8, dtype: torch.dtype = torch.bfloat16):
        cfg.check_tp(tp.world)
        self.cfg, self.w, self.device, self.dtype = cfg, weights, torch.device(device), dtype
        self.block_size, self.num_blocks, self.max_tokens, self.max_batch, self.max_attn_splits = block_size, num_blocks, max_tokens, max_batch, max_attn_splits
        dev, f32, i32, T = self.device, torch.float32, torch.int32, max_tokens
        self.W, self.Wp = cfg.hidden_size, pad16(cfg.hidden_size)
        zeros = lambda *shape, dt=dtype: torch.zeros(*shape, dtype=dt, device=dev)
        big = lambda sizes: max(sizes, default=0)
        mixers = [l.mixer for l in cfg.layers]
        lights = [m for m in mixers if isinstance(m, LightningSpec)]
        attns = [m for m in mixers if isinstance(m, PairedAttentionSpec)]
        dense = [l.mlp for l in cfg.layers if isinstance(l.mlp, GatedMlpSpec)]
        moes = [(i, l.mlp) for i, l in enumerate(cfg.layers) if isinstance(l.mlp, TableMoeSpec)]
        # activations; layers of different sizes share flat storage (row prefixes of these are what every call uses)
        self.x, self.y = zeros(T, self.Wp, dt=f32), zeros(T, self.Wp, dt=f32)
        self.h = zeros(T, self.Wp)
        sums = [ops.fixed_decay_sums(m.heads, pad16(m.vdim), dtype) for m in lights]
        self._flat = {
            "wide": zeros(T * big([self.w[f"l{i}.mix.in"].shape[0] for i in range(len(mixers))])),
            "mid": zeros(T * big([m.heads * pad16(m.vdim) for m in mixers])),
            "o": zeros(T * big([m.heads * pad16(m.vdim) for m in lights]) if dtype is f32 else 0, dt=f32),
            "sums": zeros(T * big(sums + [m.heads for m in lights]), dt=f32),
            "qa": zeros(T * big([m.heads * ops.latent_row(pad16(m.dim), 0) for m in attns])),
            "act": zeros(T * big([pad16(f.ff) for f in dense] + [f.top * pad16(f.ff) for _, f in moes])),
            "xp": zeros(T * big([f.top * self.Wp for _, f in moes])),
            "routed": zeros(T * big([f.top * self.Wp for _, f in moes])),
        }
        # places of every mixture of experts, filled for the whole model at once
        self.place = {i: zeros(T * f.top, dt=i32) for i, f in moes}
        self.offsets = {i: zeros(f.experts + 1, dt=i32) for i, f in moes}
        self.max_experts = big([f.experts for _, f in moes])
        self.tables = ops.moe_table_layers([(self.w[f"l{i}.mlp.table"], self.place[i], self.offsets[i], f.experts) for i, f in moes], dev) if moes else None
        self._init_head()
        # cache and state of every layer (slot 0 of the state is never a sequence's); a layer that takes another's keys and values has its cache
        self.cache, self.state, self.powers, self.turns = [], [], [], []
        for m in mixers:
            light = isinstance(m, LightningSpec)
            self.state.append(zeros(max_batch + 1, m.heads, pad16(m.dim), pad16(m.vdim), dt=f32) if light else None)
            self.powers.append(ops.decay_powers(m.decay, dev) if light else None)
            self.turns.append(None if light or m.rot is None or not m.rot.dims else ops.rotation_turns(m.rot.dims, m.rot.base, dev))
            if light:
                self.cache.append(None)
            elif m.kv_from is not None:
                self.cache.append(self.cache[m.kv_from])
            else:
                self.cache.append(zeros(num_blocks * m.kv_heads * block_size, ops.latent_row(pad16(m.dim), pad16(m.vdim))))
        self.attn_ctas_per_row = max([m.kv_heads * ((m.heads // m.kv_heads + 15) // 16) for m in attns], default=1)
        self.scan_heads = min([m.heads for m in lights], default=0)
        self._groups = 0
        two_forms = bool(attns) and dtype is torch.bfloat16 and all(ops.paired_prefill_fits(pad16(m.dim), pad16(m.vdim)) for m in attns)
        self.rows_form_max = self.ROWS_FORM_MAX if two_forms else 1 << 60
        self.l2_prefetch = os.environ.get("TBV_L2_PREFETCH", "1") != "0"

    @staticmethod
    def load_weights(cfg: BobaraxConfig, source, tp: TPGroup, device, dtype):
        from ..utils.weights import load_bobarax
        return load_bobarax(cfg, source, device, dtype)

    def _group_scratch(self, groups: int) -> torch.Tensor:
        """States of the groups of cut segments, grown on demand (never inside a captured step)."""
        if groups > self._groups:
            size = max(s[0].numel() for s in self.state if s is not None)
            self._flat["starts"] = torch.empty(groups * size, dtype=torch.float32, device=self.device)
            self._groups = groups
        return self._flat["starts"]

    @staticmethod
    def layer_splits(m: PairedAttentionSpec, splits: int) -> int:
        """CTAs per row of a layer whose rows see at most a window or chunk: at least 64 keys each."""
        seen = m.window or m.chunk
        while splits > 1 and seen and seen // splits < 64:
            splits //= 2
        return splits

    # -- sublayers ---------------------------------------------------------------------------------------
    def _lightning(self, b: StepBatch, i: int, m: LightningSpec) -> dict:
        w, p, T = self.w, f"l{i}.mix.", b.T
        K, V = m.heads * pad16(m.dim), m.heads * pad16(m.vdim)
        wide, out = self._buf("wide", T, 2 * K + 2 * V), self._buf("mid", T, V)
        one = b.seg_of_row is None
        sums = self._buf("sums", T, m.heads if one else ops.fixed_decay_sums(m.heads, pad16(m.vdim), self.dtype))
        ops.linear(self.h[:T], w[p + "in"], wide, act=ops.ACT_SILU, act_cols=2 * K + V)
        args = (*wide.split((K, K, V, V), 1), w[p + "norm"], self.powers[i], self.state[i], out, sums, b.segs, b.positions)
        if one:
            ops.fixed_decay_step(*args)
        else:
            ops.fixed_decay_scan(*args, groups=b.scan_groups, scratch=self._group_scratch(b.scan_groups.shape[0]) if b.scan_cut else None,
                                 o=self._buf("o", T, V) if self.dtype is torch.float32 else None)
        self._announce(i, T)
        ops.linear(out, w[p + "o"], self.y[:T])
        return dict(y1=self.y[:T], sums=(sums, m.heads * m.vdim))

    def _attention(self, b: StepBatch, i: int, m: PairedAttentionSpec) -> dict:
        w, p, T, n = self.w, f"l{i}.mix.", b.T, b.n_rows_form
        H, D, V, own = m.heads, pad16(m.dim), pad16(m.vdim), m.kv_from is None
        G = m.kv_heads
        at = H * D + (G * (D + V) if own else 0)
        wide, out, qa = self._buf("wide", T, at + (H * V if m.gated else 0)), self._buf("mid", T, H * V), self._buf("qa", n, H, ops.latent_row(D, 0))
        cache, cap, gate = self.cache[i], m.softcap or 0.0, wide[:, at:] if m.gated else None
        ops.linear(self.h[:T], w[p + "in"], wide)
        ops.paired_attention_prep(wide, qa, cache if own else None, w[p + "q.norm"], w[p + "k.norm"] if own else None, self.turns[i], b.positions, b.slots, n, H,
                                  G if own else 0, m.dim, self.block_size, self.cfg.rms_eps)
        if n:
            ops.paired_attention_rows(qa, cache, b.tables, b.seq_of_row, b.ctx, out[:n].view(n, H, V), G, self.block_size, cap, m.window, m.chunk,
                                      None if gate is None else gate[:n], splits=self.layer_splits(m, b.attn_splits))
        if n < T:
            ops.paired_attention_prefill(wide, cache, b.tables, b.seq_of_row, b.dense_tiles, out, H, G, D, self.block_size, cap, m.window, m.chunk, gate)
        self._announce(i, T)
        ops.linear(out, w[p + "o"], self.y[:T])
        return dict(y1=self.y[:T])

    def _announce(self, i: int, T: int) -> None:
        """Decode: the out-projection asks for the gate / up weights that follow it (ops.prefetch_next)."""
        if self.l2_prefetch and T <= 64 and isinstance(self.cfg.layers[i].mlp, GatedMlpSpec) and self.dtype is torch.bfloat16:
            ops.prefetch_next(self.w[f"l{i}.mlp.gate_up"])

    def _dense(self, b: StepBatch, i: int, f: GatedMlpSpec) -> dict:
        p, act = f"l{i}.mlp.", self._buf("act", b.T, pad16(f.ff))
        ops.linear(self.h[: b.T], self.w[p + "gate_up"], act, glu=ops.RELU_GLU)
        ops.linear(act, self.w[p + "down"], self.y[: b.T])
        return dict(y1=self.y[: b.T])

    def _experts(self, b: StepBatch, i: int, f: TableMoeSpec) -> dict:
        w, p, T, P = self.w, f"l{i}.mlp.", b.T, b.T * f.top
        xp, act, routed = self._buf("xp", P, self.Wp), self._buf("act", P, pad16(f.ff)), self._buf("routed", P, self.Wp)
        ops.linear_rows(xp, w[p + "gate_up"], act, self.offsets[i], f.experts, T, glu=(f.limit, f.slope, 1.0))
        ops.linear_rows(act, w[p + "down"], routed, self.offsets[i], f.experts, T)
        return dict(routed=(routed, self.place[i][:P].view(T, f.top), 1.0 / f.top))

    # -- between sublayers -------------------------------------------------------------------------------
    def _norm(self, b: StepBatch, weight: str, experts_of: Optional[int] = None, **terms) -> None:
        """The residual stream takes ``terms``; its norm goes to the next sublayer's input, the mixture of experts of layer ``experts_of`` or ``h``."""
        h, T = self.h[: b.T], b.T
        if experts_of is not None:
            top = self.cfg.layers[experts_of].mlp.top
            h, terms["place"] = self._buf("xp", T * top, self.Wp), self.place[experts_of][: T * top].view(T, top)
        ops.residual(self.x[:T], self.w[weight], h, self.W, self.cfg.rms_eps, **terms)

    def _leave(self, b: StepBatch, hl: torch.Tensor, **terms) -> None:
        """The final norm of the rows whose logits are wanted."""
        ops.residual(self.x[: b.T], self.w["final.norm"], hl, self.W, self.cfg.rms_eps, rows=b.logit_rows, last=True, **terms)

    # -- one step ----------------------------------------------------------------------------------------
    def forward_batch(self, b: StepBatch, layer_begin: int = 0, layer_end: Optional[int] = None,
                      on_layer: Optional[Callable[[int, torch.Tensor], None]] = None) -> None:
        """Runs the rows of ``b``; greedy tokens go to ``b.out_tokens`` and / or logits to ``b.logits_out``.  ``layer_begin`` /
        ``layer_end`` run a slice of the layers (what lies between slices is in the static buffers); ``on_layer(i, x)`` sees the
        residual stream [T, width] after every layer."""
        cfg, w, T, n = self.cfg, self.w, b.T, b.n_logits
        layers = cfg.layers
        layer_end = len(layers) if layer_end is None else layer_end
        assert 0 < T <= self.max_tokens
        hl = self._head_rows(n)
        if layer_begin == 0:
            if self.tables is not None:
                ops.moe_place_table(b.ids, self.tables, self.max_experts, cfg.vocab_size)
            self._norm(b, "l0.norm1" if layers else "final.norm", embed=(b.ids, w["embed"][: cfg.vocab_size], 1.0, None))
            if not layers and n:
                self._leave(b, hl)
        for i in range(layer_begin, layer_end):
            m, f, p = layers[i].mixer, layers[i].mlp, f"l{i}."
            terms = dict((self._lightning if isinstance(m, LightningSpec) else self._attention)(b, i, m), post=w[p + "norm1b"])
            if f is not None:
                moe = isinstance(f, TableMoeSpec)
                self._norm(b, p + "norm2", i if moe else None, **terms)
                terms = dict((self._experts if moe else self._dense)(b, i, f), post=w[p + "norm2b"])
            if on_layer is not None:
                self._norm(b, "final.norm", **terms)
                on_layer(i, self.x[:T, : self.W])
                terms = {}
            if i + 1 < len(layers):
                self._norm(b, f"l{i + 1}.norm1", **terms)
            elif n:
                self._leave(b, hl, **terms)
        if layer_end == len(layers) and n:
            self._head(b, hl)
