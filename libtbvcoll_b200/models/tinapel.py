"""Tinapel decoder: gated linear attention, WKV and attention layers (values = unnormalised keys), each beside a mixture of experts in a parallel
block, over one fp32 residual stream; a position vector in the embedding, layers that run more than once, the embedding as output head.

What lies between two layers is ONE kernel (``ops.residual``: sum of the branches, the experts' weighted results included, loop terms, both
norms of the next layer, in a decode step also its mixes with the previous token).  A layer:

    gla     q, k, v, gate and low-rank decay GEMM -> [decay GEMM -> recurrence -> head norm + gate]  -> out-projection GEMM (fp32)
    wkv     five mixes with the previous token -> r, k, v, gate, low-rank decay GEMMs (grouped) -> [the same with a bonus] -> out-projection GEMM (fp32)
            in brackets: one kernel when every sequence has one row
    attn    query + key GEMM -> norm, temperature and cache write -> rows kernel over the cache (few rows) or tiled kernel (many) -> out-projection GEMM (fp32)
    moe     router GEMM (fp32) -> choice and dispatch -> gate / up GEMM over each expert's rows -> down GEMM;  shared expert: gate / up GEMM -> down GEMM (fp32)

``dtype`` float32 runs the same sequence with 32-bit weights, activations and products (rows kernel for every row).
All buffers of a decode step are preallocated, so the step can be captured in a CUDA graph."""
from __future__ import annotations

import os
from typing import Callable, Dict, Optional

import torch

from .. import ops
from ..engine.batch import StepBatch
from ..parallel.tp import TPGroup
from .config import GlaSpec, MoeSpec, SharedKvSpec, TinapelConfig, WkvSpec
from .decoder import StreamDecoder, pad16 as _pad16


class Tinapel(StreamDecoder):
    # from this many rows on, the mixes of a WKV layer go through separate many-token products instead of the grouped one
    GROUPED_MAX = 384

    def __init__(self, cfg: TinapelConfig, tp: TPGroup, weights: Dict[str, torch.Tensor], device, max_tokens: int, max_batch: int,
                 num_blocks: int, block_size: int = 16, max_attn_splits: int = 8, dtype: torch.dtype = torch.bfloat16):
        cfg.check_tp(tp.world)
        self.cfg, self.w, self.device, self.dtype = cfg, weights, torch.device(device), dtype
        self.block_size, self.num_blocks, self.max_tokens, self.max_batch, self.max_attn_splits = block_size, num_blocks, max_tokens, max_batch, max_attn_splits
        dev, f32, T = self.device, torch.float32, max_tokens
        self.W, self.Wp = cfg.hidden_size, _pad16(cfg.hidden_size)
        zeros = lambda *shape, dt=dtype: torch.zeros(*shape, dtype=dt, device=dev)
        big = lambda sizes: max(sizes, default=0)
        mixers = [(i, l.mixer) for i, l in enumerate(cfg.layers)]
        recurrent = [(i, m) for i, m in mixers if not isinstance(m, SharedKvSpec)]
        wkvs = [(i, m) for i, m in mixers if isinstance(m, WkvSpec)]
        attns = [m for _, m in mixers if isinstance(m, SharedKvSpec)]
        moes = [l.mlp for l in cfg.layers if l.mlp is not None]
        # activations; layers of different sizes share flat storage (row prefixes of these are what every call uses)
        self.turns = ops.position_turns(self.W, dev)
        self.x, self.y1, self.y2 = (zeros(T, self.Wp, dt=f32) for _ in range(3))
        self.x0 = zeros(T, self.Wp, dt=f32) if cfg.loop is not None and cfg.loop.times > 1 else None
        self.h1, self.h2 = zeros(T, self.Wp), zeros(T, self.Wp)
        self.h1f = zeros(T if wkvs else 0, self.Wp, dt=f32)
        self._flat = {
            "mixes": zeros(T * 5 * self.Wp if wkvs else 0),
            "wide": zeros(T * big([self.w[f"l{i}.mix.in"].shape[0] for i, _ in mixers])),
            "mid": zeros(T * big([m.heads * _pad16(getattr(m, "vdim", m.dim)) for _, m in mixers])),
            "z": zeros(T * big([m.heads * _pad16(m.dim) for _, m in recurrent]), dt=f32),
            "o": zeros(T * big([m.heads * _pad16(getattr(m, "vdim", m.dim)) for _, m in recurrent]), dt=f32),
            "low": zeros(T * big([self.w[f"l{i}.mix.decay"].shape[1] for i, _ in wkvs]), dt=f32),
            "low_h": zeros(T * big([self.w[f"l{i}.mix.decay"].shape[1] for i, _ in wkvs]) if dtype is torch.bfloat16 else 0),
            "qa": zeros(T * big([m.heads * ops.latent_row(_pad16(m.dim), 0) for m in attns])),
            "shared": zeros(T * big([_pad16(f.shared_ff or 0) for f in moes])),
            **self._expert_buffers(moes),
        }
        self._init_head()
        # cache and state, one per layer run (a looped layer has one per pass); slot 0 of the state is never a sequence's
        self.cache, self.state, self.shift = [], [], []
        slots = max_batch + 1
        for i in cfg.runs:
            m = cfg.layers[i].mixer
            attn = isinstance(m, SharedKvSpec)
            self.cache.append(zeros(num_blocks * m.kv_heads * block_size, ops.latent_row(_pad16(m.dim), 0)) if attn else None)
            self.state.append(None if attn else zeros(slots, m.heads, _pad16(m.dim), _pad16(getattr(m, "vdim", m.dim)), dt=f32))
            self.shift.append(zeros(slots, self.Wp, dt=f32) if isinstance(m, WkvSpec) else None)
        self.attn_ctas_per_row = max([m.kv_heads * ((m.heads // m.kv_heads + 15) // 16) for m in attns], default=1)
        self.scan_heads = min([m.heads for _, m in recurrent], default=0)
        self._groups = 0
        self.side = [torch.cuda.Stream(device=dev) for _ in range(2)] if os.environ.get("TBV_BRANCH_STREAMS", "1") != "0" and dev.type == "cuda" else []
        two_forms = bool(attns) and dtype is torch.bfloat16 and all(_pad16(m.dim) <= ops.SHARED_PREFILL_MAX_DIM for m in attns)
        self.rows_form_max = self.ROWS_FORM_MAX if two_forms else 1 << 60

    def _group_scratch(self, groups: int) -> tuple:
        """(states, decay totals) of the groups of cut segments, grown on demand (never inside a captured step)."""
        if groups > self._groups:
            sizes = [(m.heads * _pad16(m.dim), _pad16(getattr(m, "vdim", m.dim))) for m in (l.mixer for l in self.cfg.layers) if not isinstance(m, SharedKvSpec)]
            self._flat["starts"] = torch.empty(groups * max(k * v for k, v in sizes), dtype=torch.float32, device=self.device)
            self._flat["totals"] = torch.empty(groups * max(k for k, _ in sizes), dtype=torch.float32, device=self.device)
            self._groups = groups
        return self._flat["starts"], self._flat["totals"]

    @staticmethod
    def load_weights(cfg: TinapelConfig, source, tp: TPGroup, device, dtype):
        from ..utils.weights import load_tinapel
        return load_tinapel(cfg, source, device, dtype)

    def _scan(self, b: StepBatch, run: int, p: str, q, k, v, g, low, V: int, out, args: dict) -> None:
        """Recurrence over many rows; ``low`` is what enters the second decay product, which the chunked kernels do themselves."""
        w, z = self.w, None
        if b.scan_groups is not None:
            args = {**args, "groups": b.scan_groups, "scratch": self._group_scratch(b.scan_groups.shape[0]) if b.scan_cut else None}
        if b.scan_groups is not None and low.shape[1] <= ops.DECAY_RANK_MAX:
            args["low"] = (low, w[p + "decay"], w[p + "decay.b"])
        else:
            z = self._buf("z", b.T, w[p + "decay"].shape[0])
            ops.linear(low, w[p + "decay"], z, bias=w[p + "decay.b"])
        ops.decay_scan(q, k, v, g, z, w[p + "norm"], self.state[run], self._buf("o", b.T, V), out, b.segs, b.positions, **args)

    # -- branches of a layer -------------------------------------------------------------------------
    def _gla(self, b: StepBatch, run: int, i: int, m: GlaSpec, y) -> None:
        w, p, T = self.w, f"l{i}.mix.", b.T
        K, V = m.heads * _pad16(m.dim), m.heads * _pad16(m.vdim)
        wide, out = self._buf("wide", T, w[p + "in"].shape[0]), self._buf("mid", T, V)
        ops.linear(self.h1[:T], w[p + "in"], wide)
        q, k, v, g, low = wide.split((K, K, V, V, w[p + "decay"].shape[1]), 1)
        args = dict(vdim=m.vdim, eps=self.cfg.rms_eps, qscale=m.dim ** -0.5, tau=m.tau)
        if b.seg_of_row is None:
            ops.decay_step(q, k, v, g, low, w[p + "decay"], w[p + "decay.b"], w[p + "norm"], self.state[run], out, b.segs, b.positions, **args)
        else:
            self._scan(b, run, p, q, k, v, g, low, V, out, args)
        ops.linear(out, w[p + "o"], y)

    def _wkv(self, b: StepBatch, run: int, i: int, m: WkvSpec, y) -> None:
        w, p, T, Wp = self.w, f"l{i}.mix.", b.T, self.Wp
        K, R = m.heads * _pad16(m.dim), w[p + "decay"].shape[1]
        mixes, wide, out = self._buf("mixes", T, 5 * Wp), self._buf("wide", T, 4 * K + R), self._buf("mid", T, K)
        args = dict(vdim=m.dim, eps=self.cfg.rms_eps, u=w[p + "u"])
        r, k, v, g, low = wide.split((K, K, K, K, R), 1)
        if b.seg_of_row is None:                             # the mixes were written by the kernel between the layers
            ops.linear(mixes, w[p + "in"], wide, groups=4, x_group=Wp, y_group=K, last=R)
            ops.decay_step(r, k, v, g, low, w[p + "decay"], w[p + "decay.b"], w[p + "norm"], self.state[run], out, b.segs, b.positions, **args)
        else:
            ops.token_shift(self.h1f[:T], w[p + "mu"], self.shift[run], mixes, b.segs, b.seg_of_row, b.positions)
            if T < self.GROUPED_MAX or self.dtype is torch.float32:
                ops.linear(mixes, w[p + "in"][: 4 * K], wide, groups=4, x_group=Wp, y_group=K)
            else:
                for s, t in enumerate((r, k, v, g)):
                    ops.linear(mixes[:, s * Wp: (s + 1) * Wp], w[p + "in"][s * K: (s + 1) * K], t)
            lf = self._buf("low", T, R)
            lh = self._buf("low_h", T, R) if self.dtype is torch.bfloat16 else None
            ops.linear(mixes[:, 4 * Wp:], w[p + "in"][4 * K:], lf, act=ops.ACT_SOFTCAP, act_arg=1.0, copy=lh)          # tanh
            self._scan(b, run, p, r, k, v, g, lf if lh is None else lh, K, out, {**args, "shift": (self.h1f[:T], self.shift[run])})
        ops.linear(out, w[p + "o"], y)

    def _attention(self, b: StepBatch, run: int, i: int, m: SharedKvSpec, y) -> None:
        w, p, T, n = self.w, f"l{i}.mix.", b.T, b.n_rows_form
        H, G, D = m.heads, m.kv_heads, _pad16(m.dim)
        qk, out, qa = self._buf("wide", T, (H + G) * D), self._buf("mid", T, H * D), self._buf("qa", n, H, ops.latent_row(D, 0))
        cap, cache = m.softcap or 0.0, self.cache[run]
        ops.linear(self.h1[:T], w[p + "in"], qk)
        ops.shared_attention_prep(qk, qa, cache, w[p + "fold"], b.positions, b.slots, n, H, G, m.dim, self.block_size, self.cfg.rms_eps, m.temp_coef, m.temp_every)
        if n:
            ops.shared_attention_rows(qa, cache, b.tables, b.seq_of_row, b.ctx, out[:n].view(n, H, D), G, self.block_size, cap, splits=b.attn_splits)
        if n < T:
            ops.shared_attention_prefill(qk, cache, b.tables, b.seq_of_row, b.dense_tiles, out, H, G, self.block_size, cap)
        ops.linear(out, w[p + "o"], y)

    def _shared(self, b: StepBatch, i: int, f: MoeSpec, y) -> None:
        p, sh = f"l{i}.mlp.shared.", self._buf("shared", b.T, _pad16(f.shared_ff))
        ops.linear(self.h2[: b.T], self.w[p + "gate_up"], sh, glu=ops.SILU_GLU)
        ops.linear(sh, self.w[p + "down"], y)

    def _layer(self, b: StepBatch, run: int, i: int) -> dict:
        """Runs the branches of layer ``i``; returns their results as arguments of ``ops.residual``.  In a captured step the branches are
        parallel branches of the graph: each is a chain of kernels too small to fill the GPU."""
        lay, y1, y2 = self.cfg.layers[i], self.y1[: b.T], self.y2[: b.T]
        mixer = {GlaSpec: self._gla, WkvSpec: self._wkv, SharedKvSpec: self._attention}[type(lay.mixer)]
        out, branches = dict(y1=y1), []
        if lay.mlp is not None:
            branches.append(lambda: out.update(routed=self._experts(b, f"l{i}.mlp.", lay.mlp, self.h2[: b.T])))
            if lay.mlp.shared_ff:
                out["y2"] = y2
                branches.append(lambda: self._shared(b, i, lay.mlp, y2))
        if self.side and branches and torch.cuda.is_current_stream_capturing():
            main = torch.cuda.current_stream(self.device)
            for s, fn in zip(self.side, branches):
                s.wait_stream(main)
                with torch.cuda.stream(s):
                    fn()
            mixer(b, run, i, lay.mixer, y1)
            for s, _ in zip(self.side, branches):
                main.wait_stream(s)
        else:
            mixer(b, run, i, lay.mixer, y1)
            for fn in branches:
                fn()
        return out

    # -- between layers --------------------------------------------------------------------------------
    def _enter(self, b: StepBatch, run: int, **terms) -> None:
        """``ops.residual`` with ``terms``, the loop's terms and the norms of layer run ``run``."""
        i, t = self.cfg.schedule[run]
        lay, w, p, T = self.cfg.layers[i], self.w, f"l{i}.", b.T
        if t is not None:
            terms["step"] = w["loop.step"][t]
            if t > 0:
                terms["x0"] = self.x0[:T]
        if lay.mlp is not None:
            terms.update(g2=w[p + "norm2"], h2=self.h2[:T])
        h1 = self.h1
        if isinstance(lay.mixer, WkvSpec):
            h1 = self.h1f
            if b.seg_of_row is None:
                terms["mix"] = (w[p + "mix.mu"], self._buf("mixes", T, 5 * self.Wp), self.shift[run], b.segs)
        ops.residual(self.x[:T], w[p + "norm1"], h1[:T], self.W, self.cfg.rms_eps, positions=b.positions, **terms)

    def _leave(self, b: StepBatch, hl: torch.Tensor, **terms) -> None:
        """The final norm of the rows whose logits are wanted."""
        ops.residual(self.x[: b.T], self.w["final.norm"], hl, self.W, self.cfg.rms_eps, rows=b.logit_rows, last=True, **terms)

    # -- one step ----------------------------------------------------------------------------------------
    def forward_batch(self, b: StepBatch, layer_begin: int = 0, layer_end: Optional[int] = None,
                      on_layer: Optional[Callable[[int, torch.Tensor], None]] = None) -> None:
        """Runs the rows of ``b``; greedy tokens go to ``b.out_tokens`` and / or logits to ``b.logits_out``.  ``layer_begin`` /
        ``layer_end`` run a slice of the layer runs (what lies between slices is in the static buffers); ``on_layer(run, x)`` sees the
        residual stream [T, width] after every layer run."""
        cfg, w, T = self.cfg, self.w, b.T
        schedule = cfg.schedule
        layer_end = len(schedule) if layer_end is None else layer_end
        assert 0 < T <= self.max_tokens
        n = b.n_logits
        hl = self._head_rows(n)
        if layer_begin == 0:
            embed = (b.ids, w["embed"][: cfg.vocab_size], cfg.embedding_scale, self.turns)
            x0 = {} if self.x0 is None else {"x0": self.x0[:T]}
            if schedule:
                self._enter(b, 0, embed=embed, **x0)
            else:
                ops.residual(self.x[:T], w["final.norm"], self.h1[:T], self.W, cfg.rms_eps, embed=embed, positions=b.positions)
                self._leave(b, hl)
        for r in range(layer_begin, layer_end):
            terms = self._layer(b, r, schedule[r][0])
            if on_layer is not None:
                ops.residual(self.x[:T], w["final.norm"], self.h1[:T], self.W, cfg.rms_eps, **terms)
                on_layer(r, self.x[:T, : self.W])
                terms = {}
            if r + 1 < len(schedule):
                self._enter(b, r + 1, **terms)
            elif n:
                self._leave(b, hl, **terms)
        if layer_end < len(schedule) or not n:
            return
        self._head(b, hl)
