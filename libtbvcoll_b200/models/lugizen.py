"""Lugizen decoder: delta-rule recurrences with a decay per key channel, attention with norms per head and values mixed with an earlier layer's, windowed latent
attention; dense GELU feed-forwards or mixtures of experts; one norm behind every sublayer, none before; a short convolution over what a mixer reads.

What lies between two sublayers is ONE kernel (``ops.residual`` with ``post``: norm of the branch, residual sum and, when every sequence has one row, the next
layer's convolution; otherwise ``ops.short_conv`` follows).  Feed-forwards read the residual stream itself.

    delta       q, k, v, low-rank decay and gate, step size GEMM -> [convolution + SiLU -> decay GEMM (fp32, softplus inside), gate GEMM -> recurrence with unit norms, head norm and
                gate] -> out-projection GEMM (fp32); in brackets: one kernel when every sequence has one row
    attention   q, k, v GEMM -> norms, rotation, value mix, cache write -> rows kernel over the cache (few rows) or tiled kernel (many) -> out-projection GEMM (fp32)
    latent      query latent, latent, rotated key GEMM -> norms, rotation, cache write -> query GEMM -> rotation -> latent attention with a window ->
                out-projection GEMM (fp32)
    dense       up GEMM (GELU inside) -> down GEMM (fp32)
    experts     router GEMM (fp32) -> choice and dispatch -> gate / up GEMM over each expert's rows -> down GEMM

``dtype`` float32 runs the same sequence with 32-bit weights, activations and products (rows kernels for every row).  All buffers of a decode step are
preallocated, so the step can be captured in a CUDA graph."""
from __future__ import annotations

import os
from typing import Callable, Dict, Optional

import torch

from .. import ops
from ..engine.batch import StepBatch
from ..parallel.tp import TPGroup
from .config import ChannelDeltaSpec, GeluMlpSpec, HeadAttentionSpec, LatentSpec, LugizenConfig, MoeSpec
from .decoder import StreamDecoder, pad16
from .latent import LatentAttention


class Lugizen(StreamDecoder, LatentAttention):
    head_weight = "head"

    def __init__(self, cfg: LugizenConfig, tp: TPGroup, weights: Dict[str, torch.Tensor], device, max_tokens: int, max_batch: int,
                 num_blocks: int, block_size: int = 16, max_attn_splits: int = 8, dtype: torch.dtype = torch.bfloat16):
        cfg.check_tp(tp.world)
        self.cfg, self.w, self.device, self.dtype = cfg, weights, torch.device(device), dtype
        self.block_size, self.num_blocks, self.max_tokens, self.max_batch, self.max_attn_splits = block_size, num_blocks, max_tokens, max_batch, max_attn_splits
        dev, f32, T = self.device, torch.float32, max_tokens
        self.W, self.Wp = cfg.hidden_size, pad16(cfg.hidden_size)
        zeros = lambda *shape, dt=dtype: torch.zeros(*shape, dtype=dt, device=dev)
        big = lambda sizes: max(sizes, default=0)
        mixers = [(i, l.mixer) for i, l in enumerate(cfg.layers)]
        deltas = [(i, m) for i, m in mixers if isinstance(m, ChannelDeltaSpec)]
        attns = [m for _, m in mixers if isinstance(m, HeadAttentionSpec)]
        self.latents = [m for _, m in mixers if isinstance(m, LatentSpec)]
        mixed = [i for i, m in mixers if isinstance(m, HeadAttentionSpec) and m.v_mix]
        self.first_values = mixed[0] if mixed else -1          # the layer whose values the others mix in
        dense = [l.mlp for l in cfg.layers if isinstance(l.mlp, GeluMlpSpec)]
        moes = [l.mlp for l in cfg.layers if isinstance(l.mlp, MoeSpec)]
        # activations; layers of different sizes share flat storage (row prefixes of these are what every call uses)
        self.x, self.y = zeros(T, self.Wp, dt=f32), zeros(T, self.Wp, dt=f32)
        self.h = zeros(T, self.Wp)
        rows_of = lambda i, name: self.w[f"l{i}.mix.{name}"].shape[0]
        self._flat = {
            "wide": zeros(T * big([rows_of(i, "uq" if isinstance(m, LatentSpec) else "in") for i, m in mixers])),
            "low": zeros(T * big([rows_of(i, "down") for i, m in mixers if isinstance(m, LatentSpec)])),
            "mid": zeros(T * big([m.heads * pad16(m.vdim) for _, m in mixers])),
            "conv": zeros(T * big([self.w[f"l{i}.mix.conv"].shape[1] for i, _ in deltas])),
            "z": zeros(T * big([m.heads * pad16(m.dim) for _, m in deltas]), dt=f32),
            "gate": zeros(T * big([m.heads * pad16(m.vdim) for _, m in deltas])),
            "o": zeros(T * big([m.heads * pad16(m.vdim) for _, m in deltas]), dt=f32),
            "first": zeros(T * big([m.kv_heads * pad16(m.vdim) for m in attns if m.v_mix])),
            "qa": zeros(T * big([m.heads * ops.latent_row(pad16(m.dim), 0) for m in attns] + [m.heads * self.latent_row(m) for m in self.latents])),
            "lat": zeros(T * big([m.heads * pad16(m.kv_rank) for m in self.latents])),
            **self._expert_buffers(moes, extra_act=big([pad16(f.ff) for f in dense])),
        }
        self._init_head()
        # cache and state of every layer (slot 0 of the state is never a sequence's)
        slots = max_batch + 1
        self.past = [zeros(slots, cfg.canon_taps - 1, self.Wp, dt=f32) for _ in mixers]
        self.cache, self.state, self.conv, self.turns = [], [], [], []
        for i, m in mixers:
            delta = isinstance(m, ChannelDeltaSpec)
            self.state.append(zeros(slots, m.heads, pad16(m.dim), pad16(m.vdim), dt=f32) if delta else None)
            self.conv.append(zeros(slots, m.conv - 1, self.w[f"l{i}.mix.conv"].shape[1], dt=f32) if delta else None)
            self.turns.append(None if delta or m.rot is None or not m.rot.dims else ops.rotation_turns(m.rot.dims, m.rot.base, dev))
            if delta:
                self.cache.append(None)
            elif isinstance(m, LatentSpec):
                self.cache.append(zeros(num_blocks * block_size, self.latent_row(m)))
            else:
                self.cache.append(zeros(num_blocks * m.kv_heads * block_size, ops.latent_row(pad16(m.dim), pad16(m.vdim))))
        self.expands_context = bool(self.latents)
        self.context_window = max(m.window for m in self.latents) if self.latents and all(m.window for m in self.latents) else 0
        self.attn_ctas_per_row = 0                             # the engine's choice follows the context alone; layer_splits knows each layer's CTAs
        self.scan_heads = min([m.heads for _, m in deltas], default=0)
        two_forms = bool(attns or self.latents) and dtype is torch.bfloat16 and all(ops.paired_prefill_fits(pad16(m.dim), pad16(m.vdim)) for m in attns) \
            and all(ops.latent_prefill_fits(pad16(m.dim), pad16(m.rot_dim), pad16(m.vdim)) for m in self.latents)
        self.rows_form_max = self.ROWS_FORM_MAX if two_forms else 1 << 60
        self.sms = torch.cuda.get_device_properties(dev).multi_processor_count if dev.type == "cuda" else 1
        self.l2_prefetch = os.environ.get("TBV_L2_PREFETCH", "1") != "0"

    @staticmethod
    def load_weights(cfg: LugizenConfig, source, tp: TPGroup, device, dtype):
        from ..utils.weights import load_lugizen
        return load_lugizen(cfg, source, device, dtype)

    def scan_group_rows(self, rows) -> int:
        """The recurrence takes whole segments: what a piece of one does to the state is a matrix, not a factor per channel."""
        if self.dtype is not torch.bfloat16 or not self.scan_heads:
            return 0
        return -(-int(rows.max()) // self.SCAN_CHUNK) * self.SCAN_CHUNK

    def _sets_scratch(self, size: int) -> Optional[torch.Tensor]:
        """Operands of all chunks of a recurrence, grown on demand (never inside a captured step)."""
        if not size:
            return None
        if "sets" not in self._flat or self._flat["sets"].numel() < size:
            self._flat["sets"] = torch.empty(size, dtype=torch.uint8, device=self.device)
        return self._flat["sets"]

    def layer_splits(self, m, rows: int, splits: int) -> int:
        """CTAs per row of an attention layer, at most ``splits``: what runs at once (an SM holds two CTAs of the kernel over paired rows, one over latents), and at
        least 64 visible keys for each."""
        latent = isinstance(m, LatentSpec)
        units = rows * ((m.heads + 15) // 16 if latent else m.kv_heads * ((m.heads // m.kv_heads + 15) // 16))
        while splits > 1 and (units * splits > self.attn_cta_slots(splits, self.sms) // (2 if latent else 1) or (latent and m.window and m.window // splits < 64)):
            splits //= 2
        return splits

    # -- sublayers ---------------------------------------------------------------------------------------
    def _delta(self, b: StepBatch, i: int, m: ChannelDeltaSpec) -> dict:
        w, p, T = self.w, f"l{i}.mix.", b.T
        K, V, R = m.kv_heads * pad16(m.dim), m.heads * pad16(m.vdim), w[p + "a2"].shape[1]
        C = 2 * K + V
        wide, out = self._buf("wide", T, w[p + "in"].shape[0]), self._buf("mid", T, V)
        ops.linear(self.h[:T], w[p + "in"], wide)
        qkv, low_a, low_g, beta = wide.split((C, R, R, pad16(m.heads)), 1)
        one = b.seg_of_row is None
        inside = one and m.kv_heads == m.heads             # the recurrence's kernel does the convolution too
        if not inside:
            raw, qkv = qkv, self._buf("conv", T, C)
            ops.short_conv(raw, qkv, w[p + "conv"], self.conv[i], b.segs, b.seg_of_row, b.positions)
        q, k, v = qkv.split((K, K, V), 1)
        args = dict(kv_heads=m.kv_heads, dim=m.dim, vdim=m.vdim, eps=self.cfg.rms_eps)
        if one:
            ops.delta_step(q, k, v, beta, low_a, low_g, w[p + "a2"], w[p + "dt_bias"], w[p + "g2"], w[p + "rate"], w[p + "norm"], self.state[i], out, b.segs, b.positions,
                           conv=(w[p + "conv"], self.conv[i]) if inside else None, **args)
        else:
            z, gate = self._buf("z", T, w[p + "a2"].shape[0]), self._buf("gate", T, V)
            ops.linear(low_a, w[p + "a2"], z, bias=w[p + "dt_bias"], act=ops.ACT_SOFTPLUS)
            ops.linear(low_g, w[p + "g2"], gate)
            ops.delta_scan(q, k, v, beta, z, gate, w[p + "rate"], w[p + "norm"], self.state[i], self._buf("o", T, V), out, b.segs, b.positions, groups=b.scan_groups,
                           sets=None if b.scan_groups is None else self._sets_scratch(ops.delta_sets(T, b.scan_groups.shape[0], self.state[i])), **args)
        return self._project(b, i, out)

    def _attention(self, b: StepBatch, i: int, m: HeadAttentionSpec) -> dict:
        w, p, T, n = self.w, f"l{i}.mix.", b.T, b.n_rows_form
        H, G, D, V = m.heads, m.kv_heads, pad16(m.dim), pad16(m.vdim)
        wide, out, qa, cache = self._buf("wide", T, (H + G) * D + G * V), self._buf("mid", T, H * V), self._buf("qa", n, H, ops.latent_row(D, 0)), self.cache[i]
        ops.linear(self.h[:T], w[p + "in"], wide)
        ops.head_attention_prep(wide, qa, cache, w[p + "qscale"], self.turns[i], b.positions, b.slots, n, H, G, m.dim, D, self.block_size, self.cfg.rms_eps,
                                v_first=self._buf("first", T, G * V) if m.v_mix else None, mix=w[p + "vmix"] if m.v_mix and i != self.first_values else None)
        if n:
            ops.paired_attention_rows(qa, cache, b.tables, b.seq_of_row, b.ctx, out[:n].view(n, H, V), G, self.block_size, splits=self.layer_splits(m, n, b.attn_splits))
        if n < T:
            ops.paired_attention_prefill(wide, cache, b.tables, b.seq_of_row, b.dense_tiles, out, H, G, D, self.block_size)
        return self._project(b, i, out)

    def _latent(self, b: StepBatch, i: int, m: LatentSpec) -> dict:
        w, p, T, n = self.w, f"l{i}.mix.", b.T, b.n_rows_form
        H, D, V, R, Rq, rot = m.heads, pad16(m.dim), pad16(m.vdim), pad16(m.kv_rank), pad16(m.q_rank), pad16(m.rot_dim)
        low, q, out = self._buf("low", T, Rq + R + rot), self._buf("wide", T, H * (D + rot)), self._buf("mid", T, H * V)
        qa, cache = self._buf("qa", n, H, self.latent_row(m)), self.cache[i]
        prep = lambda low, q, gamma, latent: ops.latent_prep(low, q, qa, cache, gamma, self.turns[i], 1.0, b.positions, b.slots, n, H * D, Rq, Rq + R, H, m.kv_rank, R, rot,
                                                             self.cfg.rms_eps, query_latent=latent)
        ops.linear(self.h[:T], w[p + "down"], low)
        prep(low, None, w[p + "dkv.norm"], (0, m.q_rank, w[p + "dq.norm"]))
        ops.linear(low[:, :Rq], w[p + "uq"], q)
        prep(None, q, None, None)
        self._latent_attend(b, p, m, q, qa, cache, out, self.layer_splits(m, n, b.attn_splits))
        return self._project(b, i, out)

    def _project(self, b: StepBatch, i: int, out: torch.Tensor) -> dict:
        y = self.y[: b.T]
        if self.l2_prefetch and b.T <= 64 and isinstance(self.cfg.layers[i].mlp, GeluMlpSpec) and self.dtype is torch.bfloat16:
            ops.prefetch_next(self.w[f"l{i}.mlp.up"])      # decode: the out-projection asks for the weights that follow it
        ops.linear(out, self.w[f"l{i}.mix.o"], y)
        return dict(y1=y)

    def _dense(self, b: StepBatch, i: int, f: GeluMlpSpec) -> dict:
        p, fp, y = f"l{i}.mlp.", pad16(f.ff), self.y[: b.T]
        act = self._buf("act", b.T, fp)
        ops.linear(self.h[: b.T], self.w[p + "up"], act, act=ops.ACT_GELU, act_cols=fp)
        ops.linear(act, self.w[p + "down"], y)
        return dict(y1=y)

    # -- between sublayers -------------------------------------------------------------------------------
    def _enter(self, b: StepBatch, i: int, **terms) -> None:
        """The residual stream takes ``terms``; what the mixer of layer ``i`` reads goes to ``h``."""
        x, h, taps = self.x[: b.T], self.h[: b.T], self.w[f"l{i}.canon1"]
        if b.seg_of_row is None:
            ops.residual(x, None, h, self.W, self.cfg.rms_eps, positions=b.positions, conv=(taps, self.past[i], b.segs), **terms)
        else:
            if terms:
                ops.residual(x, None, None, self.W, self.cfg.rms_eps, positions=b.positions, **terms)
            ops.short_conv(x, h, taps, self.past[i], b.segs, b.seg_of_row, b.positions, add=True)

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
        if self.latents and b.n_rows_form < T:
            self._context_scratch(b.dense_slots.shape[0])
        hl = self._head_rows(n)
        if layer_begin == 0:
            embed = (b.ids, w["embed"], 1.0, None)
            if layers:
                self._enter(b, 0, embed=embed)
            else:
                ops.residual(self.x[:T], None, None, self.W, cfg.rms_eps, embed=embed)
                if n:
                    self._leave(b, hl)
        mixers = {ChannelDeltaSpec: self._delta, HeadAttentionSpec: self._attention, LatentSpec: self._latent}
        for i in range(layer_begin, layer_end):
            m, f, p = layers[i].mixer, layers[i].mlp, f"l{i}."
            terms = dict(mixers[type(m)](b, i, m), post=w[p + "norm1"])
            if f is not None:
                ops.residual(self.x[:T], None, self.h[:T], self.W, cfg.rms_eps, **terms)
                terms = dict(dict(routed=self._experts(b, p + "mlp.", f, self.h[:T])) if isinstance(f, MoeSpec) else self._dense(b, i, f), post=w[p + "norm2"])
            if on_layer is not None:
                ops.residual(self.x[:T], None, None, self.W, cfg.rms_eps, **terms)
                on_layer(i, self.x[:T, : self.W])
                terms = {}
            if i + 1 < len(layers):
                self._enter(b, i + 1, **terms)
            elif n:
                self._leave(b, hl, **terms)
        if layer_end == len(layers) and n:
            self._head(b, hl)
