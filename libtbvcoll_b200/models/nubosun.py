"""Nubosun decoder: selective-scan (Mamba) and latent-attention layers, optional clamped gated feed-forwards, layer scale,
several residual streams with hyper-connections, layers that run more than once, soft-capped logits.

Per sublayer the residual streams (fp32) are read and written by ONE kernel (``ops.hyper_mix``: layer scale, stream mixing, next
norm).  Between two of them:

    mamba   in-projection GEMM -> convolution + SiLU -> x-projection GEMM (fp32 + bf16 copy) -> step-size GEMM (fp32)
            -> selective scan with the softplus before and the gate after it, replacing the carried state -> out-projection GEMM (fp32)
    latent  query + latent GEMM -> rotation, latent norm and cache write -> attention -> out-projection GEMM (fp32); attention is
            fold W_uk into the query (grouped GEMM) -> rows kernel over the cache -> expand with W_uv (grouped GEMM)    few rows
            or gather -> expand keys and values (GEMM) -> tiled kernel                                                  many rows
    mlp     gate / up GEMM with the clamped gated unit in its epilogue -> down GEMM (fp32)

``dtype`` float32 runs the same sequence with 32-bit weights, activations and products (rows kernel for every row).
All buffers of a decode step are preallocated, so the step can be captured in a CUDA graph."""
from __future__ import annotations

import os
from typing import Callable, Dict, Optional

import torch

from .. import ops
from ..engine.batch import StepBatch
from ..parallel.tp import TPGroup
from .config import LatentSpec, MambaSpec, NubosunConfig
from .latent import LatentAttention, pad16 as _pad16


class Nubosun(LatentAttention):
    # portions of at most this many tokens take the attention's rows form
    ROWS_FORM_MAX = 32
    uses_state = True
    expands_context = True

    @staticmethod
    def attn_cta_slots(splits: int, sms: int) -> int:
        """CTAs of the rows kernel that run at once: one per SM, but clusters of eight find only about four fifths of the SMs."""
        return sms if splits < 8 else sms * 4 // 5

    def __init__(self, cfg: NubosunConfig, tp: TPGroup, weights: Dict[str, torch.Tensor], device, max_tokens: int, max_batch: int,
                 num_blocks: int, block_size: int = 16, max_attn_splits: int = 8, dtype: torch.dtype = torch.bfloat16):
        cfg.check_tp(tp.world)
        self.cfg, self.w, self.device, self.dtype = cfg, weights, torch.device(device), dtype
        self.block_size, self.num_blocks, self.max_tokens, self.max_batch, self.max_attn_splits = block_size, num_blocks, max_tokens, max_batch, max_attn_splits
        dev, f32, T = self.device, torch.float32, max_tokens
        self.W, self.Wp, self.Vp = cfg.hidden_size, _pad16(cfg.hidden_size), _pad16(cfg.vocab_size)
        zeros = lambda *shape, dt=dtype: torch.zeros(*shape, dtype=dt, device=dev)
        mambas = [l.mixer for l in cfg.layers if isinstance(l.mixer, MambaSpec)]
        self.latents = latents = [l.mixer for l in cfg.layers if isinstance(l.mixer, LatentSpec)]
        mlps = [l.mlp for l in cfg.layers if l.mlp is not None]
        # activations; layers of different sizes share flat storage (row prefixes of these are what every call uses)
        self.x = zeros(T, cfg.streams, self.Wp, dt=f32)
        self.h = zeros(T, self.Wp)
        self.y = zeros(T, self.Wp, dt=f32)
        big = lambda sizes: max(sizes, default=0)
        self._flat = {
            "wide": zeros(T * big([2 * _pad16(m.inner) for m in mambas] + [self._qkv_cols(m) for m in latents])),
            "mid": zeros(T * big([_pad16(m.inner) for m in mambas] + [m.heads * _pad16(m.vdim) for m in latents] + [_pad16(m.ff) for m in mlps])),
            "proj": zeros(T * big([_pad16(m.dt_rank + 2 * m.state) for m in mambas]), dt=f32),
            "proj_h": zeros(T * big([_pad16(m.dt_rank + 2 * m.state) for m in mambas]) if dtype is torch.bfloat16 else 0),
            "dt": zeros(T * big([_pad16(m.inner) for m in mambas]), dt=f32),
            "qa": zeros(T * big([m.heads * self.latent_row(m) for m in latents])),
            "lat": zeros(T * big([m.heads * _pad16(m.kv_rank) for m in latents])),
        }
        self.ones = torch.ones(cfg.streams, dtype=f32, device=dev)
        self.hl = zeros(max_batch, self.Wp)
        self.logits = zeros(max_batch, self.Vp, dt=f32)
        self.argmax_ws = ops.argmax_workspace(max_batch, dev)
        self.argmax_val = zeros(max_batch, dt=f32)
        # cache and state, one per layer run (a looped layer has one per pass); slot 0 of the state is never a sequence's
        self.cache, self.conv, self.ssm, self.rot = [], [], [], {}
        slots = max_batch + 1
        for i in cfg.runs:
            m = cfg.layers[i].mixer
            if isinstance(m, MambaSpec):
                self.cache.append(None)
                self.conv.append(zeros(slots, m.conv - 1, _pad16(m.inner), dt=f32))
                self.ssm.append(zeros(slots, m.inner, m.state, dt=f32))
            else:
                self.cache.append(zeros(num_blocks * block_size, self.latent_row(m)))
                self.conv.append(None)
                self.ssm.append(None)
                if i not in self.rot:
                    f, factor = ops.rope_frequencies(m.rot.dims, m.rot.base, m.rot.scaling)
                    self.rot[i] = (ops.frequency_turns(f, dev), factor)
        self.attn_ctas_per_row = max([(m.heads + 15) // 16 for m in latents], default=1)
        two_forms = bool(latents) and dtype is torch.bfloat16 and all(ops.latent_prefill_fits(_pad16(m.dim), _pad16(m.rot_dim), _pad16(m.vdim)) for m in latents)
        self.rows_form_max = self.ROWS_FORM_MAX if two_forms else 1 << 60
        self.l2_prefetch = os.environ.get("TBV_L2_PREFETCH", "1") != "0"

    @staticmethod
    def scan_group_rows(rows) -> int:
        """The selective scan takes whole segments."""
        return 0

    @staticmethod
    def load_weights(cfg: NubosunConfig, source, tp: TPGroup, device, dtype):
        from ..utils.weights import load_nubosun
        return load_nubosun(cfg, source, device, dtype)

    @staticmethod
    def _qkv_cols(m: LatentSpec) -> int:
        return m.heads * (_pad16(m.dim) + _pad16(m.rot_dim)) + _pad16(m.kv_rank) + _pad16(m.rot_dim)

    def _buf(self, name: str, rows: int, *shape: int) -> torch.Tensor:
        n = rows
        for s in shape:
            n *= s
        return self._flat[name][:n].view(rows, *shape)

    # -- sublayers: h [T, Wp] -> y [T, Wp] fp32 ------------------------------------------------------
    def _mamba(self, b: StepBatch, run: int, i: int, m: MambaSpec, h, y) -> None:
        w, p, T = self.w, f"l{i}.mix.", b.T
        ip, pp, kd = _pad16(m.inner), _pad16(m.dt_rank + 2 * m.state), _pad16(m.dt_rank)
        xz, u = self._buf("wide", T, 2 * ip), self._buf("mid", T, ip)
        proj, dt = self._buf("proj", T, pp), self._buf("dt", T, ip)
        ops.linear(h, w[p + "in"], xz)
        ops.causal_conv_silu(xz, u, w[p + "conv"], w[p + "conv.b"], self.conv[run], b.segs, b.seg_of_row, b.positions)
        if self.dtype is torch.bfloat16:
            low = self._buf("proj_h", T, pp)
            ops.linear(u, w[p + "x"], proj, copy=low)
        else:
            low = proj
            ops.linear(u, w[p + "x"], proj)
        ops.linear(low[:, :kd], w[p + "dt"], dt, bias=w[p + "dt.b"])
        ops.selective_scan(u, xz, ip, dt, proj, m.dt_rank, m.dt_rank + m.state, w[p + "a2"], w[p + "D"], self.ssm[run], self.conv[run], u, b.segs,
                           b.positions, one_token=b.seg_of_row is None)
        self._announce_mlp(i, T)
        ops.linear(u, w[p + "o"], y)

    def _latent(self, b: StepBatch, run: int, i: int, m: LatentSpec, h, y) -> None:
        w, p, T, n = self.w, f"l{i}.mix.", b.T, b.n_rows_form
        H, D, V, R, rot = m.heads, _pad16(m.dim), _pad16(m.vdim), _pad16(m.kv_rank), _pad16(m.rot_dim)
        q_rot = H * D
        c_off = q_rot + H * rot
        qkv, out = self._buf("wide", T, self._qkv_cols(m)), self._buf("mid", T, H * V)
        qa = self._buf("qa", n, H, self.latent_row(m))
        turns, factor = self.rot[i]
        cache = self.cache[run]
        ops.linear(h, w[p + "qkv"], qkv)
        ops.latent_prep(qkv, qkv, qa, cache, w[p + "dkv.norm"], turns, factor, b.positions, b.slots, n, q_rot, c_off, c_off + R, H, m.kv_rank, R, rot,
                        self.cfg.rms_eps)
        self._latent_attend(b, p, m, qkv, qa, cache, out, b.attn_splits)
        self._announce_mlp(i, T)
        ops.linear(out, w[p + "o"], y)

    def _announce_mlp(self, i: int, T: int) -> None:
        """Decode: the out-projection asks for the gate / up weights that follow it (ops.prefetch_next)."""
        if self.l2_prefetch and T <= 64 and self.cfg.layers[i].mlp is not None and self.dtype is torch.bfloat16:
            ops.prefetch_next(self.w[f"l{i}.mlp.gate_up"])

    def _mlp(self, b: StepBatch, i: int, m, h, y) -> None:
        p = f"l{i}.mlp."
        act = self._buf("mid", b.T, _pad16(m.ff))
        ops.linear(h, self.w[p + "gate_up"], act, glu=(m.limit, m.slope))
        ops.linear(act, self.w[p + "down"], y)

    # -- one step ----------------------------------------------------------------------------------------
    def forward_batch(self, b: StepBatch, layer_begin: int = 0, layer_end: Optional[int] = None,
                      on_layer: Optional[Callable[[int, torch.Tensor], None]] = None) -> None:
        """Runs the rows of ``b``; greedy tokens go to ``b.out_tokens`` and / or logits to ``b.logits_out``.  ``layer_begin`` /
        ``layer_end`` run a slice of the layer runs (the state between slices lives in the static buffers); ``on_layer(run, streams)`` sees the
        streams [T, streams, width] after every layer run."""
        cfg, w, T, eps, W = self.cfg, self.w, b.T, self.cfg.rms_eps, self.W
        runs = cfg.runs
        layer_end = len(runs) if layer_end is None else layer_end
        assert 0 < T <= self.max_tokens
        x, h, y = self.x[:T], self.h[:T], self.y[:T]
        if b.n_rows_form < T:
            self._context_scratch(b.dense_slots.shape[0])
        n = b.n_logits
        hl = self.hl[:n] if n <= self.max_batch else torch.empty(n, self.Wp, dtype=self.dtype, device=self.device)
        if layer_begin == 0:
            p = f"l{runs[0]}." if runs else None
            ops.hyper_embed(b.ids, w["embed"], cfg.embedding_scale, x, w[p + "hc1.in"] if p else self.ones, w[p + "norm1"] if p else w["final.norm"], h, W, eps)
            if not runs:
                hl.copy_(h if b.logit_rows is None else h[b.logit_rows])
        for r in range(layer_begin, layer_end):
            i = runs[r]
            lay, p = cfg.layers[i], f"l{i}."
            if isinstance(lay.mixer, MambaSpec):
                self._mamba(b, r, i, lay.mixer, h, y)
            else:
                self._latent(b, r, i, lay.mixer, h, y)
            end = (p + "ls1", p + "hc1.out", p + "hc1.mix")
            if lay.mlp is not None:
                ops.hyper_mix(y, *(w[k] for k in end), x, w[p + "hc2.in"], w[p + "norm2"], h, W, eps)
                self._mlp(b, i, lay.mlp, h, y)
                end = (p + "ls2", p + "hc2.out", p + "hc2.mix")
            if r + 1 < len(runs):
                q = f"l{runs[r + 1]}."
                ops.hyper_mix(y, *(w[k] for k in end), x, w[q + "hc1.in"], w[q + "norm1"], h, W, eps)
            else:
                if n:
                    ops.hyper_mix(y, *(w[k] for k in end), x, self.ones, w["final.norm"], hl, W, eps, rows=b.logit_rows, last=True)
                if on_layer is not None:
                    ops.hyper_mix(y, *(w[k] for k in end), x, self.ones, w["final.norm"], h, W, eps)
            if on_layer is not None:
                on_layer(r, x[:, :, :W])
        if layer_end < len(runs) or not n:
            return
        logits = self.logits[:n] if n <= self.max_batch else torch.empty(n, self.Vp, dtype=torch.float32, device=self.device)
        cap = cfg.logit_softcap
        ops.linear(hl, w["head"], logits, act=ops.ACT_SOFTCAP if cap else ops.ACT_NONE, act_arg=cap or 0.0)
        if b.logits_out is not None:
            b.logits_out.copy_(logits[:, : cfg.vocab_size])
        if b.out_tokens is not None:
            assert n <= self.max_batch
            ops.argmax(logits[:, : cfg.vocab_size], self.argmax_ws, 0, self.argmax_val[:n], b.out_tokens[:n])
