#!/usr/bin/env python3
"""Nubosun beside the closest other model (Llama) at equal width, depth, feed-forward, heads and vocabulary: prefill and decode
throughput through the engine, and every kernel of both at the same shapes against its roofline.

    python bench.py --compare nubosun [--sizes 2k,8b]          (or: python -m libtbvcoll_b200.bench_nubosun)

Random weights, random token ids.  Model numbers: device time of captured decode steps (CUDA events), prefill by events around
the engine's prefill.  Kernel numbers: ``reps`` distinct sets of operands (more than the L2 in total) cycled inside one CUDA graph; roofline
time = max(bytes / measured copy bandwidth, FLOPs / measured bf16 rate, for the scan also exponentials / 16 per clock and SM at 1965 MHz),
fraction = roofline time / measured time."""
from __future__ import annotations

import argparse
import json
import math
import statistics

import torch

PAIRS = {"2k": ("nubosun-2k", "llama3-2k"), "8b": ("nubosun-8b", "llama3-8b")}


def _pad16(n):
    return (n + 15) // 16 * 16


# ---- whole models ---------------------------------------------------------------------------------------------------------
def model_numbers(name: str, batches=(1, 8, 32), prompt: int = 512, long_prompt: int = 4096, steps: int = 32) -> dict:
    from .engine.engine import Engine
    from .models.config import get_config
    cfg = get_config(name)
    B = max(batches)
    eng = Engine(cfg, device="cuda:0", seed=0, max_batch=B, max_seq_len=max(prompt + 4 * steps + 16, long_prompt + 16),
                 max_cache_tokens=max(B * (prompt + 4 * steps + 32), long_prompt + 32), prefill_chunk=4096)
    g = torch.Generator().manual_seed(7)
    out = {"model": name, "params": cfg.param_count(), "decode": {}, "prefill": {}}

    def timed(fn, reps=3):
        best = []
        for _ in range(reps):
            e0, e1 = torch.cuda.Event(enable_timing=True), torch.cuda.Event(enable_timing=True)
            torch.cuda.synchronize()
            e0.record()
            fn()
            e1.record()
            torch.cuda.synchronize()
            best.append(e0.elapsed_time(e1))
        return statistics.median(best)
    for nb, L in ((8, prompt), (1, long_prompt)):
        prompts = [torch.randint(0, cfg.vocab_size, (L,), generator=g).tolist() for _ in range(nb)]
        eng.prefill(prompts, 8)
        ms = timed(lambda: eng.prefill(prompts, 8))
        out["prefill"][f"{nb}x{L}"] = {"ms": round(ms, 3), "tokens_per_s": round(nb * L / ms * 1e3, 1)}
    for nb in batches:
        prompts = [torch.randint(0, cfg.vocab_size, (prompt,), generator=g).tolist() for _ in range(nb)]
        first = eng.prefill(prompts, 4 * steps + 8)
        splits = eng.attn_splits_for(nb, prompt + 4 * steps)
        eng._load_decode_inputs(nb, first, [prompt] * nb)
        eng.step_counter.zero_()
        graph = eng.capture(nb, splits, True)
        for _ in range(4):
            graph.replay()

        def run():
            for _ in range(steps):
                graph.replay()
        ms = timed(run) / steps
        out["decode"][str(nb)] = {"ms_per_step": round(ms, 4), "tokens_per_s": round(nb / ms * 1e3, 1), "launches_per_step": eng.launches_per_step}
    del eng
    torch.cuda.empty_cache()
    return out


# ---- kernel by kernel -------------------------------------------------------------------------------------------------------
class _Kernels:
    def __init__(self, only: str = ""):
        self.only = only
        from .bench_ops import peaks
        self.hbm, self.tf, self.src = peaks()
        self.rows = []
        self.sms = torch.cuda.get_device_properties(0).multi_processor_count

    def time(self, group: str, name: str, make, bytes_, flops=0.0, exps=0.0, fp32=0.0):
        """make(i) -> callable on the i-th set of operands; sets are made until they exceed the L2.  ``exps`` run at 16, ``fp32`` instructions (FMA or
        other) at 128 per clock and SM."""
        if self.only not in name:
            return
        from .bench_ops import time_graph
        torch.cuda.empty_cache()
        sets = max(2, min(64, math.ceil(400e6 / max(bytes_, 1.0))))
        us = time_graph([make(i) for i in range(sets)])
        ideal = max(bytes_ / (self.hbm * 1e3), flops / (self.tf * 1e6), exps / (16 * self.sms * 1.965e3), fp32 / (128 * self.sms * 1.965e3))
        self.rows.append({"group": group, "kernel": name, "us": round(us, 2), "roofline_us": round(ideal, 2), "of_measured_peak": round(ideal / us, 3)})


def _w(*shape):
    return (torch.randn(*shape, device="cuda") * 0.02).to(torch.bfloat16)


def _linear(k: _Kernels, group, name, T, M, K, f32=False, glu=None, act=0, copy=False, silu=False, groups=1):
    from . import ops
    out_bytes = T * groups * (M // 2 if glu or silu else M) * (4 if f32 else 2) + (T * M * 2 if copy else 0)

    def make(i):
        x, w = _w(T, groups * K), _w(groups * M, K)
        if silu:
            out = torch.empty(T, M // 2, dtype=torch.bfloat16, device="cuda")
            return lambda: ops.gemm(x, w, out=out, epi=ops.EPI_SILU_MUL)
        out = torch.empty(T, groups * (M // 2 if glu else M), dtype=torch.float32 if f32 else torch.bfloat16, device="cuda")
        c = torch.empty(T, M, dtype=torch.bfloat16, device="cuda") if copy else None
        if groups > 1:
            return lambda: ops.linear(x, w, out, groups=groups, x_group=K, y_group=M)
        return lambda: ops.linear(x, w, out, glu=glu, act=act, act_arg=30.0, copy=c)
    k.time(group, name, make, T * groups * K * 2 + groups * M * K * 2 + out_bytes, 2.0 * T * groups * M * K)


def kernel_numbers(size: str, T: int, seqs: int, ctx: int, only: str = "") -> list:
    """T rows in ``seqs`` sequences: T == seqs is a decode step over ``ctx`` cached tokens, otherwise whole prompts."""
    from . import ops
    from .engine.batch import dense_context
    from .models.config import LatentSpec, MambaSpec, get_config
    from .models.llama import LlamaTP
    from .models.nubosun import Nubosun
    nb, ll = (get_config(n) for n in PAIRS[size])
    m = next(l.mixer for l in nb.layers if isinstance(l.mixer, MambaSpec))
    a = next(l.mixer for l in nb.layers if isinstance(l.mixer, LatentSpec))
    k, W, S, dev = _Kernels(only), nb.hidden_size, nb.streams, "cuda"
    decode = T == seqs
    L = T // seqs
    bf, f32, i32 = torch.bfloat16, torch.float32, torch.int32
    bs = 16
    blocks = (ctx + bs - 1) // bs
    tables = (torch.arange(seqs * blocks, dtype=i32).view(seqs, blocks) + 1).to(dev)
    nslots = (seqs * blocks + 1) * bs
    seq_of_row = torch.arange(seqs, dtype=i32).repeat_interleave(L).to(dev)
    pos = (torch.full((seqs,), ctx - 1, dtype=i32) if decode else torch.arange(L, dtype=i32).repeat(seqs)).to(dev)
    ctx_lens = pos + 1
    slots = (tables[seq_of_row.long(), (pos // bs).long()].long() * bs + pos % bs)
    segs = torch.tensor([[s * L, L, s + 1, 0] for s in range(seqs)], dtype=i32, device=dev)
    pairs_causal = seqs * L * (L + 1) / 2 if not decode else seqs * ctx

    # residual + norm
    def mk_hyper(i):
        x, y, h = torch.zeros(T, S, W, device=dev), torch.zeros(T, W, device=dev), torch.empty(T, W, dtype=bf, device=dev)
        v, c, mx = torch.ones(W, device=dev), torch.ones(S, device=dev), torch.eye(S, device=dev)
        return lambda: ops.hyper_mix(y, v, c, mx, x, c, v, h, W, 1e-5)
    k.time("residual + norm", f"nubosun hyper_mix ({S} streams, fp32)", mk_hyper, T * W * (8 * S + 4 + 2))

    def mk_norm(i):
        x, r, gm = _w(T, W), _w(T, W), _w(W)
        return lambda: ops.add_rmsnorm(x, r, gm, 1e-5)
    k.time("residual + norm", "llama add_rmsnorm (bf16)", mk_norm, T * W * 8)

    # matrix products
    _linear(k, "gemm", "nubosun mamba in", T, 2 * m.inner, W)
    _linear(k, "gemm", "nubosun mamba x (fp32 + copy)", T, _pad16(m.dt_rank + 2 * m.state), m.inner, f32=True, copy=True)
    _linear(k, "gemm", "nubosun mamba dt (fp32)", T, m.inner, _pad16(m.dt_rank), f32=True)
    _linear(k, "gemm", "nubosun mamba out (fp32)", T, W, m.inner, f32=True)
    Dk = _pad16(a.kv_rank) + _pad16(a.rot_dim)
    _linear(k, "gemm", "nubosun latent q + kv", T, a.heads * (a.dim + a.rot_dim) + Dk, W)
    if decode:
        _linear(k, "gemm", "nubosun fold W_uk (grouped)", T, a.kv_rank, a.dim, groups=a.heads)
        _linear(k, "gemm", "nubosun expand W_uv (grouped)", T, a.vdim, a.kv_rank, groups=a.heads)
    else:
        _linear(k, "gemm", "nubosun expand keys / values", T, a.heads * (a.dim + a.vdim), a.kv_rank)
    _linear(k, "gemm", "nubosun latent out (fp32)", T, W, a.heads * a.vdim, f32=True)
    ff = nb.layers[0].mlp.ff
    _linear(k, "gemm", "nubosun gate_up (clamped unit)", T, 2 * ff, W, glu=(7.0, 1.702))
    _linear(k, "gemm", "nubosun down (fp32)", T, W, ff, f32=True)
    _linear(k, "gemm", "nubosun head (softcap, fp32)", min(T, seqs), _pad16(nb.vocab_size), W, f32=True, act=ops.ACT_SOFTCAP)
    D, nq, nkv = ll.head_dim, ll.num_heads, ll.num_kv_heads
    cs = ops.rope_cos_sin(D, 8192, 5e5, dev)

    def mk_qkv(i):
        x, w, qkv = _w(T, W), _w((nq + 2 * nkv) * D, W), torch.empty(T, (nq + 2 * nkv) * D, dtype=bf, device=dev)
        kc, vc = _w(nslots, nkv, D), _w(nslots, nkv, D)
        return lambda: ops.gemm_qkv_rope(x, w, qkv, pos, cs, slots, kc, vc, nq, nkv)
    M = (nq + 2 * nkv) * D
    k.time("gemm", "llama qkv + rope", mk_qkv, (T * W + M * W + T * M + 2 * T * nkv * D) * 2, 2.0 * T * M * W)
    _linear(k, "gemm", "llama out", T, W, nq * D)
    _linear(k, "gemm", "llama gate_up (silu)", T, 2 * ff, W, silu=True)
    _linear(k, "gemm", "llama down", T, W, ff)
    _linear(k, "gemm", "llama head", min(T, seqs), nb.vocab_size, W)

    # selective scan
    ip = _pad16(m.inner)

    def mk_conv(i):
        xz, u = _w(T, 2 * ip), torch.empty(T, ip, dtype=bf, device=dev)
        t, b, st = torch.ones(m.conv, ip, device=dev), torch.zeros(ip, device=dev), torch.zeros(seqs + 1, m.conv - 1, ip, device=dev)
        return lambda: ops.causal_conv_silu(xz, u, t, b, st, segs, seq_of_row, pos)
    k.time("scan", "nubosun convolution", mk_conv, T * ip * 4 + (seqs * (m.conv - 1) * ip * 4 if decode else 0))

    def mk_scan(i):
        xz, u, dt = _w(T, 2 * ip), _w(T, ip), torch.rand(T, ip, device=dev) * 0.1
        pp = _pad16(m.dt_rank + 2 * m.state)
        bc = torch.randn(T, pp, device=dev)
        a2, d = -torch.rand(m.inner, m.state, device=dev), torch.ones(m.inner, device=dev)
        ssm, st = torch.zeros(seqs + 1, m.inner, m.state, device=dev), torch.zeros(seqs + 1, m.conv - 1, ip, device=dev)
        return lambda: ops.selective_scan(u, xz, ip, dt, bc, m.dt_rank, m.dt_rank + m.state, a2, d, ssm, st, u, segs, pos, one_token=decode)
    k.time("scan", "nubosun selective scan", mk_scan, T * ip * 10 + T * m.state * 8 + seqs * m.inner * m.state * (8 if decode else 4) + m.inner * m.state * 4,
           exps=float(T) * m.inner * m.state)

    # attention
    R, rot, H = _pad16(a.kv_rank), _pad16(a.rot_dim), a.heads
    qc = H * (a.dim + rot) + R + rot
    turns = ops.rotation_turns(rot, 1e4, dev)
    nr = T if decode else 0

    def mk_prep(i):
        qkv, qa, cache = _w(T, qc), torch.empty(max(nr, 1), H, Dk + 8, dtype=bf, device=dev), _w(nslots, Dk + 8)
        gm = torch.ones(R, device=dev)
        return lambda: ops.latent_prep(qkv, qkv, qa[:nr], cache, gm, turns, 1.0, pos, slots, nr, H * a.dim, H * (a.dim + rot), H * (a.dim + rot) + R, H, R, R, rot, 1e-5)
    k.time("attention", "nubosun rotation + latent norm + cache write", mk_prep, T * (2 * H * rot + 2 * Dk) * 2)
    sink = torch.zeros(H, device=dev)
    sms = torch.cuda.get_device_properties(0).multi_processor_count

    def splits(units, slots):
        s = 1
        while s < 8 and seqs * units * s * 2 <= slots(s * 2, sms) and ctx // (s * 2) >= 64:
            s *= 2
        return s
    if decode:
        def mk_rows(i):
            qa, cache, o = _w(T, H, Dk + 8), _w(nslots, Dk + 8), torch.empty(T, H, R, dtype=bf, device=dev)
            sp = splits((H + 15) // 16, Nubosun.attn_cta_slots)
            return lambda: ops.latent_attention_rows(qa, cache, tables, seq_of_row, ctx_lens, sink, o, R, a.scale, bs, splits=sp)
        k.time("attention", "nubosun latent attention, rows form", mk_rows, seqs * ctx * Dk * 2 + T * H * (Dk + R) * 2, 2.0 * pairs_causal * H * (Dk + R))

        def mk_paged(i):
            q, kc, vc, o = _w(T, nq, D), _w(nslots, nkv, D), _w(nslots, nkv, D), torch.empty(T, nq, D, dtype=bf, device=dev)
            sp = splits(nkv, LlamaTP.attn_cta_slots)
            return lambda: ops.paged_attention(q, kc, vc, tables, ctx_lens, o, D ** -0.5, bs, splits=sp)
        k.time("attention", "llama paged attention", mk_paged, seqs * ctx * nkv * D * 4 + T * nq * D * 4, 4.0 * pairs_causal * nq * D)
    else:
        tb = tables.cpu().numpy()
        tl, sl = dense_context([s * L for s in range(seqs)], [L] * seqs, [0] * seqs, list(range(seqs)), tb, bs)
        tl, sl = torch.from_numpy(tl).to(dev), torch.from_numpy(sl).to(dev)

        def mk_gather(i):
            cache, c, kr = _w(nslots, Dk + 8), torch.empty(T, R, dtype=bf, device=dev), torch.empty(T, rot, dtype=bf, device=dev)
            return lambda: ops.latent_gather(cache, sl, c, kr)
        k.time("attention", "nubosun gather of the latents", mk_gather, 2 * T * Dk * 2)

        def mk_pre(i):
            qkv, kv, kr = _w(T, qc), _w(T, H * (a.dim + a.vdim)), _w(T, rot)
            o = torch.empty(T, H * a.vdim, dtype=bf, device=dev)
            return lambda: ops.latent_attention_prefill(qkv, H * a.dim, kv, kr, tl, sink, o, H, a.dim, a.vdim, a.scale)
        k.time("attention", "nubosun latent attention, prefill form", mk_pre, T * H * (2 * a.dim + rot + 2 * a.vdim) * 2,
               2.0 * pairs_causal * H * (a.dim + rot + a.vdim))
        tiles = ops.prefill_tiles(seq_of_row.cpu(), nq // nkv).to(dev)

        def mk_lpre(i):
            q, kc, vc, o = _w(T, nq, D), _w(nslots, nkv, D), _w(nslots, nkv, D), torch.empty(T, nq, D, dtype=bf, device=dev)
            return lambda: ops.prefill_attention(q, kc, vc, tables, ctx_lens, seq_of_row, tiles, o, D ** -0.5, bs)
        k.time("attention", "llama prefill attention", mk_lpre, T * nq * D * 4 + T * nkv * D * 4, 4.0 * pairs_causal * nq * D)
    return k.rows


CASES = {"decode 8 rows, 640 cached tokens": (8, 8, 640), "decode 32 rows, 640 cached tokens": (32, 32, 640),
         "decode 32 rows, 8192 cached tokens": (32, 32, 8192),
         "prefill 8 x 512": (4096, 8, 512), "prefill 1 x 4096": (4096, 1, 4096)}


def run(sizes, kernels=True, models=True, only="", case="") -> dict:
    out = {"bench": "nubosun beside llama", "data": "synthetic (random token ids, random weights)", "dtype": "bf16", "sizes": {}}
    for s in sizes:
        r = out["sizes"][s] = {}
        if models:
            r["models"] = [model_numbers(n) for n in PAIRS[s]]
        if kernels:
            r["kernels"] = {c: kernel_numbers(s, *v, only=only) for c, v in CASES.items() if case in c}
    return out


def main(run=run, doc=__doc__) -> int:
    ap = argparse.ArgumentParser(description=doc, formatter_class=argparse.RawDescriptionHelpFormatter)
    ap.add_argument("--sizes", default="2k,8b")
    ap.add_argument("--no-kernels", action="store_true")
    ap.add_argument("--no-models", action="store_true")
    ap.add_argument("--only", default="", help="kernels whose name contains this")
    ap.add_argument("--case", default="", help="cases whose name contains this")
    ap.add_argument("--table", action="store_true", help="print kernel rows as text")
    a = ap.parse_args()
    r = run(a.sizes.split(","), not a.no_kernels, not a.no_models, a.only, a.case)
    if a.table:
        for s, v in r["sizes"].items():
            for m in v.get("models", []):
                print(s, json.dumps(m))
            for case, rows in v.get("kernels", {}).items():
                print(f"-- {s}: {case}")
                for x in rows:
                    print(f"{x['group']:16s} {x['kernel']:48s} {x['us']:9.2f} us  roofline {x['roofline_us']:8.2f}  {x['of_measured_peak']:.3f}")
    else:
        print(json.dumps(r))
    return 0


if __name__ == "__main__":
    raise SystemExit(main())
