#!/usr/bin/env python3
"""Tinapel beside the closest other models (Nubosun, Llama) at equal width, depth, heads, vocabulary and feed-forward weights per token: prefill
and decode throughput through the engine, and every kernel of the designs at the same shapes against its roofline.

    python bench.py --compare tinapel [--sizes 2k,8b]          (or: python -m libtbvcoll_b200.bench_tinapel)

Timing as in ``bench_nubosun``.  Roofline of the matrix-state recurrence: its bytes, or three fp32 instructions per state element and token
(decay product, rank-one update, readout) at 128 per clock and SM.  Weight bytes of experts are those of the experts that have rows."""
from __future__ import annotations

import torch

from . import bench_nubosun
from .bench_nubosun import CASES, _Kernels, _linear, _pad16, _w, model_numbers

TRIPLES = {"2k": ("tinapel-2k", "nubosun-2k", "llama3-2k"), "8b": ("tinapel-8b", "nubosun-8b", "llama3-8b")}


def kernel_numbers(size: str, T: int, seqs: int, ctx: int, only: str = "") -> list:
    """T rows in ``seqs`` sequences: T == seqs is a decode step over ``ctx`` cached tokens, otherwise whole prompts."""
    from . import ops
    from .engine.batch import dense_context, scan_groups
    from .models.config import GlaSpec, SharedKvSpec, get_config
    from .models.tinapel import Tinapel
    cfg = get_config(TRIPLES[size][0])
    r = next(l.mixer for l in cfg.layers if isinstance(l.mixer, GlaSpec))
    a = next(l.mixer for l in cfg.layers if isinstance(l.mixer, SharedKvSpec))
    f = cfg.layers[0].mlp
    k, W, dev, decode, L = _Kernels(only), cfg.hidden_size, "cuda", T == seqs, T // seqs
    bf, i32 = torch.bfloat16, torch.int32
    bs = 16
    blocks = (ctx + bs - 1) // bs
    tables = (torch.arange(seqs * blocks, dtype=i32).view(seqs, blocks) + 1).to(dev)
    nblocks = seqs * blocks + 1
    seq_of_row = torch.arange(seqs, dtype=i32).repeat_interleave(L).to(dev)
    pos = (torch.full((seqs,), ctx - 1, dtype=i32) if decode else torch.arange(L, dtype=i32).repeat(seqs)).to(dev)
    slots = (tables[seq_of_row.long(), (pos // bs).long()].long() * bs + pos % bs)
    segs = torch.tensor([[s * L, L, s + 1, 0] for s in range(seqs)], dtype=i32, device=dev)
    pairs_causal = seqs * L * (L + 1) / 2 if not decode else seqs * ctx
    ones = lambda *s: torch.ones(*s, device=dev)
    zeros = lambda *s: torch.zeros(*s, device=dev)
    place = torch.stack([torch.randperm(T * f.top, device=dev)[:T] for _ in range(f.top)], 1).to(i32).contiguous()

    def mk_residual(i):
        x, y1, y2, ro = zeros(T, W), zeros(T, W), zeros(T, W), _w(T * f.top, W)
        h1, h2, g, wt = torch.empty(T, W, dtype=bf, device=dev), torch.empty(T, W, dtype=bf, device=dev), ones(W), ones(T, f.top)
        return lambda: ops.residual(x, g, h1, W, 1e-5, g2=g, h2=h2, y1=y1, y2=y2, routed=(ro, place, wt))
    k.time("residual + norm", "tinapel residual (branches, experts, both norms)", mk_residual, T * W * (16 + 4 + 2 * f.top))

    # mixers' products
    K, V, R = r.heads * _pad16(r.dim), r.heads * _pad16(r.vdim), _pad16(r.decay_rank)
    _linear(k, "gemm", "tinapel gla q, k, v, gate, decay", T, 2 * K + 2 * V + R, W)
    if decode:
        def mk_mix_gemm(i):
            x, w, out = _w(T, 5 * W), _w(4 * K + R, W), torch.empty(T, 4 * K + R, dtype=bf, device=dev)
            return lambda: ops.linear(x, w, out, groups=4, x_group=W, y_group=K, last=R)
        k.time("gemm", "tinapel wkv r, k, v, gate, decay (grouped)", mk_mix_gemm, (T * 5 * W + (4 * K + R) * W + T * (4 * K + R)) * 2, 2.0 * T * (4 * K + R) * W)
    else:
        _linear(k, "gemm", "tinapel wkv r / k / v / gate, each", T, K, W)
        _linear(k, "gemm", "tinapel decay first (tanh, fp32 + copy)", T, R, W, f32=True, act=ops.ACT_SOFTCAP, copy=True)
    _linear(k, "gemm", "tinapel attention q + k", T, (a.heads + a.kv_heads) * a.dim, W)
    _linear(k, "gemm", "tinapel mixer out (fp32)", T, W, V, f32=True)
    _linear(k, "gemm", "tinapel head (fp32)", min(T, seqs), _pad16(cfg.vocab_size), W, f32=True)

    # recurrence
    if not decode:
        def mk_shift(i):
            h, mu, st, mixes = zeros(T, W), zeros(5, W), zeros(seqs + 1, W), torch.empty(T, 5 * W, dtype=bf, device=dev)
            return lambda: ops.token_shift(h, mu, st, mixes, segs, seq_of_row, pos)
        k.time("scan", "tinapel mixes with the previous token", mk_shift, T * W * (4 + 10))
    for name, u in (("gla", None), ("wkv", zeros(K))):
        def mk_rec(i):
            wide, st, out, norm = _w(T, 2 * K + 2 * V + R), zeros(seqs + 1, r.heads, _pad16(r.dim), _pad16(r.vdim)), torch.empty(T, V, dtype=bf, device=dev), ones(V)
            q, kk, v, g, low = wide.split((K, K, V, V, R), 1)
            if decode:
                w2, b2 = _w(K, R), _w(K)
                return lambda: ops.decay_step(q, kk, v, g, low, w2, b2, norm, st, out, segs, pos, vdim=r.vdim, eps=1e-5, tau=16.0, u=u)
            model = Tinapel.__new__(Tinapel)           # its choice of groups only
            model.dtype, model.scan_heads, model.device = bf, r.heads, dev
            gr = scan_groups(segs.cpu().numpy(), model.scan_group_rows(segs[:, 1].cpu().numpy()))
            cut, gr = len(gr) > seqs, torch.from_numpy(gr).to(dev)
            scratch = (torch.empty(len(gr) * K * _pad16(r.vdim), device=dev), torch.empty(len(gr) * K, device=dev)) if cut else None
            w2, b2, o = _w(K, R), _w(K), torch.empty(T, V, device=dev)
            return lambda: ops.decay_scan(q, kk, v, g, None, norm, st, o, out, segs, pos, vdim=r.vdim, eps=1e-5, tau=16.0, u=u, groups=gr, scratch=scratch, low=(low, w2, b2))
        state = seqs * K * r.vdim * 4
        if decode:
            k.time("scan", f"tinapel {name} step (decay product, norm, gate)", mk_rec, 2 * state + T * (2 * K + 3 * V + R) * 2 + K * R * 2)
        else:
            k.time("scan", f"tinapel {name} recurrence (decay product, norm, gate)", mk_rec, state + T * (2 * K + 3 * V + R) * 2 + K * R * 2, fp32=3.0 * T * K * r.vdim)

    # attention
    H, G, D = a.heads, a.kv_heads, _pad16(a.dim)
    nr = T if decode else 0

    def mk_prep(i):
        qk, qa, cache, fold = _w(T, (H + G) * D), torch.empty(max(nr, 1), H, D + 8, dtype=bf, device=dev), _w(nblocks * G * bs, D + 8), ones(D)
        return lambda: ops.shared_attention_prep(qk, qa[:nr], cache, fold, pos, slots, nr, H, G, a.dim, bs, 1e-5, 0.1, 4096)
    k.time("attention", "tinapel norms + temperature + cache write", mk_prep, T * 2 * (H + G) * D * 2)
    if decode:
        sms, sp = torch.cuda.get_device_properties(0).multi_processor_count, 1
        units = G * ((H // G + 15) // 16)
        while sp < 8 and seqs * units * sp * 2 <= Tinapel.attn_cta_slots(sp * 2, sms) and ctx // (sp * 2) >= 64:
            sp *= 2

        def mk_rows(i):
            qa, cache, o = _w(T, H, D + 8), _w(nblocks * G * bs, D + 8), torch.empty(T, H, D, dtype=bf, device=dev)
            return lambda: ops.shared_attention_rows(qa, cache, tables, seq_of_row, ctx_lens, o, G, bs, 50.0, splits=sp)
        ctx_lens = pos + 1
        k.time("attention", "tinapel attention, rows form", mk_rows, seqs * ctx * G * (D + 2) * 2 + T * H * D * 4, 4.0 * pairs_causal * H * D)
    else:
        tl, _ = dense_context([s * L for s in range(seqs)], [L] * seqs, [0] * seqs, list(range(seqs)), tables.cpu().numpy(), bs)
        tl = torch.from_numpy(tl).to(dev)

        def mk_pre(i):
            qk, cache, o = _w(T, (H + G) * D), _w(nblocks * G * bs, D + 8), torch.empty(T, H * D, dtype=bf, device=dev)
            return lambda: ops.shared_attention_prefill(qk, cache, tables, seq_of_row, tl, o, H, G, bs, 50.0)
        k.time("attention", "tinapel attention, prefill form", mk_pre, T * (2 * H + G) * D * 2, 4.0 * pairs_causal * H * D)

    # mixture of experts
    E, fp, P = f.experts, _pad16(f.ff), T * f.top
    _linear(k, "experts", "tinapel router (fp32)", T, _pad16(E), W, f32=True)
    logits = torch.randn(T, _pad16(E), device=dev)
    pl, wt, off = torch.empty(T, f.top, dtype=i32, device=dev), zeros(T, f.top), torch.zeros(E + 1, dtype=i32, device=dev)
    cnt, ch = torch.zeros(E, dtype=i32, device=dev), torch.zeros(2 * P, dtype=i32, device=dev)

    def mk_route(i):
        h, xp = _w(T, W), torch.empty(P, W, dtype=bf, device=dev)
        return lambda: ops.moe_route(logits, h, xp, pl, wt, off, cnt, ch, E, 1.0)
    k.time("experts", "tinapel choice + dispatch", mk_route, T * W * 2 * (1 + f.top))
    ops.moe_route(logits, _w(T, W), torch.empty(P, W, dtype=bf, device=dev), pl, wt, off, cnt, ch, E, 1.0)
    active = int((off[1:] > off[:-1]).sum())

    def mk_rows_gemm(M, Kc, glu):
        def mk(i):
            x, w, out = _w(P, Kc), _w(E * M, Kc), torch.empty(P, M // 2 if glu else M, dtype=bf, device=dev)
            return lambda: ops.linear_rows(x, w, out, off, E, T, glu=ops.SILU_GLU if glu else None)
        return mk
    k.time("experts", "tinapel experts gate_up (silu)", mk_rows_gemm(2 * fp, W, True), (P * W + active * 2 * fp * W + P * fp) * 2, 4.0 * P * fp * W)
    k.time("experts", "tinapel experts down", mk_rows_gemm(W, fp, False), (P * fp + active * fp * W + P * W) * 2, 2.0 * P * fp * W)
    _linear(k, "experts", "tinapel shared gate_up (silu)", T, 2 * f.shared_ff, W, glu=ops.SILU_GLU)
    _linear(k, "experts", "tinapel shared down (fp32)", T, W, f.shared_ff, f32=True)
    return k.rows


def run(sizes, kernels=True, models=True, only="", case="") -> dict:
    out = {"bench": "tinapel beside nubosun and llama", "data": "synthetic (random token ids, random weights)", "dtype": "bf16", "sizes": {}}
    for s in sizes:
        r = out["sizes"][s] = {}
        if models:
            r["models"] = [model_numbers(n) for n in TRIPLES[s]]
        if kernels:
            r["kernels"] = {c: kernel_numbers(s, *v, only=only) + bench_nubosun.kernel_numbers(s, *v, only=only) for c, v in CASES.items() if case in c}
    return out


if __name__ == "__main__":
    raise SystemExit(bench_nubosun.main(run, __doc__))
