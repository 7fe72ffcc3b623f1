#!/usr/bin/env python3
"""Lugizen beside the closest other models (Tinapel, Nubosun, Llama) at equal width, depth, heads, vocabulary and feed-forward weights per token: prefill and
decode throughput through the engine, and every kernel of the designs at the same shapes against its roofline.

    python bench.py --compare lugizen [--sizes 2k,8b]          (or: python -m libtbvcoll_b200.bench_lugizen)

Timing as in ``bench_nubosun``.  Roofline of the delta rule: its bytes, or four fp32 instructions per state element and token (decay, both readouts, rank-one
update; three in the recurrences without the delta) at 128 per clock and SM.  Attention is charged for the visible keys only, experts for the weights of those that
have rows."""
from __future__ import annotations

import torch

from . import bench_nubosun, bench_tinapel
from .bench_bobarax import visible_pairs
from .bench_nubosun import CASES, _Kernels, _linear, _pad16, _w, model_numbers

MODELS = {"2k": ("lugizen-2k", "tinapel-2k", "nubosun-2k", "llama3-2k"), "8b": ("lugizen-8b", "tinapel-8b", "nubosun-8b", "llama3-8b")}


def kernel_numbers(size: str, T: int, seqs: int, ctx: int, only: str = "") -> list:
    """T rows in ``seqs`` sequences: T == seqs is a decode step over ``ctx`` cached tokens, otherwise whole prompts."""
    from . import ops
    from .engine.batch import dense_context, scan_groups
    from .models.config import ChannelDeltaSpec, GeluMlpSpec, HeadAttentionSpec, LatentSpec, MoeSpec, get_config
    from .models.lugizen import Lugizen
    cfg = get_config(MODELS[size][0])
    of = lambda kind, part: next(getattr(l, part) for l in cfg.layers if isinstance(getattr(l, part), kind))
    r, a, la, dense, f = of(ChannelDeltaSpec, "mixer"), of(HeadAttentionSpec, "mixer"), of(LatentSpec, "mixer"), of(GeluMlpSpec, "mlp"), of(MoeSpec, "mlp")
    k, W, dev, decode, L = _Kernels(only), cfg.hidden_size, "cuda", T == seqs, T // seqs
    bf, i32 = torch.bfloat16, torch.int32
    bs, taps = 16, cfg.canon_taps
    blocks = (ctx + bs - 1) // bs
    tables = (torch.arange(seqs * blocks, dtype=i32).view(seqs, blocks) + 1).to(dev)
    nblocks = seqs * blocks + 1
    seq_of_row = torch.arange(seqs, dtype=i32).repeat_interleave(L).to(dev)
    positions = [ctx - 1] * seqs if decode else list(range(L)) * seqs
    pos = torch.tensor(positions, dtype=i32, device=dev)
    slots = (tables[seq_of_row.long(), (pos // bs).long()].long() * bs + pos % bs)
    segs = torch.tensor([[s * L, L, s + 1, 0] for s in range(seqs)], dtype=i32, device=dev)
    ones = lambda *s: torch.ones(*s, device=dev)
    zeros = lambda *s: torch.zeros(*s, device=dev)
    empty = lambda *s: torch.empty(*s, dtype=bf, device=dev)
    E, fp, P = f.experts, _pad16(f.ff), T * f.top
    place = torch.stack([torch.randperm(P, device=dev)[:T] for _ in range(f.top)], 1).to(i32).contiguous()
    model = Lugizen.__new__(Lugizen)                   # its choices only
    model.dtype, model.scan_heads, model.device, model.sms = bf, r.heads, dev, torch.cuda.get_device_properties(0).multi_processor_count

    # between sublayers
    def mk_residual(experts, to):
        def mk(i):
            x, y, ro, g, h = zeros(T, W), zeros(T, W), _w(P, W), ones(W), empty(T, W)
            past, w = zeros(seqs + 1, taps - 1, W), ones(taps, W)
            branch = dict(routed=(ro, place, ones(T, f.top))) if experts else dict(y1=y)
            if to == "ff":
                return lambda: ops.residual(x, None, h, W, 1e-5, post=g, **branch)
            if decode:
                return lambda: ops.residual(x, None, h, W, 1e-5, post=g, positions=pos, conv=(w, past, segs), **branch)
            return lambda: ops.residual(x, None, None, W, 1e-5, post=g, **branch)
        return mk
    state = seqs * (taps - 1) * W * 8
    k.time("residual + norm", "lugizen residual (branch norm, to the feed-forward)", mk_residual(False, "ff"), T * W * (8 + 4 + 2))
    for name, experts in (("dense", False), ("experts", True)):
        k.time("residual + norm", f"lugizen residual (from {name}, {'convolution' if decode else 'stream only'})", mk_residual(experts, "mixer"),
               T * W * (8 + (2 * f.top if experts else 4) + (2 if decode else 0)) + (state if decode else 0))
    if not decode:
        def mk_stream_conv(i):
            x, h, past, w = zeros(T, W), empty(T, W), zeros(seqs + 1, taps - 1, W), ones(taps, W)
            return lambda: ops.short_conv(x, h, w, past, segs, seq_of_row, pos, add=True)
        k.time("residual + norm", "lugizen convolution of the stream", mk_stream_conv, T * W * (4 + 2))

    # matrix products
    G, H, D, V, R = r.kv_heads, r.heads, _pad16(r.dim), _pad16(r.vdim), _pad16(max(r.decay_rank, r.gate_rank))
    K, C = G * D, 2 * G * D + H * V
    X = C + 2 * R + _pad16(H)
    _linear(k, "gemm", "lugizen delta q, k, v, decay, gate, step", T, X, W)
    if not decode:
        _linear(k, "gemm", "lugizen decay second (softplus, fp32)", T, H * D, R, f32=True, act=ops.ACT_SOFTPLUS)
        _linear(k, "gemm", "lugizen gate second", T, H * V, R)
    Da, Va = _pad16(a.dim), _pad16(a.vdim)
    _linear(k, "gemm", "lugizen attention q, k, v", T, (a.heads + a.kv_heads) * Da + a.kv_heads * Va, W)
    Rk, Rq, rot, Hl, Dl, Vl = _pad16(la.kv_rank), _pad16(la.q_rank), _pad16(la.rot_dim), la.heads, _pad16(la.dim), _pad16(la.vdim)
    _linear(k, "gemm", "lugizen latent down", T, Rq + Rk + rot, W)
    _linear(k, "gemm", "lugizen latent queries", T, Hl * (Dl + rot), Rq)
    if decode:
        _linear(k, "gemm", "lugizen fold W_uk (grouped)", T, Rk, Dl, groups=Hl)
        _linear(k, "gemm", "lugizen expand W_uv (grouped)", T, Vl, Rk, groups=Hl)
    else:
        _linear(k, "gemm", "lugizen expand keys / values", T, Hl * (Dl + Vl), Rk)
    _linear(k, "gemm", "lugizen mixer out (fp32)", T, W, H * V, f32=True)

    def mk_up(i):
        x, w, out = _w(T, W), _w(dense.ff, W), empty(T, dense.ff)
        return lambda: ops.linear(x, w, out, act=ops.ACT_GELU, act_cols=dense.ff)
    k.time("gemm", "lugizen dense up (gelu)", mk_up, (T * W + dense.ff * (W + T)) * 2, 2.0 * T * dense.ff * W)
    _linear(k, "gemm", "lugizen dense down (fp32)", T, W, dense.ff, f32=True)
    _linear(k, "gemm", "lugizen head (fp32)", min(T, seqs), _pad16(cfg.vocab_size), W, f32=True)

    # recurrence
    args = dict(kv_heads=G, dim=r.dim, vdim=r.vdim, eps=1e-5)
    conv_state = (r.conv - 1) * C * 4

    def mk_conv(i):
        wide, out, st, w = _w(T, X), empty(T, C), zeros(seqs + 1, r.conv - 1, C), ones(r.conv, C)
        return lambda: ops.short_conv(wide, out, w, st, segs, seq_of_row, pos)

    def mk_rec(i):
        wide, st, out, norm, rate = _w(T, X), zeros(seqs + 1, H, D, V), empty(T, H * V), ones(V), ones(H)
        if decode:
            w_a, b_a, w_g, past, w = _w(H * D, R), _w(H * D), _w(H * V, R), zeros(seqs + 1, r.conv - 1, C), ones(r.conv, C)
            q, kk, v, low_a, low_g, beta = wide.split((K, K, H * V, R, R, _pad16(H)), 1)
            return lambda: ops.delta_step(q, kk, v, beta, low_a, low_g, w_a, b_a, w_g, rate, norm, st, out, segs, pos, conv=(w, past), **args)
        q, kk, v = _w(T, C).split((K, K, H * V), 1)
        z, gate, o, beta = torch.rand(T, H * D, device=dev) * 0.1, _w(T, H * V), zeros(T, H * V), wide[:, C + 2 * R:]
        gr = torch.from_numpy(scan_groups(segs.cpu().numpy(), model.scan_group_rows(segs[:, 1].cpu().numpy()))).to(dev)
        size = ops.delta_sets(T, seqs, st)
        sets = torch.empty(size, dtype=torch.uint8, device=dev) if size else None
        return lambda: ops.delta_scan(q, kk, v, beta, z, gate, rate, norm, st, o, out, segs, pos, groups=gr, sets=sets, **args)
    matrix = seqs * H * D * V * 4
    if decode:
        k.time("scan", "lugizen delta step (convolution, products, norm, gate)", mk_rec,
               2 * matrix + 2 * seqs * conv_state + T * (C + 2 * R + H + H * V) * 2 + H * (D + V) * R * 2 + r.conv * C * 4)
    else:
        k.time("scan", "lugizen convolution of q, k, v", mk_conv, T * C * 4)
        k.time("scan", "lugizen delta recurrence (norm, gate)", mk_rec, matrix + T * (C + 2 * H * V) * 2 + T * H * D * 4, fp32=4.0 * T * H * D * V)

    # attention
    nr, seen = T if decode else 0, visible_pairs(positions, 0, 1 << 30)
    most = 1                                           # CTAs per row as the engine would hand them out
    while most < 8 and ctx // (most * 2) >= 64:
        most *= 2
    Ha, Ga, cols = a.heads, a.kv_heads, (a.heads + a.kv_heads) * Da + a.kv_heads * Va
    turns, ltable = ops.rotation_turns(a.rot.dims, a.rot.base, dev), ops.rotation_turns(la.rot.dims, la.rot.base, dev)

    def mk_prep(i):
        wide, qa, cache, first, lam = _w(T, cols), empty(max(nr, 1), Ha, Da + 8), _w(nblocks * Ga * bs, Da + Va + 8), _w(T, Ga * Va), ones(1)
        qs = ones(Ha)
        return lambda: ops.head_attention_prep(wide, qa[:nr], cache, qs, turns, pos, slots, nr, Ha, Ga, a.dim, Da, bs, 1e-5, v_first=first, mix=lam)
    k.time("attention", "lugizen norms + rotation + value mix + cache write", mk_prep, T * 2 * ((Ha + Ga) * Da * 2 + Ga * Va * 3))
    Dk, lcols = Rk + rot, Rq + Rk + rot

    def mk_lprep(i):
        low, cache, g, gq = _w(T, lcols), _w(nblocks * bs, Dk + 8), ones(la.kv_rank), ones(la.q_rank)
        return lambda: ops.latent_prep(low, None, None, cache, g, ltable, 1.0, pos, slots, nr, 0, Rq, Rq + Rk, Hl, la.kv_rank, Rk, rot, 1e-5, query_latent=(0, la.q_rank, gq))

    def mk_qprep(i):
        q, qa, cache = _w(T, Hl * (Dl + rot)), empty(max(nr, 1), Hl, Dk + 8), _w(nblocks * bs, Dk + 8)
        return lambda: ops.latent_prep(None, q, qa[:nr], cache, None, ltable, 1.0, pos, slots, nr, Hl * Dl, 0, 0, Hl, la.kv_rank, Rk, rot, 1e-5)
    k.time("attention", "lugizen latent norms + key rotation + cache write", mk_lprep, T * 2 * (2 * Rq + 2 * Dk))
    k.time("attention", "lugizen latent query rotation", mk_qprep, T * 2 * 2 * Hl * rot)
    lseen = visible_pairs(positions, la.window, 0)
    if decode:
        ctx_lens = pos + 1

        def mk_rows(i):
            qa, cache, o = _w(T, Ha, Da + 8), _w(nblocks * Ga * bs, Da + Va + 8), empty(T, Ha, Va)
            sp = model.layer_splits(a, T, most)
            return lambda: ops.paired_attention_rows(qa, cache, tables, seq_of_row, ctx_lens, o, Ga, bs, splits=sp)
        k.time("attention", "lugizen attention, rows form", mk_rows, seen * Ga * (Da + Va) * 2 + T * Ha * (Da + Va) * 2, 2.0 * seen * Ha * (Da + Va))

        def mk_lrows(i):
            qa, cache, o = _w(T, Hl, Dk + 8), _w(nblocks * bs, Dk + 8), empty(T, Hl, Rk)
            sp = model.layer_splits(la, T, most)
            return lambda: ops.latent_attention_rows(qa, cache, tables, seq_of_row, ctx_lens, None, o, la.kv_rank, la.scale, bs, splits=sp, window=la.window)
        k.time("attention", "lugizen latent attention, rows form", mk_lrows, lseen * Dk * 2 + T * Hl * (Dk + Rk) * 2, 2.0 * lseen * Hl * (Dk + Rk))
    else:
        host = tables.cpu().numpy()
        tl, sl = dense_context([s * L for s in range(seqs)], [L] * seqs, [0] * seqs, list(range(seqs)), host, bs, la.window)
        tl, sl = torch.from_numpy(tl).to(dev), torch.from_numpy(sl).to(dev)

        def mk_pre(i):
            wide, cache, o = _w(T, cols), _w(nblocks * Ga * bs, Da + Va + 8), empty(T, Ha * Va)
            return lambda: ops.paired_attention_prefill(wide, cache, tables, seq_of_row, tl, o, Ha, Ga, Da, bs)
        k.time("attention", "lugizen attention, prefill form", mk_pre, T * ((Ha + Ga) * Da + (Ga + Ha) * Va) * 2, 2.0 * seen * Ha * (Da + Va))

        def mk_gather(i):
            cache, c, kr = _w(nblocks * bs, Dk + 8), empty(len(sl), Rk), empty(len(sl), rot)
            return lambda: ops.latent_gather(cache, sl, c, kr)
        k.time("attention", "lugizen gather of the latents", mk_gather, 2 * T * Dk * 2)

        def mk_lpre(i):
            q, kv, kr, o = _w(T, Hl * (Dl + rot)), _w(len(sl), Hl * (Dl + Vl)), _w(len(sl), rot), empty(T, Hl * Vl)
            return lambda: ops.latent_attention_prefill(q, Hl * Dl, kv, kr, tl, None, o, Hl, Dl, Vl, la.scale, la.window)
        k.time("attention", "lugizen latent attention, prefill form", mk_lpre, T * Hl * (2 * Dl + rot + 2 * Vl) * 2, 2.0 * lseen * Hl * (Dl + rot + Vl))

    # mixture of experts
    _linear(k, "experts", "lugizen router (fp32)", T, _pad16(E), W, f32=True)
    logits = torch.randn(T, _pad16(E), device=dev)
    pl, wt, off = torch.empty(T, f.top, dtype=i32, device=dev), zeros(T, f.top), torch.zeros(E + 1, dtype=i32, device=dev)
    cnt, ch = torch.zeros(E, dtype=i32, device=dev), torch.zeros(2 * P, dtype=i32, device=dev)

    def mk_route(i):
        h, xp = _w(T, W), empty(P, W)
        return lambda: ops.moe_route(logits, h, xp, pl, wt, off, cnt, ch, E, 1.0)
    k.time("experts", "lugizen choice + dispatch", mk_route, T * W * 2 * (1 + f.top))
    ops.moe_route(logits, _w(T, W), empty(P, W), pl, wt, off, cnt, ch, E, 1.0)
    active = int((off[1:] > off[:-1]).sum())

    def mk_rows_gemm(M, Kc, glu):
        def mk(i):
            x, w, out = _w(P, Kc), _w(E * M, Kc), empty(P, M // 2 if glu else M)
            return lambda: ops.linear_rows(x, w, out, off, E, T, glu=ops.SILU_GLU if glu else None)
        return mk
    k.time("experts", "lugizen experts gate_up (silu)", mk_rows_gemm(2 * fp, W, True), (P * W + active * 2 * fp * W + P * fp) * 2, 4.0 * P * fp * W)
    k.time("experts", "lugizen experts down", mk_rows_gemm(W, fp, False), (P * fp + active * fp * W + P * W) * 2, 2.0 * P * fp * W)
    return k.rows


def run(sizes, kernels=True, models=True, only="", case="") -> dict:
    out = {"bench": "lugizen beside tinapel, nubosun and llama", "data": "synthetic (random token ids, random weights)", "dtype": "bf16", "sizes": {}}
    for s in sizes:
        r = out["sizes"][s] = {}
        if models:
            r["models"] = [model_numbers(n) for n in MODELS[s]]
        if kernels:
            r["kernels"] = {c: sum((m.kernel_numbers(s, *v, only=only) for m in (bench_tinapel, bench_nubosun)), kernel_numbers(s, *v, only=only))
                            for c, v in CASES.items() if case in c}
    return out


if __name__ == "__main__":
    raise SystemExit(bench_nubosun.main(run, __doc__))
