#!/usr/bin/env python3
"""Bobarax beside the closest other models (Tinapel, Llama) at equal width, depth, heads, vocabulary and feed-forward weights per token: prefill and
decode throughput through the engine, and every kernel of the designs at the same shapes against its roofline.

    python bench.py --compare bobarax [--sizes 2k,8b]          (or: python -m libtbvcoll_b200.bench_bobarax)

Timing as in ``bench_nubosun``.  Attention is charged for the visible keys only; the recurrence for its bytes, or the products of its chunked form (one per operand
pair, however many parts an operand has).  Weight bytes of experts are those of the experts that have rows."""
from __future__ import annotations

import torch

from . import bench_nubosun, bench_tinapel
from .bench_nubosun import CASES, _Kernels, _linear, _pad16, _w, model_numbers

TRIPLES = {"2k": ("bobarax-2k", "tinapel-2k", "llama3-2k"), "8b": ("bobarax-8b", "tinapel-8b", "llama3-8b")}


def visible_pairs(positions, window: int, chunk: int) -> int:
    """(query, key) pairs of queries at the given positions."""
    if window:
        return sum(min(p + 1, window) for p in positions)
    return sum(p % chunk + 1 if chunk else p + 1 for p in positions)


def kernel_numbers(size: str, T: int, seqs: int, ctx: int, only: str = "") -> list:
    """T rows in ``seqs`` sequences: T == seqs is a decode step over ``ctx`` cached tokens, otherwise whole prompts."""
    from . import ops
    from .engine.batch import dense_context, scan_groups
    from .models.bobarax import Bobarax
    from .models.config import GatedMlpSpec, LightningSpec, TableMoeSpec, get_config
    cfg = get_config(TRIPLES[size][0])
    r = next(l.mixer for l in cfg.layers if isinstance(l.mixer, LightningSpec))
    attns = [next(l.mixer for l in cfg.layers if getattr(l.mixer, kind, 0)) for kind in ("window", "chunk")]
    ff = next(l.mlp.ff for l in cfg.layers if isinstance(l.mlp, GatedMlpSpec))
    f = next(l.mlp for l in cfg.layers if isinstance(l.mlp, TableMoeSpec))
    k, W, dev, decode, L = _Kernels(only), cfg.hidden_size, "cuda", T == seqs, T // seqs
    bf, i32 = torch.bfloat16, torch.int32
    bs = 16
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

    # experts' places
    ids, offsets = torch.randint(0, cfg.vocab_size, (T,), device=dev), torch.zeros(E + 1, dtype=i32, device=dev)
    table = torch.rand(cfg.vocab_size, E, device=dev).argsort(1)[:, : f.top].to(i32).contiguous()
    place = torch.zeros(T, f.top, dtype=i32, device=dev)
    n_moe = sum(isinstance(l.mlp, TableMoeSpec) for l in cfg.layers)
    layers = [(table, place, offsets, E)] + [(table, torch.zeros_like(place), torch.zeros_like(offsets), E) for _ in range(n_moe - 1)]
    records = ops.moe_table_layers(layers, dev)
    k.time("experts", f"bobarax places of {n_moe} mixtures", lambda i: lambda: ops.moe_place_table(ids, records, E, cfg.vocab_size), n_moe * P * 8)
    ops.moe_place_table(ids, records, E, cfg.vocab_size)
    active = int((offsets[1:] > offsets[:-1]).sum())

    # between sublayers
    def mk_residual(joint, experts):
        def mk(i):
            x, y, ro, g = zeros(T, W), zeros(T, W), _w(P, W), ones(W)
            h, sums = empty(P if experts == "to" else T, W), ones(T, r.heads)
            if experts == "from":
                return lambda: ops.residual(x, g, h, W, 1e-5, post=g, routed=(ro, place, 1.0 / f.top))
            return lambda: ops.residual(x, g, h, W, 1e-5, post=g, y1=y, sums=(sums, r.heads * r.vdim) if joint else None, place=place if experts else None)
        return mk
    k.time("residual + norm", "bobarax residual (branch norm, next norm)", mk_residual(False, None), T * W * (8 + 4 + 2))
    k.time("residual + norm", "bobarax residual (joint norm, to experts' rows)", mk_residual(True, "to"), T * W * (8 + 4 + 2 * f.top))
    k.time("residual + norm", "bobarax residual (from experts' rows)", mk_residual(False, "from"), T * W * (8 + 2 * f.top + 2))

    # matrix products
    K, V = r.heads * _pad16(r.dim), r.heads * _pad16(r.vdim)

    def mk_in(i):
        x, w, out = _w(T, W), _w(2 * K + 2 * V, W), empty(T, 2 * K + 2 * V)
        return lambda: ops.linear(x, w, out, act=ops.ACT_SILU, act_cols=2 * K + V)
    k.time("gemm", "bobarax lightning q, k, v, gate (silu)", mk_in, (T * W + (2 * K + 2 * V) * (W + T)) * 2, 2.0 * T * (2 * K + 2 * V) * W)
    for a in attns:
        D, Va, H, G = _pad16(a.dim), _pad16(a.vdim), a.heads, a.kv_heads
        _linear(k, "gemm", f"bobarax {'window' if a.window else 'chunk'} attention in", T, H * D + G * (D + Va) + (H * Va if a.gated else 0), W)
    _linear(k, "gemm", "bobarax mixer out (fp32)", T, W, V, f32=True)
    _linear(k, "gemm", "bobarax dense gate_up (relu)", T, 2 * ff, W, glu=ops.RELU_GLU)
    _linear(k, "gemm", "bobarax dense down (fp32)", T, W, ff, f32=True)
    _linear(k, "gemm", "bobarax head (fp32)", min(T, seqs), _pad16(cfg.vocab_size), W, f32=True)

    def mk_rows_gemm(M, Kc, glu):
        def mk(i):
            x, w, out = _w(P, Kc), _w(E * M, Kc), empty(P, M // 2 if glu else M)
            return lambda: ops.linear_rows(x, w, out, offsets, E, T, glu=(f.limit, f.slope, 1.0) if glu else None)
        return mk
    k.time("experts", "bobarax experts gate_up (clamped unit)", mk_rows_gemm(2 * fp, W, True), (P * W + active * 2 * fp * W + P * fp) * 2, 4.0 * P * fp * W)
    k.time("experts", "bobarax experts down", mk_rows_gemm(W, fp, False), (P * fp + active * fp * W + P * W) * 2, 2.0 * P * fp * W)

    # recurrence
    def mk_rec(i):
        wide, st, out, norm = _w(T, 2 * K + 2 * V), zeros(seqs + 1, r.heads, _pad16(r.dim), _pad16(r.vdim)), empty(T, V), ones(V)
        powers = ops.decay_powers(r.decay, dev)
        parts = wide.split((K, K, V, V), 1)
        if decode:
            sums = zeros(T, r.heads)
            return lambda: ops.fixed_decay_step(*parts, norm, powers, st, out, sums, segs, pos)
        model = Bobarax.__new__(Bobarax)               # its choice of groups only
        model.dtype, model.scan_heads, model.device = bf, r.heads, dev
        gr = scan_groups(segs.cpu().numpy(), model.scan_group_rows(segs[:, 1].cpu().numpy()))
        cut, gr = len(gr) > seqs, torch.from_numpy(gr).to(dev)
        scratch = torch.empty(len(gr) * K * _pad16(r.vdim), device=dev) if cut else None
        sums = zeros(T, ops.fixed_decay_sums(r.heads, _pad16(r.vdim), bf))
        return lambda: ops.fixed_decay_scan(*parts, norm, powers, st, out, sums, segs, pos, groups=gr, scratch=scratch)
    state = seqs * K * r.vdim * 4
    C = Bobarax.SCAN_CHUNK
    if decode:
        k.time("scan", "bobarax lightning step (gate inside)", mk_rec, 2 * state + T * (2 * K + 3 * V) * 2)
    else:
        k.time("scan", "bobarax lightning recurrence (gate inside)", mk_rec, state + T * (2 * K + 3 * V) * 2, 4.0 * T * K * r.vdim + T * C * (K + V))

    # attention
    nr = T if decode else 0
    for a in attns:
        D, Va, H, G = _pad16(a.dim), _pad16(a.vdim), a.heads, a.kv_heads
        name, seen = "window" if a.window else "chunk", visible_pairs(positions, a.window, a.chunk)
        cols, turns = H * D + G * (D + Va) + (H * Va if a.gated else 0), ops.rotation_turns(a.rot.dims, a.rot.base, dev) if a.rot else None
        cap = a.softcap or 0.0

        def mk_prep(i):
            wide, qa, cache = _w(T, cols), empty(max(nr, 1), H, D + 8), _w(nblocks * G * bs, D + Va + 8)
            qn, kn = ones(H * D), ones(G * D)
            return lambda: ops.paired_attention_prep(wide, qa[:nr], cache, qn, kn, turns, pos, slots, nr, H, G, a.dim, bs, 1e-5)
        k.time("attention", f"bobarax {name} norms + rotation + cache write", mk_prep, T * 2 * (H * D + G * (D + Va)) * 2)
        if decode:
            sms, sp, units = torch.cuda.get_device_properties(0).multi_processor_count, 1, G * ((H // G + 15) // 16)
            while sp < 8 and seqs * units * sp * 2 <= Bobarax.attn_cta_slots(sp * 2, sms) and ctx // (sp * 2) >= 64:
                sp *= 2
            sp, ctx_lens = Bobarax.layer_splits(a, sp), pos + 1

            def mk_rows(i):
                qa, cache, o, wide = _w(T, H, D + 8), _w(nblocks * G * bs, D + Va + 8), empty(T, H, Va), _w(T, H * Va)
                return lambda: ops.paired_attention_rows(qa, cache, tables, seq_of_row, ctx_lens, o, G, bs, cap, a.window, a.chunk, wide if a.gated else None, splits=sp)
            k.time("attention", f"bobarax {name} attention, rows form", mk_rows, seen * G * (D + Va) * 2 + T * H * (D + 2 * Va) * 2, 2.0 * seen * H * (D + Va))
        else:
            tl, _ = dense_context([s * L for s in range(seqs)], [L] * seqs, [0] * seqs, list(range(seqs)), tables.cpu().numpy(), bs)
            tl = torch.from_numpy(tl).to(dev)

            def mk_pre(i):
                wide, cache, o = _w(T, cols), _w(nblocks * G * bs, D + Va + 8), empty(T, H * Va)
                gate = wide[:, cols - H * Va:] if a.gated else None
                return lambda: ops.paired_attention_prefill(wide, cache, tables, seq_of_row, tl, o, H, G, D, bs, cap, a.window, a.chunk, gate)
            k.time("attention", f"bobarax {name} attention, prefill form", mk_pre, T * (H * D + G * (D + Va) + H * Va) * 2, 2.0 * seen * H * (D + Va))
    return k.rows


def run(sizes, kernels=True, models=True, only="", case="") -> dict:
    out = {"bench": "bobarax beside tinapel and llama", "data": "synthetic (random token ids, random weights)", "dtype": "bf16", "sizes": {}}
    for s in sizes:
        r = out["sizes"][s] = {}
        if models:
            r["models"] = [model_numbers(n) for n in TRIPLES[s]]
        if kernels:
            r["kernels"] = {c: sum((m.kernel_numbers(s, *v, only=only) for m in (bench_tinapel, bench_nubosun)), kernel_numbers(s, *v, only=only))
                            for c, v in CASES.items() if case in c}
    return out


if __name__ == "__main__":
    raise SystemExit(bench_nubosun.main(run, __doc__))
