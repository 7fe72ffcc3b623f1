"""Entry points of the mixer operators: residual streams with hyper-connections, one residual stream with parallel branches, short
convolution + selective scan and linear recurrences over carried state, attention over a compressed (latent) paged cache, over
a cache whose rows are keys and values at once and over one with both side by side, and the routing of a mixture of experts.  bf16 or fp32 activations; what enters a softmax, a
norm, a recurrence or the residual sum is fp32 in both.

``segs`` is the device int32 [nseg, 4] list of a ragged batch: (first row, rows, state slot, 0) per sequence, rows of a
sequence consecutive and in position order."""
from __future__ import annotations

import math
from typing import Optional

import torch

from . import _chk, _count, _p, _st, lib


def _is_bf16(t: torch.Tensor) -> int:
    assert t.dtype in (torch.bfloat16, torch.float32), t.dtype
    return 1 if t.dtype is torch.bfloat16 else 0


def hyper_embed(ids, table, scale: float, x, hin, gamma, h, width: int, eps: float) -> None:
    """Every stream of row r := table[ids[r]] * scale (x fp32 [rows, streams, ld]); h := RMSNorm(sum_s hin[s] x_s) * gamma."""
    rows, S, ld = x.shape
    assert x.dtype is torch.float32 and table.dtype is h.dtype and table.shape[1] == ld and ids.dtype is torch.int64
    _chk(lib().tbv_op_hyper_embed(_p(ids), _p(table), table.shape[0], scale, _p(x), _p(hin), _p(gamma), _p(h), rows, S, width, ld, h.stride(0),
                                  eps, _is_bf16(h), _st()), "tbv_op_hyper_embed")
    _count()


def hyper_mix(y, scale, hout, hmix, x, hin, gamma, h, width: int, eps: float, rows: Optional[torch.Tensor] = None, last: bool = False) -> None:
    """End of one sublayer and start of the next: x_t <- sum_s hmix[s, t] x_s + hout[t] * scale * y, then
    h := RMSNorm(sum_t hin[t] x_t) * gamma.  ``last``: only the rows listed in ``rows`` (None = all) give an h, packed, and x is not written."""
    n, S, ld = x.shape
    assert x.dtype is torch.float32 and y.dtype is torch.float32 and y.stride(0) == ld and hmix.shape == (S, S)
    assert rows is None or (last and rows.dtype is torch.int64)
    _chk(lib().tbv_op_hyper_mix(_p(y), _p(scale), _p(hout), _p(hmix), _p(x), _p(hin), _p(gamma), _p(h), _p(rows), int(last), h.shape[0] if last else n,
                                S, width, ld, h.stride(0), eps, _is_bf16(h), _st()), "tbv_op_hyper_mix")
    _count()


def causal_conv_silu(x, out, taps, bias, conv_state, segs, seg_of_row, positions) -> None:
    """out = silu(causal depthwise convolution of the first taps.shape[1] columns of x); taps fp32 [K, C] with the last row
    weighing the current token; inputs before a segment's first row come from conv_state [slots, K - 1, C]."""
    K, C = taps.shape
    assert conv_state.shape[1:] == (K - 1, C) and conv_state.dtype is torch.float32 and x.dtype is out.dtype
    _chk(lib().tbv_op_causal_conv_silu(_p(x), _p(out), _p(taps), _p(bias), _p(conv_state), _p(segs), _p(seg_of_row), _p(positions), x.shape[0],
                                       x.stride(0), out.stride(0), C, K, _is_bf16(x), _st()), "tbv_op_causal_conv_silu")
    _count()


def selective_scan(u, xz, z_off: int, dt, bc, b_off: int, c_off: int, a_log2e, d, ssm, conv_state, out, segs, positions,
                   one_token: bool = False) -> None:
    """Per channel c and state n, dt = softplus of the given values: S <- exp2(dt a_log2e) S + dt u B; y = sum_n S C + d u; out = y * silu(z), z at columns z_off.. of xz.
    a_log2e fp32 [inner, N] (= -exp(A_log) * log2 e); ssm fp32 [slots, inner, N] and conv_state (the convolution's last inputs, from
    the first columns of xz) are replaced.  ``out`` may be ``u``.
    ``one_token``: every segment has one row (a decode step)."""
    inner, N = a_log2e.shape
    assert ssm.shape[1:] == (inner, N) and ssm.dtype is torch.float32 and dt.dtype is torch.float32 and bc.dtype is torch.float32
    assert u.dtype is xz.dtype is out.dtype and segs.dtype is torch.int32
    _chk(lib().tbv_op_selective_scan(_p(u), _p(xz), _p(dt), _p(bc), _p(a_log2e), _p(d), _p(ssm), _p(conv_state), _p(out), _p(segs), _p(positions),
                                     segs.shape[0], inner, N, u.stride(0), xz.stride(0), z_off, dt.stride(0), bc.stride(0), b_off, c_off,
                                     out.stride(0), conv_state.shape[2], conv_state.shape[1] + 1, int(one_token), _is_bf16(u), _st()), "tbv_op_selective_scan")
    _count()


def short_conv(x, out, taps, state, segs, seg_of_row, positions, add: bool = False) -> None:
    """out = silu(conv(x)), or x + conv(x) with ``add`` (x fp32 then): causal depthwise convolution over time of the first taps.shape[1] columns of x; taps fp32
    [K, C] with the last row weighing the current token.  state fp32 [slots, K - 1, C] holds the inputs before a segment's first row and is replaced by its last ones."""
    K, C = taps.shape
    assert state.shape[1:] == (K - 1, C) and state.dtype is taps.dtype is torch.float32 and (x.dtype is out.dtype or (add and x.dtype is torch.float32))
    _chk(lib().tbv_op_short_conv(_p(x), _p(out), _p(taps), _p(state), _p(segs), _p(seg_of_row), _p(positions), x.shape[0], x.stride(0), out.stride(0), C, K, int(add),
                                 _is_bf16(out), _st()), "tbv_op_short_conv")
    _count()


LATENT_ROW_PAD = 8


def latent_row(rank_p: int, rot_p: int) -> int:
    """Values between two rows of the latent cache (and of the folded queries): latent, rotated part, pad (the pitch the rows
    kernel wants in shared memory)."""
    return rank_p + rot_p + LATENT_ROW_PAD


def latent_prep(low, q, qa, cache, gamma, turns, mscale: float, positions, slots, n_rows_form: int, q_off: int, c_off: int, k_off: int, heads: int,
                rank: int, rank_p: int, rot_p: int, eps: float, query_latent=None) -> None:
    """Rotates the query parts of q (columns q_off.., heads x rot_p; interleaved pairs) and writes the cache row: RMSNorm of the latent of low
    (c_off..) and its rotated key part (k_off..).  The first n_rows_form rows' query parts go to qa [rows, heads, row], the
    others stay in place.  Rows of qa and cache: ``latent_row``.  ``turns`` of ``rotation_turns``; cos and sin are multiplied by mscale.  ``query_latent`` =
    (column, size, weight fp32): that part of low is RMS-normed in place.  low or q may be None (then its part is left out)."""
    act = low if low is not None else q
    assert act.dtype is cache.dtype and cache.shape[1] == latent_row(rank_p, rot_p) and positions.dtype is torch.int32 and turns.dtype is torch.float32
    assert (q is None or (qa.dtype is q.dtype and q.stride(1) == 1)) and (low is None or (slots.dtype is torch.int64 and gamma.dtype is torch.float32))
    col, size, weight = query_latent if query_latent is not None else (0, 0, None)
    _chk(lib().tbv_op_latent_prep(_p(low), _p(q), _p(qa), _p(cache), _p(gamma), _p(weight), _p(turns), _p(positions), _p(slots), act.shape[0], n_rows_form,
                                  low.stride(0) if low is not None else 0, q.stride(0) if q is not None else 0, q_off, c_off, k_off, col, size, heads, rank, rank_p,
                                  rot_p, turns.shape[0], eps, mscale, _is_bf16(act), _st()), "tbv_op_latent_prep")
    _count()


def latent_attention_rows(qa, cache, tables, seq_of_row, ctx_lens, sink, out, rank: int, scale: float, block_size: int, splits: int = 1, window: int = 0) -> None:
    """qa [rows, heads, row] against the cache rows (keys over all columns of ``latent_row`` but the pad, values = the first out.shape[2] columns); softmax with
    exp(sink) in the denominator (sink fp32 [heads] or None); a row sees the last ``window`` keys (0: all)."""
    rows, H, row = qa.shape
    Rp, Dk = out.shape[2], row - LATENT_ROW_PAD
    assert qa.is_contiguous() and out.is_contiguous() and cache.shape[1] == row and qa.dtype is cache.dtype is out.dtype
    assert tables.dtype is torch.int32 and ctx_lens.dtype is torch.int32
    _chk(lib().tbv_op_latent_attn_rows(_p(qa), _p(cache), _p(tables), _p(seq_of_row), _p(ctx_lens), _p(sink), _p(out), rows, H, rank, Rp, Dk - Rp,
                                       block_size, tables.shape[1], splits, scale, window, _is_bf16(qa), _st()), "tbv_op_latent_attn_rows")
    _count()


def latent_gather(cache, slots, c, kr) -> None:
    """Cache rows ``slots`` (int64) -> dense latents c [n, Rp] and rotated key parts kr [n, rotp] (bf16)."""
    assert cache.dtype is torch.bfloat16 and slots.dtype is torch.int64 and c.is_contiguous() and kr.is_contiguous()
    _chk(lib().tbv_op_latent_gather(_p(cache), _p(slots), _p(c), _p(kr), slots.shape[0], c.shape[1], kr.shape[1], _st()), "tbv_op_latent_gather")
    _count()


def latent_prefill_fits(dim_p: int, rot_p: int, v_p: int) -> bool:
    return bool(lib().tbv_op_latent_prefill_fits(dim_p, rot_p, v_p))


def latent_attention_prefill(qkv, q_rot_off: int, kv, kr, tiles, sink, out, heads: int, dim_p: int, v_p: int, scale: float, window: int = 0) -> None:
    """Many query rows against expanded keys / values: kv [ctx rows, heads * dim_p | heads * v_p], rotated key parts kr [ctx rows, rot_p];
    tiles int32 [n, 4] = (first query row, rows <= 64, ctx row of the sequence's first token, keys the first row sees).  With a ``window`` rows before the first
    visible key's tile of 64 positions are not read (and need not be there: that ctx row may lie before the first one)."""
    assert qkv.dtype is kv.dtype is kr.dtype is out.dtype is torch.bfloat16 and tiles.dtype is torch.int32
    _chk(lib().tbv_op_latent_prefill(_p(qkv), _p(kv), _p(kr), _p(tiles), _p(sink), _p(out), tiles.shape[0], heads, qkv.stride(0), q_rot_off,
                                     kv.stride(0), heads * dim_p, out.stride(0), dim_p, kr.shape[1], v_p, scale, window, _st()), "tbv_op_latent_prefill")
    _count()


# ---- one residual stream with parallel branches -----------------------------------------------------------------------------
def position_turns(width: int, device, base: float = 10000.0) -> torch.Tensor:
    """fp32 [ceil(width / 2), 2]: turns per position of every sine / cosine pair of the position vector, as high and low part."""
    return frequency_turns(base ** (-2.0 * torch.arange((width + 1) // 2, dtype=torch.float64) / width), device)


def rotation_turns(dims: int, base: float, device) -> torch.Tensor:
    """fp32 [dims / 2, 2]: the same for the pairs of a rotation over ``dims`` dimensions."""
    return frequency_turns(float(base) ** (-2.0 * torch.arange(dims // 2, dtype=torch.float64) / max(dims, 1)), device)


def frequency_turns(freq: torch.Tensor, device) -> torch.Tensor:
    """fp32 [n, 2]: turns per position of the angular frequencies ``freq`` (float64), as high and low part."""
    f = freq / (2.0 * math.pi)
    hi = f.to(torch.float32)
    return torch.stack((hi, (f - hi.double()).to(torch.float32)), 1).contiguous().to(device)


def residual(x, g1, h1, width: int, eps: float, g2=None, h2=None, embed=None, positions=None, y1=None, y2=None, routed=None, x0=None, step=None,
             rows: Optional[torch.Tensor] = None, last: bool = False, mix=None, post=None, sums=None, place=None, conv=None) -> None:
    """x <- x + y1 + y2 + sum_j weight_j * routed_j (+ x0 + step);  h1 := RMSNorm(x) * g1,  h2 := RMSNorm(x) * g2.

    x, y1, y2, x0 fp32 [rows, ld].  ``routed`` = (rows of the experts' results, place int32 [rows, top], weight fp32 [rows, top]).
    ``embed`` = (ids, table, scale, turns): x := table[ids] * scale + position vector instead, kept in ``x0`` as well if that is given.
    h1 may be fp32 beside bf16 activations.  ``last``: only the rows listed in ``rows`` (None = all) give an h1, packed, and x is not written.
    ``mix`` = (mu fp32 [n, ld], mixes [rows, n * ld], shift fp32 [slots, ld], segs): one row per segment; instead of h1 its mixes
    h1 + (previous h1 - h1) * mu_s are written, and shift is replaced.
    ``post`` (fp32 [ld]): x <- x + RMSNorm(branches) * post instead, the branches being y1 and ``routed``, whose weight may be one number.  ``sums`` = (square sums
    fp32 [rows, n], width): y1 is divided by sqrt(sum / width + eps) first.  ``place`` int32 [rows, top]: h1 goes to these rows of ``h1``.
    ``turns`` None: no position vector.
    g1 None: h1 := x.  h1 None: only x is written.  ``conv`` = (taps fp32 [k, ld], past fp32 [slots, k - 1, ld], segs): one row per segment; the causal
    convolution of h1 over time is added to it, past is replaced (``short_conv`` for many rows)."""
    ld = x.shape[1]
    n = h1.shape[0] if last else x.shape[0]
    taps, past, conv_segs = conv if conv is not None else (None, None, None)
    assert taps is None or (taps.shape[1] == ld and taps.dtype is past.dtype is torch.float32 and past.shape[1:] == (taps.shape[0] - 1, ld) and mix is None)
    assert x.dtype is torch.float32 and x.is_contiguous() and (h2 is None or h2.stride(0) == h1.stride(0)) and (rows is None or (last and rows.dtype is torch.int64))
    for t in (y1, y2, x0):
        assert t is None or (t.dtype is torch.float32 and t.stride(0) == ld)
    ids, table, scale, turns = embed if embed is not None else (None, None, 0.0, None)
    ro, source, weight = routed if routed is not None else (None, None, None)
    const = weight if isinstance(weight, float) else 0.0
    weight = None if isinstance(weight, float) else weight
    sq, sum_width = sums if sums is not None else (None, 0)
    mu, mixes, shift, segs = mix if mix is not None else (None, None, None, None)
    act = [t.dtype for t in (table, ro, h2, mixes, h1) if t is not None] or [torch.float32]
    h1_f32 = h1 is not None and h1.dtype is torch.float32
    assert all(d is act[0] for d in act[:-1]) and (h1 is None or h1.dtype is act[0] or h1_f32)
    segs = conv_segs if segs is None else segs
    assert ro is None or (ro.stride(0) == ld and source.dtype is torch.int32 and source.is_contiguous() and (weight is None or weight.dtype is torch.float32))
    assert place is None or (place.dtype is torch.int32 and place.is_contiguous() and place.shape[0] == x.shape[0] and h1.shape[0] >= place.numel())
    assert sq is None or (sq.dtype is torch.float32 and sq.is_contiguous() and post is not None)
    assert post is None or (post.dtype is torch.float32 and y2 is None and x0 is None and step is None)
    assert mu is None or (mixes.shape[1] == mu.shape[0] * ld and shift.shape[1] == ld and shift.dtype is torch.float32)
    _chk(lib().tbv_op_residual(_p(ids), _p(table), _p(turns), _p(positions), scale, table.shape[0] if table is not None else 0, _p(x), _p(x0), _p(y1), _p(y2),
                               _p(step), _p(ro), _p(source), _p(weight), source.shape[1] if source is not None else 0, _p(g1), _p(g2), _p(h1), _p(h2),
                               int(h1_f32), _p(rows), int(last), _p(mu), _p(mixes), _p(shift), _p(segs),
                               mu.shape[0] if mu is not None else 0, _p(post), _p(sq), sq.shape[1] if sq is not None else 0, sum_width, const, _p(place),
                               place.shape[1] if place is not None else 0, _p(taps), _p(past), taps.shape[0] if taps is not None else 0, n, width, ld,
                               h1.stride(0) if h1 is not None else ld, eps, int(act[0] is torch.bfloat16), _st()), "tbv_op_residual")
    _count()


def token_shift(h, mu, shift, mixes, segs, seg_of_row, positions) -> None:
    """mixes[t] = n mixes of h_t (fp32 [rows, ld]) with h_{t-1}: h_t + (h_{t-1} - h_t) * mu_s; the row before a segment's first is shift[slot] (zeros at a
    sequence's start).  shift is left as it is (``decay_scan`` replaces it)."""
    n, ld = mu.shape
    assert h.dtype is mu.dtype is shift.dtype is torch.float32 and h.is_contiguous() and mixes.is_contiguous() and mixes.shape[1] == n * ld
    _chk(lib().tbv_op_token_shift(_p(h), _p(mu), _p(shift), _p(mixes), _p(segs), _p(seg_of_row), _p(positions), h.shape[0], ld, n, _is_bf16(mixes), _st()),
         "tbv_op_token_shift")
    _count()


# ---- linear recurrences with a matrix state -----------------------------------------------------------------------------------
DECAY_RANK_MAX = 128                  # of the decay product inside decay_scan


def decay_scan(q, k, v, g, z, norm, state, o, out, segs, positions, vdim: int, eps: float, qscale: float = 1.0, tau: float = 1.0, u=None,
               shift=None, groups=None, scratch=None, low=None) -> None:
    """Per head S_t = diag(a_t) S_{t-1} + k_t v_t^T over the rows of every segment, then out = RMSNorm(o) * norm * silu(g).
    u None (gated linear attention): a = sigmoid(z)^(1 / tau), o_t = S_t^T (qscale q_t).  u fp32 [heads * Dp] (WKV): a = exp(-exp(z)),
    o_t = (S_{t-1} + diag(u) k_t v_t^T)^T q_t.

    q, k, v, g: column views [rows, heads * size] of one buffer; z fp32 [rows, heads * Dp]; state fp32 [slots, heads, Dp, Vp] is replaced;
    ``groups`` (bf16; None: the sequential kernel): the segments cut into groups of rows, int32 [n, 4] (engine.batch.scan_groups), for the chunked
    tensor-core kernels; ``scratch`` = fp32 (states of n * heads * Dp * Vp, totals of n * heads * Dp) if a segment has several groups, else None.
    ``low`` (with groups) = (low [rows, rank], w2 [heads * Dp, rank], b2 [heads * Dp]) instead of z: z = low @ w2^T + b2 computed inside,
    rank at most ``DECAY_RANK_MAX``.
    o: fp32 scratch [rows, heads * Vp]; ``shift`` = (h fp32 [rows, ld], shift fp32 [slots, ld]): every segment's last row of h is kept."""
    _, H, Dp, Vp = state.shape
    rows = q.shape[0]
    assert state.dtype is torch.float32 and o.dtype is torch.float32 and o.numel() >= rows * H * Vp and q.dtype is out.dtype
    assert (z is None) == (low is not None) and (z is None or z.dtype is torch.float32)
    lo, w2, b2 = low if low is not None else (None, None, None)
    assert lo is None or (lo.dtype is w2.dtype is b2.dtype is torch.bfloat16 and w2.is_contiguous() and lo.shape[1] == w2.shape[1])
    assert q.stride(0) == k.stride(0) == v.stride(0) == g.stride(0) and q.shape[1] == k.shape[1] == H * Dp and v.shape[1] == g.shape[1] == H * Vp
    h1, sh = shift if shift is not None else (None, None)
    n = 0 if groups is None else groups.shape[0]
    starts, totals = scratch if scratch is not None else (None, None)
    assert groups is None or (q.dtype is torch.bfloat16 and groups.dtype is torch.int32)
    assert scratch is None or (starts.numel() >= n * H * Dp * Vp and totals.numel() >= n * H * Dp and starts.dtype is totals.dtype is torch.float32)
    _chk(lib().tbv_op_decay_scan(_p(q), _p(k), _p(v), _p(g), _p(z), _p(u), _p(norm), _p(state), _p(o), _p(out), _p(h1), _p(sh), _p(segs), _p(positions),
                                 _p(groups), n, int(scratch is not None), _p(starts), _p(totals), _p(lo), _p(w2), _p(b2), lo.stride(0) if lo is not None else 0,
                                 w2.shape[1] if w2 is not None else 0, rows, segs.shape[0], H, Dp, Vp, vdim, q.stride(0), z.stride(0) if z is not None else 0, out.stride(0), h1.shape[1] if h1 is not None else 0,
                                 qscale, tau, eps, _is_bf16(q), _st()), "tbv_op_decay_scan")
    _count(4 if scratch is not None else 2)


def decay_step(q, k, v, g, low, w2, b2, norm, state, out, segs, positions, vdim: int, eps: float, qscale: float = 1.0, tau: float = 1.0, u=None) -> None:
    """``decay_scan`` for one row per segment, with z = act(low) @ w2^T + b2 computed inside (act = tanh for WKV)."""
    _, H, Dp, Vp = state.shape
    rank = w2.shape[1]
    assert state.dtype is torch.float32 and q.dtype is low.dtype is w2.dtype is b2.dtype is out.dtype and w2.shape[0] == H * Dp and low.shape[1] == rank
    assert q.stride(0) == k.stride(0) == v.stride(0) == g.stride(0) and q.shape[1] == k.shape[1] == H * Dp and v.shape[1] == g.shape[1] == H * Vp
    _chk(lib().tbv_op_decay_step(_p(q), _p(k), _p(v), _p(g), _p(low), _p(w2), _p(b2), _p(u), _p(norm), _p(state), _p(out), _p(segs), _p(positions),
                                 segs.shape[0], H, Dp, Vp, vdim, q.stride(0), low.stride(0), rank, out.stride(0), qscale, tau, eps, _is_bf16(q), _st()),
         "tbv_op_decay_step")
    _count()


# ---- linear recurrences with one constant decay per head ------------------------------------------------------------------------
def decay_powers(decay, device) -> torch.Tensor:
    """fp32 [heads, chunk + 1]: powers of every head's decay (rounded to fp32 once), as the recurrences take them."""
    a = torch.tensor(list(decay), dtype=torch.float32).double()
    return (a[:, None] ** torch.arange(lib().tbv_op_fixed_decay_chunk() + 1, dtype=torch.float64)[None]).to(torch.float32).contiguous().to(device)


def fixed_decay_sums(heads: int, Vp: int, dtype) -> int:
    """Square sums per row that ``fixed_decay_scan`` writes."""
    return lib().tbv_op_fixed_decay_sums(heads, Vp, int(dtype is torch.bfloat16))


def fixed_decay_scan(q, k, v, g, norm, powers, state, out, sums, segs, positions, groups=None, scratch=None, o=None) -> None:
    """Per head S_t = a S_{t-1} + k_t v_t^T, o_t = S_t^T q_t over the rows of every segment; out = o * norm * sigmoid(g), sums fp32 [rows, fixed_decay_sums] =
    square sums of o (what is left of a joint norm of the heads is one factor per row: ``residual`` takes it).

    q, k, v, g: column views of one buffer, q, k and v with their activations; state fp32 [slots, heads, Dp, Vp] is replaced.  bf16: ``groups`` = the segments
    cut into groups of rows (engine.batch.scan_groups), ``scratch`` = fp32 states of n * heads * Dp * Vp if a segment has several groups, else None.
    fp32: ``o`` = fp32 scratch [rows, heads * Vp]."""
    _, H, Dp, Vp = state.shape
    rows, bf16 = q.shape[0], _is_bf16(q)
    assert q.stride(0) == k.stride(0) == v.stride(0) == g.stride(0) and q.shape[1] == k.shape[1] == H * Dp and v.shape[1] == g.shape[1] == H * Vp
    assert state.dtype is torch.float32 and q.dtype is out.dtype and sums.dtype is torch.float32 and sums.is_contiguous()
    assert sums.shape == (rows, fixed_decay_sums(H, Vp, q.dtype)) and powers.shape[0] == H and norm.dtype is torch.float32
    n = 0 if groups is None else groups.shape[0]
    assert (groups is not None and groups.dtype is torch.int32) if bf16 else (o is not None and o.dtype is torch.float32 and o.numel() >= rows * H * Vp)
    assert scratch is None or (scratch.dtype is torch.float32 and scratch.numel() >= n * H * Dp * Vp)
    _chk(lib().tbv_op_fixed_decay_scan(_p(q), _p(k), _p(v), _p(g), _p(norm), _p(powers), _p(state), _p(o), _p(out), _p(sums), _p(segs), _p(positions), _p(groups), n,
                                       int(scratch is not None), _p(scratch), rows, segs.shape[0], H, Dp, Vp, q.stride(0), out.stride(0), bf16, _st()),
         "tbv_op_fixed_decay_scan")
    _count(2 if not bf16 else (3 if scratch is not None else 1))


def fixed_decay_step(q, k, v, g, norm, powers, state, out, sums, segs, positions) -> None:
    """``fixed_decay_scan`` for one row per segment; sums [rows, heads]."""
    _, H, Dp, Vp = state.shape
    assert q.stride(0) == k.stride(0) == v.stride(0) == g.stride(0) and q.shape[1] == k.shape[1] == H * Dp and v.shape[1] == g.shape[1] == H * Vp
    assert state.dtype is torch.float32 and q.dtype is out.dtype and sums.shape == (q.shape[0], H) and sums.is_contiguous() and powers.shape[0] == H
    _chk(lib().tbv_op_fixed_decay_step(_p(q), _p(k), _p(v), _p(g), _p(norm), _p(powers), _p(state), _p(out), _p(sums), _p(segs), _p(positions), segs.shape[0], H, Dp, Vp,
                                       q.stride(0), out.stride(0), _is_bf16(q), _st()), "tbv_op_fixed_decay_step")
    _count()


# ---- gated delta rule with a decay per key channel -----------------------------------------------------------------------------------
def delta_sets(rows: int, groups: int, state: torch.Tensor) -> int:
    """Bytes of scratch with which ``delta_scan`` makes the operands of all chunks in parallel; 0 where the sizes do not allow it or enough sequences and heads
    keep the GPU busy."""
    _, H, Dp, Vp = state.shape
    return lib().tbv_op_delta_sets(rows, groups, H, Dp, Vp)


def delta_scan(q, k, v, beta, z, gate, rate, norm, state, o, out, segs, positions, kv_heads: int, dim: int, vdim: int, eps: float, groups=None, sets=None) -> None:
    """Per head, q and k of its key head made unit vectors (q times dim^-0.5), S' = diag(exp(-rate z_t)) S_{t-1}, u = sigmoid(beta_t) (v_t - S'^T k_t),
    S_t = S' + k_t u^T over the rows of every segment; out = RMSNorm(S_t^T q_t) * norm * sigmoid(gate).

    q, k [rows, kv_heads * Dp] and v [rows, heads * Vp]: column views of one buffer, behind convolution and SiLU; beta [rows, >= heads], gate [rows, heads * Vp] in the
    activation type; z fp32 [rows, heads * Dp] (softplus of the decay inputs), rate fp32 [heads], norm fp32 [Vp]; state fp32 [slots, heads, Dp, Vp] is replaced; o fp32 scratch [rows, heads * Vp].
    ``groups`` (bf16): the segments, int32 [n, 4] (engine.batch.scan_groups), for the chunked tensor-core kernels where the sizes allow; ``sets``: uint8 scratch of
    ``delta_sets`` bytes (16-byte aligned) for their form with few sequences and heads."""
    _, H, Dp, Vp = state.shape
    rows = q.shape[0]
    assert q.stride(0) == k.stride(0) == v.stride(0) and q.shape[1] == k.shape[1] == kv_heads * Dp and v.shape[1] == gate.shape[1] == H * Vp and z.shape[1] == H * Dp
    assert state.dtype is z.dtype is rate.dtype is norm.dtype is o.dtype is torch.float32 and o.numel() >= rows * H * Vp and norm.shape[0] == Vp and rate.shape[0] == H
    assert sets is None or (groups is not None and sets.dtype is torch.uint8)
    assert q.dtype is beta.dtype is gate.dtype is out.dtype and beta.shape[1] >= H and (groups is None or (q.dtype is torch.bfloat16 and groups.dtype is torch.int32))
    _chk(lib().tbv_op_delta_scan(_p(q), _p(k), _p(v), _p(beta), _p(z), _p(gate), _p(rate), _p(norm), _p(state), _p(o), _p(out), _p(segs), _p(positions), _p(groups),
                                 0 if groups is None else groups.shape[0], _p(sets), rows, segs.shape[0], H, kv_heads, Dp, Vp, dim, vdim, q.stride(0), beta.stride(0), z.stride(0),
                                 gate.stride(0), out.stride(0), eps, _is_bf16(q), _st()), "tbv_op_delta_scan")
    _count(1 if sets is None and Vp <= 128 and Dp <= 128 and groups is not None else (3 if sets is not None else 2))


def delta_step(q, k, v, beta, low_a, low_g, w_a, b_a, w_g, rate, norm, state, out, segs, positions, kv_heads: int, dim: int, vdim: int, eps: float, conv=None) -> None:
    """``delta_scan`` for one row per segment, with z = softplus(low_a @ w_a^T + b_a) and gate = low_g @ w_g^T computed inside.  ``conv`` = (taps fp32 [K, C], state fp32
    [slots, K - 1, C]), for kv_heads = heads: q, k and v are taken before convolution and SiLU, and that state is replaced."""
    _, H, Dp, Vp = state.shape
    taps, past = conv if conv is not None else (None, None)
    rank = w_a.shape[1]
    assert q.stride(0) == k.stride(0) == v.stride(0) and q.shape[1] == k.shape[1] == kv_heads * Dp and v.shape[1] == H * Vp
    assert beta.stride(0) == low_a.stride(0) == low_g.stride(0) and beta.shape[1] >= H and low_a.shape[1] == low_g.shape[1] == w_g.shape[1] == rank
    assert w_a.shape[0] == b_a.shape[0] == H * Dp and w_g.shape[0] == H * Vp and w_a.is_contiguous() and w_g.is_contiguous()
    assert state.dtype is rate.dtype is norm.dtype is torch.float32 and q.dtype is beta.dtype is low_a.dtype is w_a.dtype is b_a.dtype is w_g.dtype is out.dtype
    assert taps is None or (taps.dtype is past.dtype is torch.float32 and kv_heads == H and taps.shape[1] == H * (2 * Dp + Vp) and past.shape[1:] == (taps.shape[0] - 1, taps.shape[1]))
    _chk(lib().tbv_op_delta_step(_p(q), _p(k), _p(v), _p(beta), _p(low_a), _p(low_g), _p(w_a), _p(b_a), _p(w_g), _p(rate), _p(norm), _p(state), _p(out), _p(taps), _p(past),
                                 _p(segs), _p(positions), segs.shape[0], H, kv_heads, Dp, Vp, dim, vdim, q.stride(0), beta.stride(0), rank,
                                 taps.shape[0] if taps is not None else 0, out.stride(0), eps, _is_bf16(q), _st()), "tbv_op_delta_step")
    _count()


# ---- attention whose cached rows are keys and values at once --------------------------------------------------------------------
SHARED_PREFILL_MAX_DIM = 256          # padded head size that the prefill form takes


def shared_attention_prep(qk, qa, cache, fold, positions, slots, n_rows_form: int, heads: int, kv_heads: int, dim: int, block_size: int, eps: float,
                          temp_coef: float = 0.0, temp_every: float = 1.0) -> None:
    """qk [rows, (heads + kv_heads) * Dp]: queries := RMSNorm(q) * (1 + coef * ln(floor((p + 1) / every) + 1)) * fold, to qa [n, heads, Dp + 8] for the first
    n_rows_form rows and in place for the others; cache [blocks * kv_heads * block_size, Dp + 8] takes the key rows and their fp32 factor."""
    Dp = fold.shape[0]
    assert qk.dtype is qa.dtype is cache.dtype and cache.shape[1] == Dp + LATENT_ROW_PAD and slots.dtype is torch.int64 and positions.dtype is torch.int32
    _chk(lib().tbv_op_shared_attn_prep(_p(qk), _p(qa), _p(cache), _p(fold), _p(positions), _p(slots), qk.shape[0], n_rows_form, qk.stride(0), heads, kv_heads,
                                       dim, Dp, block_size, eps, temp_coef, temp_every, _is_bf16(qk), _st()), "tbv_op_shared_attn_prep")
    _count()


def shared_attention_rows(qa, cache, tables, seq_of_row, ctx_lens, out, kv_heads: int, block_size: int, softcap: float = 0.0, splits: int = 1) -> None:
    """qa [rows, heads, Dp + 8] against the cached rows of each row's sequence; out [rows, heads, Dp]."""
    rows, H, row = qa.shape
    Dp = row - LATENT_ROW_PAD
    assert qa.is_contiguous() and out.is_contiguous() and cache.shape[1] == row and qa.dtype is cache.dtype is out.dtype and out.shape[-1] * out.shape[-2] == H * Dp
    assert tables.dtype is torch.int32 and ctx_lens.dtype is torch.int32
    _chk(lib().tbv_op_shared_attn_rows(_p(qa), _p(cache), _p(tables), _p(seq_of_row), _p(ctx_lens), _p(out), rows, H, kv_heads, Dp, block_size,
                                       tables.shape[1], splits, softcap, _is_bf16(qa), _st()), "tbv_op_shared_attn_rows")
    _count()


def shared_attention_prefill(q, cache, tables, seq_of_row, tiles, out, heads: int, kv_heads: int, block_size: int, softcap: float = 0.0) -> None:
    """Many query rows q [rows, heads * Dp ..] in tiles int32 [n, 4] = (first row, rows <= 64, -, keys the first row sees); bf16."""
    Dp = cache.shape[1] - LATENT_ROW_PAD
    assert q.dtype is cache.dtype is out.dtype is torch.bfloat16 and tiles.dtype is torch.int32 and seq_of_row.dtype is torch.int32
    _chk(lib().tbv_op_shared_attn_prefill(_p(q), _p(cache), _p(tables), _p(seq_of_row), _p(tiles), _p(out), tiles.shape[0], q.stride(0), out.stride(0), heads,
                                          kv_heads, Dp, block_size, tables.shape[1], softcap, _st()), "tbv_op_shared_attn_prefill")
    _count()


# ---- attention whose cached rows hold a key and a value side by side --------------------------------------------------------------
def paired_prefill_fits(dim_p: int, v_p: int) -> bool:
    return bool(lib().tbv_op_paired_prefill_fits(dim_p, v_p))


def paired_attention_prep(wide, qa, cache, q_norm, k_norm, turns, positions, slots, n_rows_form: int, heads: int, kv_heads: int, dim: int, block_size: int,
                          eps: float) -> None:
    """wide [rows, >= heads * Dp + kv_heads * (Dp + Vp)] = queries, keys, values: queries and keys are normed over all their heads at once (weights fp32
    [heads * Dp], [kv_heads * Dp]), turned (``turns`` of ``rotation_turns`` or None; interleaved pairs of the first dimensions), queries go to qa [n, heads,
    Dp + 8] for the first n_rows_form rows and stay in place for the others, cache [blocks * kv_heads * block_size, Dp + Vp + 8] takes key and value.
    ``kv_heads`` 0: queries only (cache, k_norm: None)."""
    Dp = q_norm.shape[0] // heads
    Vp = 0 if cache is None else cache.shape[1] - LATENT_ROW_PAD - Dp
    assert wide.dtype is qa.dtype and (cache is None) == (kv_heads == 0) and (cache is None or cache.dtype is wide.dtype) and wide.stride(1) == 1
    assert wide.shape[1] >= heads * Dp + kv_heads * (Dp + Vp) and (cache is None or k_norm.shape[0] == kv_heads * Dp)
    assert slots.dtype is torch.int64 and positions.dtype is torch.int32 and q_norm.dtype is torch.float32
    pairs = 0 if turns is None else turns.shape[0]
    _chk(lib().tbv_op_paired_attn_prep(_p(wide), _p(qa), _p(cache), _p(q_norm), _p(k_norm), _p(turns), _p(positions), _p(slots), wide.shape[0], n_rows_form,
                                       wide.stride(0), heads, kv_heads, dim, Dp, Vp, pairs, block_size, eps, _is_bf16(wide), _st()), "tbv_op_paired_attn_prep")
    _count()


def head_attention_prep(wide, qa, cache, qscale, turns, positions, slots, n_rows_form: int, heads: int, kv_heads: int, dim: int, dim_p: int, block_size: int, eps: float,
                        v_first=None, mix=None) -> None:
    """As ``paired_attention_prep``, with norms per head and without weights, and a factor per query head (qscale fp32 [heads]).  ``v_first`` [rows, kv_heads * Vp]:
    takes this layer's values, or with ``mix`` (fp32, one number) is mixed into them: (1 - mix) v + mix v_first."""
    Vp = cache.shape[1] - LATENT_ROW_PAD - dim_p
    assert wide.dtype is qa.dtype is cache.dtype and wide.stride(1) == 1 and wide.shape[1] >= (heads + kv_heads) * dim_p + kv_heads * Vp and qscale.shape[0] == heads
    assert slots.dtype is torch.int64 and positions.dtype is torch.int32 and qscale.dtype is torch.float32 and (mix is None or (mix.dtype is torch.float32 and v_first is not None))
    assert v_first is None or (v_first.dtype is wide.dtype and v_first.is_contiguous() and v_first.shape == (wide.shape[0], kv_heads * Vp))
    _chk(lib().tbv_op_head_attn_prep(_p(wide), _p(qa), _p(cache), _p(qscale), _p(turns), _p(positions), _p(slots), _p(v_first), _p(mix), wide.shape[0], n_rows_form,
                                     wide.stride(0), heads, kv_heads, dim, dim_p, Vp, 0 if turns is None else turns.shape[0], block_size, eps, _is_bf16(wide), _st()),
         "tbv_op_head_attn_prep")
    _count()


def paired_attention_rows(qa, cache, tables, seq_of_row, ctx_lens, out, kv_heads: int, block_size: int, softcap: float = 0.0, window: int = 0, chunk: int = 0,
                          gate=None, splits: int = 1) -> None:
    """qa [rows, heads, Dp + 8] against the cached rows of each row's sequence; out [rows, heads, Vp].  A row that causally sees c keys sees the last ``window``
    of them, or those of its own ``chunk`` of positions (0: all); ``gate`` (column view [rows, heads * Vp] or None): the result is multiplied by its sigmoid."""
    rows, H, row = qa.shape
    Dp, Vp = row - LATENT_ROW_PAD, out.shape[2]
    assert qa.is_contiguous() and out.is_contiguous() and cache.shape[1] == row + Vp and qa.dtype is cache.dtype is out.dtype and out.shape == (rows, H, Vp)
    assert tables.dtype is torch.int32 and ctx_lens.dtype is torch.int32 and (gate is None or (gate.dtype is qa.dtype and gate.shape == (rows, H * Vp) and gate.stride(1) == 1))
    _chk(lib().tbv_op_paired_attn_rows(_p(qa), _p(cache), _p(tables), _p(seq_of_row), _p(ctx_lens), _p(gate), _p(out), rows, H, kv_heads, Dp, Vp,
                                       0 if gate is None else gate.stride(0), block_size, tables.shape[1], splits, softcap, window, chunk, _is_bf16(qa), _st()),
         "tbv_op_paired_attn_rows")
    _count()


def paired_attention_prefill(q, cache, tables, seq_of_row, tiles, out, heads: int, kv_heads: int, dim_p: int, block_size: int, softcap: float = 0.0,
                             window: int = 0, chunk: int = 0, gate=None) -> None:
    """Many query rows q [rows, heads * Dp ..] in tiles int32 [n, 4] = (first row, rows <= 64, -, keys the first row sees); out [rows, heads * Vp]; bf16."""
    Vp = cache.shape[1] - LATENT_ROW_PAD - dim_p
    assert q.dtype is cache.dtype is out.dtype is torch.bfloat16 and tiles.dtype is torch.int32 and seq_of_row.dtype is torch.int32 and out.shape[1] >= heads * Vp
    assert gate is None or (gate.dtype is q.dtype and gate.shape == (q.shape[0], heads * Vp) and gate.stride(1) == 1)
    _chk(lib().tbv_op_paired_attn_prefill(_p(q), _p(cache), _p(tables), _p(seq_of_row), _p(tiles), _p(gate), _p(out), tiles.shape[0], q.stride(0), out.stride(0), heads,
                                          kv_heads, dim_p, Vp, 0 if gate is None else gate.stride(0), block_size, tables.shape[1], softcap, window, chunk, _st()),
         "tbv_op_paired_attn_prefill")
    _count()


# ---- mixture of experts -----------------------------------------------------------------------------------------------------------
def moe_route(logits, h, xp, place, weight, offsets, counts, choice, experts: int, scale: float) -> None:
    """Softmax over the first ``experts`` columns of logits (fp32 [T, ..]), the place.shape[1] largest chosen, their scores / (sum + 1e-20) * scale
    to weight; h's rows copied to xp [T * top, ld], expert after expert: place int32 [T, top], offsets int32 [experts + 1].
    counts [experts] and choice [T * top * 2] are int32 scratch."""
    T, top = place.shape
    assert logits.dtype is torch.float32 and h.is_contiguous() and xp.is_contiguous() and h.dtype is xp.dtype and h.shape[1] == xp.shape[1] and xp.shape[0] >= T * top
    _chk(lib().tbv_op_moe_route(_p(logits), _p(h), _p(xp), _p(place), _p(weight), _p(offsets), _p(counts), _p(choice), T, experts, logits.stride(0), top, scale,
                                h.shape[1] * h.element_size(), _st()), "tbv_op_moe_route")
    _count(1 if T <= lib().tbv_op_moe_small() else 2)


def moe_table_layers(layers, device) -> torch.Tensor:
    """Device records of ``moe_place_table``: ``layers`` = (table int32 [vocab, top], place int32 storage, offsets int32 [experts + 1], experts) per layer.
    They hold addresses: the tensors must outlive them."""
    rec = torch.zeros(len(layers), 4, dtype=torch.int64)
    for i, (table, place, offsets, experts) in enumerate(layers):
        assert table.dtype is place.dtype is offsets.dtype is torch.int32 and table.is_contiguous() and offsets.shape[0] > experts
        rec[i] = torch.tensor([table.data_ptr(), place.data_ptr(), offsets.data_ptr(), experts | table.shape[1] << 32])
    return rec.to(device)


def moe_place_table(ids, records, max_experts: int, vocab: int) -> None:
    """For every layer of ``records``: the (token, choice) pairs laid out expert after expert, the experts of a token being its table row: place [T, top] and
    offsets [experts + 1].  One launch."""
    assert ids.dtype is torch.int64
    _chk(lib().tbv_op_moe_place_table(_p(ids), _p(records), records.shape[0], max_experts, ids.shape[0], vocab, _st()), "tbv_op_moe_place_table")
    _count()
