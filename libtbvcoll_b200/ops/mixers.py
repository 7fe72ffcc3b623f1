"""Entry points of the mixer operators: residual streams with hyper-connections, short convolution + selective scan over
carried state, and attention over a compressed (latent) paged cache.  bf16 or fp32 activations; what enters a softmax, a
norm, a recurrence or the residual sum is fp32 in both.

``segs`` is the device int32 [nseg, 4] list of a ragged batch: (first row, rows, state slot, 0) per sequence, rows of a
sequence consecutive and in position order."""
from __future__ import annotations

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


LATENT_ROW_PAD = 8


def latent_row(rank_p: int, rot_p: int) -> int:
    """Values between two rows of the latent cache (and of the folded queries): latent, rotated part, pad (the pitch the rows
    kernel wants in shared memory)."""
    return rank_p + rot_p + LATENT_ROW_PAD


def latent_prep(qkv, qa, cache, gamma, inv_freq, mscale: float, positions, slots, n_rows_form: int, q_off: int, c_off: int, k_off: int, heads: int,
                rank: int, rank_p: int, rot_p: int, eps: float) -> None:
    """Rotates the query parts (columns q_off.., heads x rot_p; interleaved pairs) and writes the cache row: RMSNorm of the latent
    (c_off..) and the rotated key part (k_off..).  The first n_rows_form rows' query parts go to qa [rows, heads, row], the
    others stay in place.  Rows of qa and cache: ``latent_row``.  cos and sin are multiplied by mscale."""
    assert qkv.dtype is qa.dtype is cache.dtype and cache.shape[1] == latent_row(rank_p, rot_p) and positions.dtype is torch.int32 and slots.dtype is torch.int64
    _chk(lib().tbv_op_latent_prep(_p(qkv), _p(qa), _p(cache), _p(gamma), _p(inv_freq), _p(positions), _p(slots), qkv.shape[0], n_rows_form,
                                  qkv.stride(0), q_off, c_off, k_off, heads, rank, rank_p, rot_p, inv_freq.shape[0], eps, mscale, _is_bf16(qkv), _st()),
         "tbv_op_latent_prep")
    _count()


def latent_attention_rows(qa, cache, tables, seq_of_row, ctx_lens, sink, out, rank: int, scale: float, block_size: int, splits: int = 1) -> None:
    """qa [rows, heads, row] against the cache rows (keys over all columns of ``latent_row`` but the pad, values = the first out.shape[2] columns); softmax with
    exp(sink) in the denominator (sink fp32 [heads] or None)."""
    rows, H, row = qa.shape
    Rp, Dk = out.shape[2], row - LATENT_ROW_PAD
    assert qa.is_contiguous() and out.is_contiguous() and cache.shape[1] == row and qa.dtype is cache.dtype is out.dtype
    assert tables.dtype is torch.int32 and ctx_lens.dtype is torch.int32
    _chk(lib().tbv_op_latent_attn_rows(_p(qa), _p(cache), _p(tables), _p(seq_of_row), _p(ctx_lens), _p(sink), _p(out), rows, H, rank, Rp, Dk - Rp,
                                       block_size, tables.shape[1], splits, scale, _is_bf16(qa), _st()), "tbv_op_latent_attn_rows")
    _count()


def latent_gather(cache, slots, c, kr) -> None:
    """Cache rows ``slots`` (int64) -> dense latents c [n, Rp] and rotated key parts kr [n, rotp] (bf16)."""
    assert cache.dtype is torch.bfloat16 and slots.dtype is torch.int64 and c.is_contiguous() and kr.is_contiguous()
    _chk(lib().tbv_op_latent_gather(_p(cache), _p(slots), _p(c), _p(kr), slots.shape[0], c.shape[1], kr.shape[1], _st()), "tbv_op_latent_gather")
    _count()


def latent_prefill_fits(dim_p: int, rot_p: int, v_p: int) -> bool:
    return bool(lib().tbv_op_latent_prefill_fits(dim_p, rot_p, v_p))


def latent_attention_prefill(qkv, q_rot_off: int, kv, kr, tiles, sink, out, heads: int, dim_p: int, v_p: int, scale: float) -> None:
    """Many query rows against expanded keys / values: kv [ctx rows, heads * dim_p | heads * v_p], rotated key parts kr [ctx rows, rot_p];
    tiles int32 [n, 4] = (first query row, rows <= 64, first ctx row of the sequence, keys the first row sees)."""
    assert qkv.dtype is kv.dtype is kr.dtype is out.dtype is torch.bfloat16 and tiles.dtype is torch.int32
    _chk(lib().tbv_op_latent_prefill(_p(qkv), _p(kv), _p(kr), _p(tiles), _p(sink), _p(out), tiles.shape[0], heads, qkv.stride(0), q_rot_off,
                                     kv.stride(0), heads * dim_p, out.stride(0), dim_p, kr.shape[1], v_p, scale, _st()), "tbv_op_latent_prefill")
    _count()
