"""Every mechanism of Nubosun on its own: the kernel against a plain statement of the same thing, at sizes that are not multiples of
anything, on inputs made so that a wrong key, edge, sink or state shows."""
import math

import pytest
import torch

import nubosun_oracle as oracle

pytestmark = pytest.mark.gpu
DEV = "cuda:0"
BF, F32 = torch.bfloat16, torch.float32


def pad16(n):
    return (n + 15) // 16 * 16


def close(got, want, dtype, scale=None):
    got, want = got.double().cpu(), want.double().cpu()
    scale = float(want.abs().max()) if scale is None else scale
    err = float((got - want).abs().max()) / max(scale, 1e-20)
    assert err < (1.2e-2 if dtype is BF else 2e-5), err


def rand(*shape, seed=0):
    return torch.randn(*shape, generator=torch.Generator().manual_seed(seed))


def padded(t, cols, dtype):
    out = torch.zeros(*t.shape[:-1], cols, dtype=dtype, device=DEV)
    out[..., : t.shape[-1]] = t.to(dtype)
    return out


# ---- residual streams --------------------------------------------------------------------------------------------------
@pytest.mark.parametrize("streams,width", [(1, 20), (2, 100), (3, 333), (4, 1600), (5, 48), (8, 4096), (2, 9000)])
@pytest.mark.parametrize("dtype", [BF, F32])
def test_streams_mix_norm_and_layer_scale(streams, width, dtype):
    from libtbvcoll_b200 import ops
    T, S, Wp, V, eps = 7, streams, pad16(width), 11, 1e-3
    emb = rand(V, width, seed=1).to(BF).float()
    ids = torch.tensor([3, 0, 10, 3, 7, 1, 2])
    hin, hout, hin2, mix = rand(S, seed=2), rand(S, seed=3), rand(S, seed=4), rand(S, S, seed=5)
    gam, gam2, ls = rand(width, seed=6), rand(width, seed=7), rand(width, seed=8)
    vec = lambda v: padded(v, Wp, F32)
    x, h = torch.full((T, S, Wp), 7.0, device=DEV), torch.empty(T, Wp, dtype=dtype, device=DEV)
    ops.hyper_embed(ids.to(DEV), padded(emb, Wp, dtype), 0.3, x, hin.to(DEV), vec(gam), h, width, eps)
    want = [emb[ids] * 0.3 for _ in range(S)]
    close(x[:, :, :width], torch.stack(want, 1), F32)
    u = sum(hin[s] * want[s] for s in range(S))
    close(h[:, :width], oracle.rms(u, eps) * gam, dtype)
    # streams that differ, then one write-back
    xs = rand(T, S, width, seed=9)
    x.zero_()
    x[:, :, :width] = xs.to(DEV)
    y = rand(T, width, seed=10)
    seen = []
    new = oracle.hyper_sublayer([xs[:, s] for s in range(S)], lambda v: seen.append(v) or y, gam, ls, hin, hout, mix, eps)
    before = x.clone()
    rows = torch.tensor([5, 0, 5], device=DEV)
    last = torch.empty(3, Wp, dtype=dtype, device=DEV)
    args = (padded(y, Wp, F32), vec(ls), hout.to(DEV), mix.to(DEV), x)
    ops.hyper_mix(*args, torch.ones(S, device=DEV), vec(gam2), last, width, eps, rows=rows, last=True)
    assert torch.equal(x, before)
    close(last[:, :width], oracle.rms(sum(new), eps)[[5, 0, 5]] * gam2, dtype)
    ops.hyper_mix(*args, hin2.to(DEV), vec(gam2), h, width, eps)
    close(x[:, :, :width], torch.stack(new, 1), F32)
    close(h[:, :width], oracle.rms(sum(hin2[s] * new[s] for s in range(S)), eps) * gam2, dtype)
    assert not h[:, width:].any() and not x[:, :, width:].any()


# ---- matrix products with the wider epilogues ----------------------------------------------------------------------------
@pytest.mark.parametrize("N,M,K", [(1, 16, 16), (5, 80, 272), (33, 272, 64), (130, 528, 336), (400, 304, 1040), (1100, 1552, 80)])
@pytest.mark.parametrize("dtype,mode", [(F32, 0), (BF, 0), (BF, 1), (BF, 2)])      # mode: selection of the many-token kernel (bf16)
def test_linear_epilogues(persist_mode, N, M, K, dtype, mode):
    from libtbvcoll_b200 import ops
    persist_mode(mode)
    x, w, b = (rand(N, K, seed=1)).to(dtype).to(DEV), (rand(M, K, seed=2) / K ** 0.5).to(dtype).to(DEV), rand(M, seed=3).to(dtype).to(DEV)
    ref = x.double() @ w.double().T + b.double()
    out = torch.empty(N, M, dtype=F32, device=DEV)
    copy = torch.empty(N, M, dtype=BF, device=DEV) if dtype is BF else None
    close(ops.linear(x, w, out, bias=b, copy=copy), ref, F32)
    if copy is not None:
        assert torch.equal(copy, out.to(BF))
    close(ops.linear(x, w, out, bias=b, act=ops.ACT_SOFTPLUS), torch.nn.functional.softplus(ref), F32)
    close(ops.linear(x, w, out, bias=b, act=ops.ACT_SOFTCAP, act_arg=1.5), 1.5 * torch.tanh(ref / 1.5), F32)
    g, u = ref[:, 0::2].clamp(max=0.9), ref[:, 1::2].clamp(-0.9, 0.9)
    act = torch.empty(N, M // 2, dtype=dtype, device=DEV)
    close(ops.linear(x, w, act, bias=b, glu=(0.9, 1.702)), g / (1 + torch.exp(-1.702 * g)) * (u + 1), dtype)
    assert not ops.gemm_error()


@pytest.mark.parametrize("dtype", [BF, F32])
@pytest.mark.parametrize("N,G,M,K,xg,yg", [(3, 5, 48, 32, 48, 56), (40, 3, 144, 16, 16, 160), (70, 2, 272, 208, 208, 272), (1, 33, 16, 512, 512, 16)])
def test_grouped_linear(dtype, N, G, M, K, xg, yg):
    from libtbvcoll_b200 import ops
    x, w = rand(N, (G - 1) * xg + K + 8, seed=1).to(dtype).to(DEV), (rand(G * M, K, seed=2) / K ** 0.5).to(dtype).to(DEV)
    out = torch.full((N, (G - 1) * yg + M + 8), 9.0, dtype=dtype, device=DEV)
    ops.linear(x, w, out, groups=G, x_group=xg, y_group=yg)
    for g in range(G):
        close(out[:, g * yg: g * yg + M], x[:, g * xg: g * xg + K].double() @ w[g * M: (g + 1) * M].double().T, dtype)
        assert bool((out[:, g * yg + M: (g + 1) * yg if g + 1 < G else None] == 9.0).all())          # the gaps between groups are left alone


# ---- convolution and scan ------------------------------------------------------------------------------------------------
def scan_case(inner, state, taps, lens, seed=0):
    """Per sequence: convolution inputs, gate, raw step sizes, B, C; and the plain result over the whole sequence."""
    g = torch.Generator().manual_seed(seed)
    n = lambda *s: torch.randn(*s, generator=g)
    par = {"taps": n(inner, taps) / taps ** 0.5, "bias": 0.3 * n(inner), "a_log": torch.log(0.02 + 3 * torch.rand(inner, state, generator=g)), "d": n(inner)}
    seqs = []
    for L in lens:
        s = {"x": n(L, inner).to(BF).float(), "z": n(L, inner).to(BF).float(), "raw": 1.5 * n(L, inner) - 1.5, "b": n(L, state), "c": n(L, state)}
        s["u"] = oracle.silu(oracle.causal_conv(s["x"], par["taps"], par["bias"]))
        seqs.append(s)
    return par, seqs


def run_scan(par, seqs, schedule, dtype, slots, one_token=False, dirty=5.0):
    """Runs the portions of ``schedule`` ([[(sequence, start, end), ..] per step]) and returns the convolution's and the scan's outputs."""
    from libtbvcoll_b200 import ops
    inner, state = par["a_log"].shape
    taps, ip, ld = par["taps"].shape[1], pad16(inner), pad16(2 * state) + 16
    conv_w, conv_b = padded(par["taps"].T.contiguous(), ip, F32), padded(par["bias"], ip, F32)
    a2, d = (-torch.exp(par["a_log"]) / math.log(2.0)).to(DEV), par["d"].to(DEV)
    nslots = max(slots.values()) + 1
    ssm, conv = torch.full((nslots, inner, state), dirty, device=DEV), torch.full((nslots, taps - 1, ip), dirty, device=DEV)   # what earlier owners left
    us, ys = [torch.zeros_like(s["x"]) for s in seqs], [torch.zeros_like(s["x"]) for s in seqs]
    for step in schedule:
        cat = lambda k: torch.cat([seqs[q][k][a:b] for q, a, b in step])
        T = sum(b - a for _, a, b in step)
        xz = torch.cat((padded(cat("x"), ip, dtype), padded(cat("z"), ip, dtype)), 1)
        dt, bc = padded(cat("raw"), ip, F32), torch.zeros(T, ld, device=DEV)
        bc[:, 8: 8 + state], bc[:, 8 + state: 8 + 2 * state] = cat("b").to(DEV), cat("c").to(DEV)
        segs, seg_of_row, pos, at = [], [], [], 0
        for i, (q, a, b) in enumerate(step):
            segs.append([at, b - a, slots[q], 0])
            seg_of_row += [i] * (b - a)
            pos += range(a, b)
            at += b - a
        segs, pos = torch.tensor(segs, dtype=torch.int32, device=DEV), torch.tensor(pos, dtype=torch.int32, device=DEV)
        sor = None if one_token else torch.tensor(seg_of_row, dtype=torch.int32, device=DEV)
        u = torch.empty(T, ip, dtype=dtype, device=DEV)
        ops.causal_conv_silu(xz, u, conv_w, conv_b, conv, segs, sor, pos)
        u0 = u.clone()
        ops.selective_scan(u, xz, ip, dt, bc, 8, 8 + state, a2, d, ssm, conv, u, segs, pos, one_token=one_token)
        at = 0
        for q, a, b in step:
            us[q][a:b], ys[q][a:b] = u0[at: at + b - a, :inner].float().cpu(), u[at: at + b - a, :inner].float().cpu()
            at += b - a
    return us, ys


@pytest.mark.parametrize("inner,state,taps", [(40, 1, 4), (72, 4, 2), (33, 7, 3), (200, 16, 4), (50, 12, 5), (64, 20, 1), (24, 50, 3), (17, 100, 4),
                                              (20, 200, 2), (1040, 16, 4)])
@pytest.mark.parametrize("dtype", [BF, F32])
def test_scan_over_portions(inner, state, taps, dtype):
    """Whole sequences, then the same in portions of changing size side by side with other sequences, state slots in any order and dirty from
    earlier owners, then a sequence that starts in a slot another has used."""
    lens = (97, 41, 70)
    par, seqs = scan_case(inner, state, taps, lens)
    want_y = []
    for s in seqs:
        u = s["u"].to(dtype).float()
        y = oracle.selective_scan(u, oracle.softplus(s["raw"]), par["a_log"], s["b"], s["c"], par["d"])
        want_y.append(y * oracle.silu(s["z"]))
    slots = {0: 3, 1: 1, 2: 3}                                     # the third follows the first in its slot
    whole = [[(0, 0, 97), (1, 0, 41)], [(2, 0, 70)]]
    cut, at = [], {0: 0, 1: 0}
    for n0, n1 in [(1, 2), (2, 1), (3, 3), (1, 1), (34, 2), (32, 30), (24, 2)]:
        cut.append([(0, at[0], at[0] + n0), (1, at[1], at[1] + n1)])
        at[0] += n0
        at[1] += n1
    assert at == {0: 97, 1: 41}
    cut += [[(2, 0, 2)], [(2, 2, 3)], [(2, 3, 67)], [(2, 67, 70)]]
    for schedule in (whole, cut):
        us, ys = run_scan(par, seqs, schedule, dtype, slots)
        for q in range(3):
            close(us[q], seqs[q]["u"], dtype)
            close(ys[q], want_y[q], dtype)
    # the first part as a portion, the rest token by token through the one-token form
    mixed = [[(0, 0, 50), (1, 0, 1)]] + [[(1, t + 1, t + 2), (0, 50 + t, 51 + t)] for t in range(40)]
    us, ys = run_scan(par, seqs, mixed[:1], dtype, slots)
    us2, ys2 = run_scan(par, seqs, [[(1, t, t + 1)] for t in range(41)], dtype, slots, one_token=True)
    close(ys2[1], want_y[1], dtype)
    close(us2[1], seqs[1]["u"], dtype)
    us3, ys3 = run_scan(par, seqs, mixed, dtype, slots)
    close(ys3[0][:90], want_y[0][:90], dtype)
    close(ys3[1], want_y[1], dtype)


@pytest.mark.parametrize("dtype", [BF, F32])
def test_scan_remembers_far_back_and_small_steps(dtype):
    """One early input with a near-zero decay must still show 900 tokens later, through many portions; tiny steps (softplus of -12) keep their
    relative accuracy."""
    inner, state, L = 16, 4, 1000
    par, seqs = scan_case(inner, state, 2, (L,), seed=3)
    s = seqs[0]
    par["a_log"].fill_(-9.0)
    s["raw"].fill_(-12.0)
    s["raw"][5] = 20.0
    s["x"][5], s["b"][5], s["c"][:] = 3.0, 2.0, 1.0
    s["u"] = oracle.silu(oracle.causal_conv(s["x"], par["taps"], par["bias"])).to(dtype).float()
    y = oracle.selective_scan(s["u"], oracle.softplus(s["raw"]), par["a_log"], s["b"], s["c"], par["d"] * 0) * oracle.silu(s["z"])
    par["d"] = par["d"] * 0
    cuts = [0, 3, 6, 260, 512, 515, 900, 1000]
    _, ys = run_scan(par, seqs, [[(0, a, b)] for a, b in zip(cuts, cuts[1:])], dtype, {0: 1})
    assert y[950].abs().mean() > 1.0
    close(ys[0], y, dtype)
    early = slice(0, 5)                                            # before the large input: outputs of size 1e-5 and less
    close(ys[0][early], y[early], dtype)


# ---- latent attention ------------------------------------------------------------------------------------------------------
class Cache:
    """Latent rows of a few sequences in scattered blocks."""

    def __init__(self, lens, R, rot, dtype, block=16, seed=0, loud=()):
        from libtbvcoll_b200 import ops
        self.R, self.rot, self.Rp, self.rp, self.block = R, rot, pad16(R), pad16(rot), block
        n = [(L + block - 1) // block for L in lens]
        order = torch.randperm(sum(n), generator=torch.Generator().manual_seed(seed)) + 1
        self.tables = torch.zeros(len(lens), max(n), dtype=torch.int32)
        self.cache = torch.full(((sum(n) + 1) * block, ops.latent_row(self.Rp, self.rp)), 3.0, dtype=dtype, device=DEV)
        self.rows, at = [], 0
        for i, L in enumerate(lens):
            self.tables[i, : n[i]] = order[at: at + n[i]]
            at += n[i]
            r = rand(L, R + rot, seed=seed + i + 1).to(BF).float()
            self.rows.append(r)
            slot = torch.tensor([self.slot(i, t) for t in range(L)], device=DEV)
            full = torch.zeros(L, self.cache.shape[1], dtype=dtype, device=DEV)
            full[:, :R], full[:, self.Rp: self.Rp + rot] = r[:, :R].to(dtype), r[:, R:].to(dtype)
            self.cache[slot] = full

    def slot(self, i, t):
        return int(self.tables[i, t // self.block]) * self.block + t % self.block


def attend(q, keys, values, scale, sink, visible):
    """q [H, D]; keys [T, D] or [H, T, D]; plain float64 with the sink in the denominator."""
    k = keys[None] if keys.dim() == 2 else keys
    v = values[None] if values.dim() == 2 else values
    s = (q[:, None].double() * k[:, :visible].double()).sum(-1) * scale
    e = torch.exp(s - s.amax(1, keepdim=True).clamp(min=0))
    den = e.sum(1, keepdim=True) + (torch.exp(sink.double()[:, None] - s.amax(1, keepdim=True).clamp(min=0)) if sink is not None else 0)
    return ((e / den)[..., None] * v[:, :visible].double()).sum(1)


@pytest.mark.parametrize("dtype", [BF, F32])
@pytest.mark.parametrize("H,R,rot,block", [(1, 20, 6, 16), (5, 112, 32, 16), (16, 52, 10, 16), (17, 160, 64, 8), (33, 512, 64, 32), (3, 700, 16, 16), (2, 40, 2, 1)])
def test_latent_rows_attention(dtype, H, R, rot, block):
    from libtbvcoll_b200 import ops
    lens = (1, 15, 16, 17, 63, 64, 65, 130, 333)
    c = Cache(lens, R, rot, dtype, block)
    rows = [(i, n) for i, L in enumerate(lens) for n in sorted({1, 2, L // 2, L - 1, L}) if 0 < n <= L]
    scale = 0.7 / math.sqrt(R + rot)
    q = rand(len(rows), H, R + rot, seed=50).to(BF).float() * 2
    for j, (i, n) in enumerate(rows):                  # one key stands out for the first head: the first, a middle one, or the last one seen
        q[j, 0] = (c.rows[i][(0, n // 2, n - 1)[j % 3]] * 1.5).to(BF).float()
    sink = rand(H, seed=51)
    qa = torch.zeros(len(rows), H, c.cache.shape[1], dtype=dtype, device=DEV)
    qa[..., :R], qa[..., c.Rp: c.Rp + rot] = q[..., :R].to(dtype).to(DEV), q[..., R:].to(dtype).to(DEV)
    seq, ctx = (torch.tensor(v, dtype=torch.int32, device=DEV) for v in zip(*rows))
    for sk in (sink, None, sink + 60.0):
        want = torch.stack([attend(q[j], c.rows[i], c.rows[i][:, :R], scale, sk, n) for j, (i, n) in enumerate(rows)])
        for splits in (1, 3, 8) if dtype is BF else (1,):
            out = torch.full((len(rows), H, c.Rp), 5.0, dtype=dtype, device=DEV)
            ops.latent_attention_rows(qa, c.cache, c.tables.to(DEV), seq, ctx, None if sk is None else sk.to(DEV), out, R, scale, block, splits=splits)
            close(out[..., :R], want, dtype, scale=float(want.abs().max()) if sk is not None and sk is not sink else 1.0)
            assert not out[..., R:].any()
    assert not ops.gemm_error()


def test_latent_rows_far_key_beside_a_sink():
    """Hundreds of keys of no weight, one far back that carries the row, in fp32 and bf16; moving the visible end by one hides it."""
    from libtbvcoll_b200 import ops
    L, H, R, rot, at = 777, 2, 96, 16, 700
    for dtype in (BF, F32):
        c = Cache((L,), R, rot, dtype)
        q = torch.stack([c.rows[0][at] * 3, c.rows[0][at] * 3]).to(BF).float()
        qa = torch.zeros(2, H, c.cache.shape[1], dtype=dtype, device=DEV)
        qa[..., :R], qa[..., c.Rp: c.Rp + rot] = q[None, :, :R].to(dtype).to(DEV), q[None, :, R:].to(dtype).to(DEV)
        out = torch.empty(2, H, c.Rp, dtype=dtype, device=DEV)
        seq, ctx = torch.zeros(2, dtype=torch.int32, device=DEV), torch.tensor([at + 1, at], dtype=torch.int32, device=DEV)
        sink = torch.tensor([-2.0, 2.0])
        ops.latent_attention_rows(qa, c.cache, c.tables.to(DEV), seq, ctx, sink.to(DEV), out, R, 0.1, 16, splits=8)
        want = torch.stack([attend(q, c.rows[0], c.rows[0][:, :R], 0.1, sink, n) for n in (at + 1, at)])
        close(out, want, dtype)
        assert (want[0] - c.rows[0][at, :R]).abs().max() < 0.2 and (want[1] - c.rows[0][at, :R]).abs().max() > 1.0


@pytest.mark.parametrize("H,dim,rot,vd", [(1, 24, 6, 20), (3, 64, 48, 80), (2, 128, 64, 128), (5, 16, 16, 48), (2, 192, 64, 256), (4, 40, 2, 90)])
def test_latent_prefill_attention(H, dim, rot, vd):
    """Several sequences with their visible starts at different places in the context; tiles end anywhere."""
    from libtbvcoll_b200 import ops
    from libtbvcoll_b200.engine.batch import dense_context
    Dp, rp, vp = pad16(dim), pad16(rot), pad16(vd)
    parts = [(0, 64), (0, 65), (100, 33), (63, 130), (511, 2), (0, 1)]               # (start, rows)
    T, C = sum(n for _, n in parts), sum(s + n for s, n in parts)
    first = [sum(n for _, n in parts[:i]) for i in range(len(parts))]
    import numpy as np
    tiles, _ = dense_context(first, [n for _, n in parts], [s for s, _ in parts], [0] * len(parts), np.zeros((1, 64), dtype=np.int32), 16)
    q, k, kr, v = rand(T, H, dim + rot, seed=1).to(BF).float(), rand(C, H, dim, seed=2).to(BF).float(), rand(C, rot, seed=3).to(BF).float(), rand(C, H, vd, seed=4).to(BF).float()
    base = [sum(s + n for s, n in parts[:i]) for i in range(len(parts))]
    for (s, n), f, b in zip(parts, first, base):                  # every row's own key stands out, and every third row's first key
        for r in range(n):
            key = b + (0 if r % 3 == 0 else s + r)
            q[f + r, 0] = (torch.cat((k[key, 0], kr[key])) * 2).to(BF).float()
    sink = rand(H, seed=5)
    qkv = torch.zeros(T, H * (Dp + rp) + 16, dtype=BF, device=DEV)
    qkv[:, : H * Dp].view(T, H, Dp)[..., :dim] = q[..., :dim].to(BF).to(DEV)
    qkv[:, H * Dp: H * (Dp + rp)].view(T, H, rp)[..., :rot] = q[..., dim:].to(BF).to(DEV)
    kv = torch.zeros(C, H * (Dp + vp), dtype=BF, device=DEV)
    kv[:, : H * Dp].view(C, H, Dp)[..., :dim] = k.to(BF).to(DEV)
    kv[:, H * Dp:].view(C, H, vp)[..., :vd] = v.to(BF).to(DEV)
    scale = 1.3 / math.sqrt(dim + rot)
    for sk in (sink, None):
        out = torch.full((T, H * vp), 5.0, dtype=BF, device=DEV)
        ops.latent_attention_prefill(qkv, H * Dp, kv, padded(kr, rp, BF), torch.from_numpy(tiles).to(DEV), None if sk is None else sk.to(DEV), out, H, Dp, vp, scale)
        got = out.view(T, H, vp)[..., :vd].cpu()
        for (s, n), f, b in zip(parts, first, base):
            keys = torch.cat((k[b: b + s + n], kr[b: b + s + n, None].expand(-1, H, -1)), -1).transpose(0, 1)
            vals = v[b: b + s + n].transpose(0, 1)
            for r in sorted({0, 1, n // 2, n - 2, n - 1, min(63, n - 1), min(64, n - 1)} & set(range(n))):
                close(got[f + r], attend(q[f + r], keys, vals, scale, sk, s + r + 1), BF, scale=1.0)


@pytest.mark.parametrize("dtype", [BF, F32])
@pytest.mark.parametrize("H,dim,rot,R,dims", [(3, 24, 10, 52, 10), (1, 48, 32, 160, 32), (5, 16, 24, 300, 12), (20, 128, 64, 512, 64)])
def test_latent_prep_rotates_norms_and_writes_the_cache(dtype, H, dim, rot, R, dims):
    from libtbvcoll_b200 import ops
    Dp, rp, Rp, T, nf, eps = pad16(dim), pad16(rot), pad16(R), 9, 4, 1e-2
    spec = {"dims": dims, "base": 300.0, "scaling": {"factor": 3.0, "original": 50, "fast": 8.0, "slow": 1.0}}
    freq, factor = ops.rope_frequencies(dims, spec["base"], spec["scaling"])
    pos = torch.tensor([0, 1, 2, 777, 3, 50, 4096, 5, 100000], dtype=torch.int32)
    qr, c, kr = (rand(T, *s, seed=i).to(BF).float() for i, s in enumerate(((H, rot), (R,), (rot,))))
    gam = rand(R, seed=9)
    cols = H * (Dp + rp) + Rp + rp
    qkv = torch.zeros(T, cols, dtype=dtype, device=DEV)
    qkv[:, H * Dp: H * (Dp + rp)].view(T, H, rp)[..., :rot] = qr.to(dtype).to(DEV)
    co = H * (Dp + rp)
    qkv[:, co: co + R], qkv[:, co + Rp: co + Rp + rot] = c.to(dtype).to(DEV), kr.to(dtype).to(DEV)
    row = ops.latent_row(Rp, rp)
    qa, cache = torch.zeros(nf, H, row, dtype=dtype, device=DEV), torch.full((40, row), 4.0, dtype=dtype, device=DEV)
    slots = torch.tensor([33, 2, 3, 17, 18, 19, 30, 1, 39])
    ops.latent_prep(qkv, qkv, qa, cache, gam.to(DEV), ops.frequency_turns(freq, DEV), factor, pos.to(DEV), slots.to(DEV), nf, H * Dp, co, co + Rp, H, R, Rp, rp, eps)
    # angles, factor aside
    ang = pos.double()[:, None] * freq[None]
    cos, sin = torch.cos(ang) * factor, torch.sin(ang) * factor

    def turn(x):
        out = x.double().clone()
        a, b = x[..., 0:dims:2].double(), x[..., 1:dims:2].double()
        cc, ss = (cos, sin) if x.dim() == 2 else (cos[:, None], sin[:, None])
        out[..., 0:dims:2], out[..., 1:dims:2] = a * cc - b * ss, b * cc + a * ss
        return out
    got = cache[slots.to(DEV)]
    close(got[:, :R], oracle.rms(c, eps) * gam, dtype)
    close(got[:, Rp: Rp + rot], turn(kr), dtype)
    assert not got[:, R:Rp].any()
    close(qa[..., Rp: Rp + rot], turn(qr)[:nf], dtype)
    close(qkv[nf:, H * Dp: H * (Dp + rp)].view(T - nf, H, rp)[..., :rot], turn(qr)[nf:], dtype)
    untouched = torch.ones(40, dtype=torch.bool)
    untouched[slots] = False
    assert bool((cache[untouched.to(DEV)] == 4.0).all())
    # the plain rotation agrees with the oracle's where the angles are small
    small = torch.tensor([0, 1, 2, 4])
    plain = oracle.rotate_pairs(qr[small], pos[small].float(), spec)
    close(turn(qr)[small], plain, F32)


def test_latent_gather():
    from libtbvcoll_b200 import ops
    cache = rand(64, ops.latent_row(48, 16)).to(BF).to(DEV)
    slots = torch.tensor([5, 63, 0, 17, 5], device=DEV)
    c, kr = torch.empty(5, 48, dtype=BF, device=DEV), torch.empty(5, 16, dtype=BF, device=DEV)
    ops.latent_gather(cache, slots, c, kr)
    assert torch.equal(c, cache[slots, :48]) and torch.equal(kr, cache[slots, 48:64])


def test_argmax_of_fp32_logits():
    from libtbvcoll_b200 import ops
    x = rand(5, 10007).to(DEV)
    x[2, 77] = x[2, 9000] = 50.0
    x[3] += torch.arange(10007, device=DEV) * 1e-9
    ws = ops.argmax_workspace(5, DEV)
    val, idx = ops.argmax(x, ws)
    assert idx[2] == 77 and torch.equal(idx, x.argmax(1)) and torch.equal(val, x.amax(1))
