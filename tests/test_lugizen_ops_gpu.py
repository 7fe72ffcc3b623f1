"""Every mechanism of Lugizen on its own: the kernel against a plain statement of the same thing, at sizes that are not multiples of
anything, on inputs made so that a wrong key, edge, decay, state or tap shows."""
import math

import numpy as np
import pytest
import torch

import lugizen_oracle as oracle

pytestmark = pytest.mark.gpu
DEV = "cuda:0"
BF, F32 = torch.bfloat16, torch.float32
I32 = dict(dtype=torch.int32, device=DEV)


def pad16(n):
    return (n + 15) // 16 * 16


def close(got, want, dtype, tol=None):
    got, want = got.double().cpu(), want.double().cpu()
    err = float((got - want).abs().max()) / max(float(want.abs().max()), 1e-20)
    assert err < (tol or (1.2e-2 if dtype is BF else 2e-5)), err


def rand(*shape, seed=0):
    return torch.randn(*shape, generator=torch.Generator().manual_seed(seed))


def padded(t, cols, dtype):
    out = torch.zeros(*t.shape[:-1], cols, dtype=dtype, device=DEV)
    out[..., : t.shape[-1]] = t.to(dtype)
    return out


def pad_heads(t, dtype):
    """[T, H, D] -> [T, H * pad16(D)]"""
    return padded(t, pad16(t.shape[-1]), dtype).flatten(1)


def ragged(lens, starts, slots):
    """(segs, segment of row, positions) of segments with the given rows, first positions and state slots."""
    first = np.cumsum([0] + list(lens[:-1]))
    segs = torch.tensor([[int(f), n, s, 0] for f, n, s in zip(first, lens, slots)], **I32)
    seg = torch.repeat_interleave(torch.arange(len(lens)), torch.tensor(lens)).to(**I32)
    pos = torch.cat([torch.arange(s, s + n) for s, n in zip(starts, lens)]).to(**I32)
    return segs, seg, pos


# ---- residual stream --------------------------------------------------------------------------------------------------------
@pytest.mark.parametrize("width,taps", [(20, 1), (100, 3), (2048, 4), (4096, 2), (9000, 6)])
@pytest.mark.parametrize("dtype", [BF, F32])
def test_norm_behind_and_the_convolution_of_one_row_per_sequence(width, taps, dtype):
    from libtbvcoll_b200 import ops
    T, Wp, eps, slots = 5, pad16(width), 1e-4, [4, 1, 6, 2, 3]
    x, y, g = rand(T, width, seed=1), 30.0 * rand(T, width, seed=2), 1.3
    w, past = rand(width, taps, seed=3), rand(8, taps - 1, width, seed=4)
    segs, _, pos = ragged([1] * T, [0, 9, 1, 0, 50], slots)
    full = lambda t: padded(t, Wp, F32)
    gain = full(torch.full((width,), g))
    want = x + oracle.scalar_norm(y, g, eps)
    xd, h = full(x), torch.full((T, Wp), 9.0, dtype=dtype, device=DEV)
    ops.residual(xd, None, h, width, eps, post=gain, y1=full(y))
    close(xd[:, :width], want, F32)
    close(h[:, :width], want, dtype)
    assert not xd[:, width:].any() and not h[:, width:].any()
    only = full(x)
    ops.residual(only, None, None, width, eps, post=gain, y1=full(y))
    assert torch.equal(only, xd)
    xd, state = full(x), full(past)
    ops.residual(xd, None, h, width, eps, post=gain, y1=full(y), positions=pos, conv=(full(w.t()), state, segs))
    new = past.clone()
    for r, s in enumerate(slots):
        before = torch.zeros(taps - 1, width) if int(pos[r]) == 0 else past[s]
        rows = torch.cat((before, want[r: r + 1]))
        close(h[r, :width], want[r] + (rows * w.t()).sum(0), dtype)
        new[s] = rows[1:]
    close(state[:, :, :width], new, F32) if taps > 1 else None
    assert torch.equal(only, xd)
    emb, ids = rand(9, width, seed=5).to(BF).float(), torch.tensor([3, 8, 0, 3, 1])
    state = full(past)
    ops.residual(xd, None, h, width, eps, embed=(ids.to(DEV), padded(emb, Wp, dtype), 1.0, None), positions=pos, conv=(full(w.t()), state, segs))
    assert torch.equal(xd[:, :width].cpu(), emb[ids])
    before = torch.stack([torch.zeros(taps - 1, width) if int(pos[r]) == 0 else past[s] for r, s in enumerate(slots)])
    close(h[:, :width], emb[ids] + (torch.cat((before, emb[ids][:, None]), 1) * w.t()).sum(1), dtype)


@pytest.mark.parametrize("add", [True, False])
@pytest.mark.parametrize("taps", [1, 2, 3, 4, 6])
@pytest.mark.parametrize("dtype", [BF, F32])
def test_short_convolution_in_portions(dtype, taps, add):
    """Sequences cut into portions of one, two and many rows, beside each other; what a slot's previous owner left is not seen."""
    from libtbvcoll_b200 import ops
    C, Cp = 44, 48
    full = {k: rand(n, C, seed=i).to(F32 if add else dtype).float() for i, (k, n) in enumerate((("a", 150), ("b", 40), ("c", 9)))}
    w = rand(C, taps, seed=7)
    want = {k: (t + oracle.causal_conv(t, w) if add else oracle.silu(oracle.causal_conv(t, w))) for k, t in full.items()}
    state = torch.full((5, taps - 1, Cp), 77.0, device=DEV)
    slot, at, got = {"a": 3, "b": 1, "c": 4}, dict.fromkeys("abc", 0), {k: [] for k in full}
    wd = padded(w.t(), Cp, F32)
    for step in ([("a", 1), ("b", 2)], [("b", 1), ("a", 2), ("c", 9)], [("a", 70), ("b", 3)], [("a", 1), ("b", 33)], [("a", 76), ("b", 1)]):
        lens, keys = [n for _, n in step], [k for k, _ in step]
        segs, seg, pos = ragged(lens, [at[k] for k in keys], [slot[k] for k in keys])
        x = padded(torch.cat([full[k][at[k]: at[k] + n] for k, n in step]), Cp + 16, F32 if add else dtype)
        x[:, Cp:] = 5.0                                                    # columns beside the convolution's
        out = torch.empty(x.shape[0], Cp, dtype=dtype, device=DEV)
        ops.short_conv(x, out, wd, state, segs, None if max(lens) == 1 else seg, pos, add=add)
        f = 0
        for k, n in step:
            got[k].append(out[f: f + n, :C])
            at[k] += n
            f += n
            if taps > 1 and at[k] >= taps - 1:
                close(state[slot[k], :, :C], full[k][at[k] - taps + 1: at[k]], F32)
    for k in full:
        close(torch.cat(got[k]), want[k][: at[k]], dtype)
    assert float(state[0].min()) == 77.0 if taps > 1 else True


# ---- epilogues ----------------------------------------------------------------------------------------------------------------
@pytest.mark.parametrize("N,K,M", [(1, 100, 176), (7, 640, 80), (40, 4096, 144), (200, 64, 400), (600, 320, 1040), (1500, 128, 2064), (20, 4096, 2112)])
@pytest.mark.parametrize("dtype", [BF, F32])
def test_gelu_and_softplus_of_products(N, K, M, dtype, persist_mode):
    """Every form of the product: split and plain decode form, both tiles of the many-token form.  Softplus keeps its relative precision where it is tiny."""
    from libtbvcoll_b200 import ops
    Kp = pad16(K)
    x, w, b = rand(N, K, seed=1).to(dtype).float(), (2.0 * rand(M, K, seed=2) / K ** 0.5).to(dtype).float(), (4 * rand(M, seed=3) - 5).to(dtype).float()
    z = x.double() @ w.double().T
    xd, wd = padded(x, Kp, dtype), padded(w, Kp, dtype)
    for mode in ((1, 2, 3) if N >= 384 and dtype is BF else (1,)):
        persist_mode(mode)
        out = torch.empty(N, M, dtype=dtype, device=DEV)
        ops.linear(xd, wd, out, act=ops.ACT_GELU, act_cols=M)
        close(out, oracle.gelu_tanh(z), dtype)
        sp = torch.empty(N, M, device=DEV)
        ops.linear(xd, wd, sp, bias=b.to(dtype).to(DEV), act=ops.ACT_SOFTPLUS)
        want = oracle.softplus(z + b)
        assert float(((sp.double().cpu() - want) / want).abs().max()) < 2e-5
    assert not ops.gemm_error()


# ---- attention: norms per head, value mix -----------------------------------------------------------------------------------------
@pytest.mark.parametrize("H,G,dim,vdim,rot", [(6, 2, 40, 24, 12), (3, 3, 20, 44, 20), (20, 1, 128, 112, 0), (4, 2, 272, 16, 100), (2, 1, 16, 300, 2)])
@pytest.mark.parametrize("dtype", [BF, F32])
def test_norms_per_head_rotation_value_mix_and_cache(dtype, H, G, dim, vdim, rot):
    """Neighbouring channels are turned: the layout in which i and i + dims / 2 of the checkpoint lie next to each other."""
    from libtbvcoll_b200 import ops
    T, nf, bs, eps, base = 9, 4, 16, 1e-3, 300.0
    Dp, Vp = pad16(dim), pad16(vdim)
    q, k, v, first = (rand(T, n, d, seed=i).to(BF).float() for i, (n, d) in enumerate(((H, dim), (G, dim), (G, vdim), (G, vdim))))
    pos = torch.tensor([0, 1, 2, 777, 3, 50, 4096, 5, 100000])
    order = [j for i in range(rot // 2) for j in (i, i + rot // 2)] + list(range(rot, dim))

    def turned(x):
        y = x.double().clone()
        a = pos.double()[:, None, None] * base ** (-2.0 * torch.arange(rot // 2, dtype=torch.float64) / max(rot, 1))
        u, s = x[:, :, : rot // 2].double(), x[:, :, rot // 2: rot].double()
        y[:, :, : rot // 2], y[:, :, rot // 2: rot] = u * a.cos() - s * a.sin(), s * a.cos() + u * a.sin()
        return oracle.rms(y, eps)[:, :, order]
    scale = 0.5 + rand(H, seed=8).abs()
    turns = ops.rotation_turns(rot, base, DEV) if rot else None
    slots = torch.tensor([33, 2, 3, 17, 18, 19, 30, 1, 39])
    for mix in (None, "store", 0.3):
        wide = torch.cat((pad_heads(q[:, :, order], dtype), pad_heads(k[:, :, order], dtype), pad_heads(v, dtype)), 1)
        qa, cache = torch.zeros(nf, H, Dp + 8, dtype=dtype, device=DEV), torch.full((3 * G * bs, Dp + Vp + 8), 4.0, dtype=dtype, device=DEV)
        vf = pad_heads(first, dtype)
        ops.head_attention_prep(wide, qa, cache, scale.to(DEV), turns, pos.to(**I32), slots.to(DEV), nf, H, G, dim, Dp, bs, eps, v_first=None if mix is None else vf,
                                mix=torch.tensor([mix], device=DEV) if isinstance(mix, float) else None)
        want = turned(q) * scale[:, None]
        close(qa[..., :dim], want[:nf], dtype)
        close(wide[nf:, : H * Dp].view(T - nf, H, Dp)[..., :dim], want[nf:], dtype)
        rows = torch.stack([cache[(s // bs * G + g) * bs + s % bs] for s in slots.tolist() for g in range(G)]).view(T, G, -1)
        close(rows[..., :dim], turned(k), dtype)
        close(rows[..., Dp: Dp + vdim], oracle.value_mix(v, first, mix) if isinstance(mix, float) else v, dtype)
        if mix == "store":
            close(vf.view(T, G, Vp)[..., :vdim], v, dtype)
        untouched = torch.ones(cache.shape[0], dtype=torch.bool)
        for s in slots.tolist():
            for g in range(G):
                untouched[(s // bs * G + g) * bs + s % bs] = False
        assert float(cache[untouched.to(DEV)].float().min()) == 4.0


# ---- latent attention: query latent, windows ---------------------------------------------------------------------------------------
@pytest.mark.parametrize("H,dim,rot,R,Q", [(3, 24, 10, 52, 36), (1, 48, 32, 160, 300), (20, 16, 64, 512, 16)])
@pytest.mark.parametrize("dtype", [BF, F32])
def test_latent_prep_in_two_parts(dtype, H, dim, rot, R, Q):
    from libtbvcoll_b200 import ops
    Dp, rp, Rp, Qp, T, nf, eps = pad16(dim), pad16(rot), pad16(R), pad16(Q), 6, 2, 1e-2
    pos = torch.tensor([0, 1, 777, 3, 4096, 100000])
    cq, c, kr, q = (rand(T, *s, seed=i).to(BF).float() for i, s in enumerate(((Q,), (R,), (rot,), (H, dim + rot))))
    gam, gq = rand(R, seed=9), rand(Q, seed=10)
    low = torch.cat((padded(cq, Qp, dtype), padded(c, Rp, dtype), padded(kr, rp, dtype)), 1)
    qd = torch.cat((pad_heads(q[:, :, :dim], dtype), pad_heads(q[:, :, dim:], dtype)), 1)
    row = ops.latent_row(Rp, rp)
    qa, cache = torch.zeros(nf, H, row, dtype=dtype, device=DEV), torch.full((40, row), 4.0, dtype=dtype, device=DEV)
    slots, turns = torch.tensor([33, 2, 3, 17, 30, 39]), ops.rotation_turns(rot, 300.0, DEV)
    args = (turns, 1.0, pos.to(**I32), slots.to(DEV), nf, H * Dp, Qp, Qp + Rp, H, R, Rp, rp, eps)
    ops.latent_prep(low, None, None, cache, gam.to(DEV), *args, query_latent=(0, Q, gq.to(DEV)))
    ang = pos.double()[:, None] * 300.0 ** (-2.0 * torch.arange(rot // 2, dtype=torch.float64) / rot)

    def turned(x, rows=slice(None)):
        a = ang[rows] if x.dim() == 2 else ang[rows, None]
        u, v = x[..., 0::2].double(), x[..., 1::2].double()
        return torch.stack((u * a.cos() - v * a.sin(), v * a.cos() + u * a.sin()), -1).flatten(-2)
    close(low[:, :Q], oracle.rms(cq, eps) * gq, dtype)
    assert not low[:, Q:Qp].any()
    close(cache[slots.to(DEV)][:, :R], oracle.rms(c, eps) * gam, dtype)
    close(cache[slots.to(DEV)][:, Rp: Rp + rot], turned(kr), dtype)
    untouched = torch.ones(40, dtype=torch.bool)
    untouched[slots] = False
    assert float(cache[untouched.to(DEV)].float().min()) == 4.0
    before = cache.clone()
    ops.latent_prep(None, qd, qa, cache, None, *args)
    assert torch.equal(cache, before)
    close(qa[:, :, Rp: Rp + rot], turned(q[:nf, :, dim:], slice(nf)), dtype)
    close(qd[nf:, H * Dp:].view(T - nf, H, rp)[..., :rot], turned(q[nf:, :, dim:], slice(nf, None)), dtype)
    close(qd[:, : H * Dp].view(T, H, Dp)[..., :dim], q[:, :, :dim], dtype)


def attend(q, keys, values, scale, lo, hi):
    """q [H, D], keys [H, T, D], values [H, T, V]; keys lo .. hi - 1 are visible."""
    p = torch.softmax((q[:, None].double() * keys[:, lo:hi].double()).sum(-1) * scale, -1)
    return (p[..., None] * values[:, lo:hi].double()).sum(1)


@pytest.mark.parametrize("window", [1, 2, 16, 33, 64, 100, 1000])
@pytest.mark.parametrize("H,R,rot,block", [(5, 112, 32, 16), (17, 52, 10, 8), (3, 700, 16, 16)])
@pytest.mark.parametrize("dtype", [BF, F32])
def test_latent_rows_with_a_window(dtype, H, R, rot, block, window):
    """For some heads one key stands out: the first that is visible, the one just before it, or a row's own."""
    from libtbvcoll_b200 import ops
    L, Rp, rp = 333, pad16(R), pad16(rot)
    nb = -(-L // block)
    tables = torch.randperm(nb, generator=torch.Generator().manual_seed(3)).to(torch.int32)[None] + 1
    keys = rand(L, R + rot, seed=1).to(BF).float()
    cache = torch.full(((nb + 1) * block, ops.latent_row(Rp, rp)), 3.0, dtype=dtype, device=DEV)
    slot = tables[0, torch.arange(L) // block].long() * block + torch.arange(L) % block
    cache[slot.to(DEV)] = torch.cat((padded(keys[:, :R], Rp, dtype), padded(keys[:, R:], rp, dtype), torch.zeros(L, 8, dtype=dtype, device=DEV)), 1)
    seen = sorted({1, 2, 15, 17, 64, 130, window, window + 1, window + 16, L} & set(range(1, L + 1)))
    q = rand(len(seen), H, R + rot, seed=2).to(BF).float()
    for j, n in enumerate(seen):
        lo = max(0, n - window)
        for h, at in enumerate((lo, max(0, lo - 1), n - 1)):
            q[j, h] = keys[at].to(BF).float() * 1.5
    qa = torch.zeros(len(seen), H, cache.shape[1], dtype=dtype, device=DEV)
    qa[..., :R], qa[..., Rp: Rp + rot] = q[..., :R].to(dtype).to(DEV), q[..., R:].to(dtype).to(DEV)
    scale = 0.7 / math.sqrt(R + rot)
    k = keys[None].expand(H, -1, -1)
    want = torch.stack([attend(q[j], k, k[..., :R], scale, max(0, n - window), n) for j, n in enumerate(seen)])
    for splits in (1, 3, 8) if dtype is BF else (1,):
        out = torch.full((len(seen), H, Rp), 5.0, dtype=dtype, device=DEV)
        ops.latent_attention_rows(qa, cache, tables.to(DEV), torch.zeros(len(seen), **I32), torch.tensor(seen, **I32), None, out, R, scale, block, splits=splits, window=window)
        close(out[..., :R], want, dtype)
    assert not ops.gemm_error()


@pytest.mark.parametrize("window", [1, 2, 63, 64, 65, 130, 5000])
@pytest.mark.parametrize("H,dim,rot,vd", [(3, 24, 6, 20), (2, 128, 64, 128), (2, 40, 2, 250)])
def test_latent_prefill_with_a_window(H, dim, rot, vd, window):
    """Portions that start anywhere; only the context that some row can see is there."""
    from libtbvcoll_b200 import ops
    from libtbvcoll_b200.engine.batch import dense_context
    Dp, rp, vp = pad16(dim), pad16(rot), pad16(vd)
    parts = [(0, 64), (0, 65), (100, 33), (263, 130), (511, 2), (0, 1)]              # (start, rows)
    T = sum(n for _, n in parts)
    first = [sum(n for _, n in parts[:i]) for i in range(len(parts))]
    tables = np.arange(len(parts) * 64, dtype=np.int32).reshape(len(parts), 64)
    tiles, slots = dense_context(first, [n for _, n in parts], [s for s, _ in parts], list(range(len(parts))), tables, 16, window)
    N = len(parts) * 64 * 16                                                          # every sequence has its own 1024 slots
    q, k, kr, v = rand(T, H, dim + rot, seed=1).to(BF).float(), rand(N, H, dim, seed=2).to(BF).float(), rand(N, rot, seed=3).to(BF).float(), rand(N, H, vd, seed=4).to(BF).float()
    keys = torch.cat((k, kr[:, None].expand(-1, H, -1)), -1)
    for i, ((s, n), f) in enumerate(zip(parts, first)):       # the first visible key, the one before it or a row's own stands out
        for r in range(n):
            lo = max(0, s + r + 1 - window)
            q[f + r, 0] = (keys[i * 1024 + (lo, max(0, lo - 1), s + r)[r % 3], 0] * 2).to(BF).float()
    qkv = torch.cat((pad_heads(q[..., :dim], BF), pad_heads(q[..., dim:], BF)), 1)
    C = torch.from_numpy(slots)
    kv = torch.cat((pad_heads(k[C], BF), pad_heads(v[C], BF)), 1)
    scale, out = 1.3 / math.sqrt(dim + rot), torch.full((T, H * vp), 5.0, dtype=BF, device=DEV)
    ops.latent_attention_prefill(qkv, H * Dp, kv, padded(kr[C], rp, BF), torch.from_numpy(tiles).to(DEV), None, out, H, Dp, vp, scale, window)
    got = out.view(T, H, vp)[..., :vd].cpu()
    for i, ((s, n), f) in enumerate(zip(parts, first)):
        kk, vv = (t[i * 1024: i * 1024 + s + n].transpose(0, 1) for t in (keys, v))
        for r in sorted({0, 1, n // 2, n - 2, n - 1, min(63, n - 1), min(64, n - 1)} & set(range(n))):
            close(got[f + r], attend(q[f + r], kk, vv, scale, max(0, s + r + 1 - window), s + r + 1), BF)


# ---- gated delta rule -------------------------------------------------------------------------------------------------------------
class Delta:
    """Inputs of a recurrence of N rows per sequence for ``seqs`` sequences, as tensors of the layer and as the kernels take them."""

    def __init__(self, H, G, D, V, N, dtype, seqs=1, kind="plain", rank=16, taps=3, seed=0):
        self.H, self.G, self.D, self.V, self.dtype, self.rank, self.taps = H, G, D, V, dtype, rank, taps
        self.Dp, self.Vp, T = pad16(D), pad16(V), N * seqs
        r16 = lambda *s, i: rand(*s, seed=100 * seed + i).to(BF).float()
        self.q, self.k, self.v, self.beta, self.gl = r16(T, G, D, i=1), r16(T, G, D, i=2), r16(T, H, V, i=3), 2 * r16(T, H, i=4), r16(T, rank, i=5)
        self.al, self.wa, self.wg, self.ba = r16(T, rank, i=6), r16(H * D, rank, i=7) / 4, r16(H * V, rank, i=8) / 4, 2 * r16(H * D, i=9) - 3
        self.rate, self.norm = torch.rand(H, generator=torch.Generator().manual_seed(10)) * 2 + 0.1, 1 + 0.3 * rand(V, seed=11)
        if kind == "strong":                   # decays far below what a quotient of products could hold
            self.rate, self.ba = self.rate * 16, self.ba + 6
        if kind == "slow":                     # keys that hardly differ, a state that hardly forgets
            self.k, self.ba = (0.3 * self.k + r16(1, G, D, i=12)).to(BF).float(), self.ba - 6
        self.eps = 1e-5

    def want(self, rows=slice(None), q=None, k=None, v=None):
        """Outputs of one sequence (its rows), double."""
        q, k, v = (t if t is not None else s[rows] for t, s in ((q, self.q), (k, self.k), (v, self.v)))
        d, rep, H = lambda t: t.double(), self.H // self.G, self.H
        qq, kk = (oracle.unit(d(t)).repeat_interleave(rep, 1) for t in (q, k))
        z = (d(self.al[rows]) @ d(self.wa).T + d(self.ba)).view(-1, H, self.D)
        g = torch.exp(-d(self.rate)[None, :, None] * oracle.softplus(z))
        o = oracle.delta_rule(qq * self.D ** -0.5, kk, d(v), oracle.sigmoid(d(self.beta[rows])), g)
        return oracle.rms(o, self.eps) * d(self.norm) * oracle.sigmoid(d(self.gl[rows]) @ d(self.wg).T).view(-1, H, self.V)

    def wide(self, rows=slice(None)):
        """[rows, q | k | v | decay low | gate low | step sizes]"""
        t = self.dtype
        return torch.cat((pad_heads(self.q[rows], t), pad_heads(self.k[rows], t), pad_heads(self.v[rows], t), self.al[rows].to(t).to(DEV), self.gl[rows].to(t).to(DEV),
                          padded(self.beta[rows], pad16(self.H), t)), 1)

    def weights(self):
        heads = lambda w, n, d: padded(w.view(n, d, -1).transpose(1, 2), pad16(d), self.dtype).transpose(1, 2).reshape(n * pad16(d), -1).contiguous()
        return heads(self.wa, self.H, self.D), pad_heads(self.ba.view(1, self.H, self.D), self.dtype)[0].contiguous(), heads(self.wg, self.H, self.V)

    def split(self, wide):
        K, HV = self.G * self.Dp, self.H * self.Vp
        return wide.split((K, K, HV, self.rank, self.rank, pad16(self.H)), 1)

    def state(self, slots=4):
        return torch.full((slots, self.H, self.Dp, self.Vp), 7.0, device=DEV)       # what a previous owner left

    @property
    def common(self):
        return dict(kv_heads=self.G, dim=self.D, vdim=self.V, eps=self.eps)

    def scan(self, rows, segs, pos, state, form):
        """``form``: sequential, chunks (one kernel) or apart (operands of all chunks first)."""
        from libtbvcoll_b200 import ops
        q, k, v, al, gl, beta = self.split(self.wide(rows))
        T, n = q.shape[0], self.H
        z = padded(oracle.softplus((self.al[rows].double() @ self.wa.double().T + self.ba.double())).float().view(-1, n, self.D), self.Dp, F32).flatten(1)
        gate = pad_heads((self.gl[rows].double() @ self.wg.double().T).float().view(-1, n, self.V), self.dtype)
        out = torch.zeros(T, n * self.Vp, dtype=self.dtype, device=DEV)
        size = ops.delta_sets(T, segs.shape[0], state) if form == "apart" else 0
        sets = torch.full((size,), 255, dtype=torch.uint8, device=DEV) if size else None        # NaN wherever it is not written
        assert sets is not None or form != "apart" or self.Dp > 128
        ops.delta_scan(q, k, v, beta, z, gate, self.rate.to(DEV), padded(self.norm, self.Vp, F32), state, torch.empty(T, n * self.Vp, device=DEV), out, segs, pos,
                       groups=None if form in ("fp32", "sequential") else segs, sets=sets, **self.common)
        got = out.view(T, n, self.Vp)
        assert not got[..., self.V:].any()
        return got[..., : self.V].cpu()


SIZES = [(4, 2, 24, 36), (3, 3, 64, 64), (2, 1, 128, 128), (2, 2, 96, 200), (1, 1, 30, 16), (2, 2, 32, 130)]


@pytest.mark.parametrize("kind", ["plain", "strong", "slow"])
@pytest.mark.parametrize("H,G,D,V", SIZES + [(2, 1, 200, 48), (1, 1, 256, 20)])
@pytest.mark.parametrize("form", ["fp32", "sequential", "chunks", "apart"])
def test_delta_recurrence_in_portions(form, H, G, D, V, kind):
    """Whole, and in portions down to one row, the state handed over in a slot that holds something else at first."""
    dtype = F32 if form == "fp32" else BF
    N = 117
    d = Delta(H, G, D, V, N, dtype, kind=kind)
    want = d.want()
    tol = 3e-5 if dtype is F32 else None
    states = []
    for portions in ([N], [1, 2, 15, 16, 17, 33, 33], [40, 1, 76]):
        st, at, got = d.state(), 0, []
        for n in portions:
            segs, _, pos = ragged([n], [at], [2])
            got.append(d.scan(slice(at, at + n), segs, pos, st, form))
            at += n
        close(torch.cat(got), want, dtype, tol)
        assert float(st[[0, 1, 3]].min()) == 7.0
        states.append(st[2])
    for s in states[1:]:
        assert float((s - states[0]).norm() / states[0].norm()) < 2e-5


@pytest.mark.parametrize("H,seqs", [(2, 60), (40, 3)])
def test_delta_chunks_with_many_heads_and_sequences(H, seqs):
    """Enough CTAs that each takes all value columns of its head: head norm and gate inside."""
    N, D, V = 45, 64, 128
    d = Delta(H, H, D, V, N, BF, seqs=seqs, kind="slow")
    segs, _, pos = ragged([N] * seqs, [0] * seqs, list(range(1, seqs + 1)))
    got = d.scan(slice(None), segs, pos, d.state(seqs + 1), "chunks")
    for s in (0, 1, seqs - 1):
        rows = slice(s * N, s * N + N)
        close(got[rows], d.want(rows), BF)
    # one of them goes on with another portion, beside the others' first
    st = d.state(seqs + 1)
    cut = 20
    segs, _, pos = ragged([cut], [0], [1])
    a = d.scan(slice(0, cut), segs, pos, st, "chunks")
    segs, _, pos = ragged([N - cut] + [N] * (seqs - 1), [cut] + [0] * (seqs - 1), list(range(1, seqs + 1)))
    b = d.scan(slice(cut, N * seqs), segs, pos, st, "chunks")
    close(torch.cat((a, b)), got, BF)


def test_delta_chunks_of_a_long_sequence():
    """Hundreds of chunks: the state stays what the sequential form makes of it, rounding of thousands of decays aside."""
    d = Delta(2, 2, 128, 64, 3000, BF, kind="slow")
    segs, _, pos = ragged([3000], [0], [1])
    a, b, c = d.state(), d.state(), d.state()
    x, y, z = (d.scan(slice(None), segs, pos, st, f) for st, f in ((a, "chunks"), (b, "sequential"), (c, "apart")))
    assert float((a[1] - b[1]).norm() / b[1].norm()) < 5e-5 and torch.equal(a, c)
    close(x, y, BF)
    close(z, y, BF)


def test_delta_sets_of_ragged_segments():
    """Segments that begin and end anywhere in the chunks of the batch, as operands made apart: each has sets of its own."""
    lens, starts, slots = [5, 40, 1, 16, 130, 3], [0, 7, 100, 0, 0, 64], [3, 1, 6, 2, 5, 4]
    d = Delta(3, 1, 40, 70, sum(lens), BF, kind="slow")
    segs, _, pos = ragged(lens, starts, slots)
    a, b = d.state(7), d.state(7)
    x, y = d.scan(slice(None), segs, pos, a, "apart"), d.scan(slice(None), segs, pos, b, "sequential")
    assert float((a - b).norm() / b.norm()) < 1e-5
    close(x, y, BF)


@pytest.mark.parametrize("H,G,D,V", SIZES + [(2, 1, 200, 48), (1, 1, 16, 1000)])
@pytest.mark.parametrize("taps", [1, 4])
@pytest.mark.parametrize("dtype", [BF, F32])
def test_delta_step_with_convolution_and_products(dtype, taps, H, G, D, V):
    """Token by token, three sequences side by side that start at different steps: convolution, low-rank products, recurrence, norm and gate."""
    from libtbvcoll_b200 import ops
    N, seqs = 12, 3
    d = Delta(H, G, D, V, N, dtype, seqs=seqs, taps=taps)
    C = 2 * G * d.Dp + H * d.Vp
    cw = [rand(n, c, taps, seed=20 + i) for i, (n, c) in enumerate(((G, D), (G, D), (H, V)))]
    taps_w = torch.cat([padded(w.permute(2, 0, 1), pad16(w.shape[1]), F32).flatten(1) for w in cw], 1).contiguous()
    want = []
    for s in range(seqs):
        rows = slice(s * N, s * N + N)
        conv = [oracle.silu(oracle.causal_conv(t[rows].flatten(1), w.flatten(0, 1))).view(t[rows].shape) for t, w in zip((d.q, d.k, d.v), cw)]
        want.append(d.want(rows, *(c.to(BF).float() if dtype is BF else c for c in conv)))
    wide, (wa, ba, wg) = d.wide(), d.weights()
    st, past = d.state(seqs + 2), torch.full((seqs + 2, taps - 1, C), 9.0, device=DEV)
    got, slot, first = [[] for _ in range(seqs)], [4, 1, 2], [0, 3, 5]
    for step in range(N + 5):
        on = [s for s in range(seqs) if 0 <= step - first[s] < N]
        rows = torch.tensor([s * N + step - first[s] for s in on], device=DEV)
        segs = torch.tensor([[i, 1, slot[s], 0] for i, s in enumerate(on)], **I32)
        pos = torch.tensor([step - first[s] for s in on], **I32)
        x = wide[rows]
        q, k, v, al, gl, beta = d.split(x)
        conv = (taps_w, past) if G == H else None
        if conv is None:
            c = torch.empty(len(on), C, dtype=dtype, device=DEV)
            ops.short_conv(x, c, taps_w, past, segs, None, pos)
            q, k, v = c.split((G * d.Dp, G * d.Dp, H * d.Vp), 1)
        out = torch.empty(len(on), H * d.Vp, dtype=dtype, device=DEV)
        ops.delta_step(q, k, v, beta, al, gl, wa, ba, wg, d.rate.to(DEV), padded(d.norm, d.Vp, F32), st, out, segs, pos, conv=conv, **d.common)
        for i, s in enumerate(on):
            got[s].append(out[i].view(H, d.Vp)[:, :V])
    for s in range(seqs):
        close(torch.stack(got[s]), want[s], dtype, None if dtype is BF else 5e-5)
    assert float(st[0].min()) == float(st[3].min()) == 7.0
