"""Every mechanism of Tinapel on its own: the kernel against a plain statement of the same thing, at sizes that are not multiples of
anything, on inputs made so that a wrong key, edge, decay, state or expert shows."""
import math

import pytest
import torch

import tinapel_oracle as oracle

pytestmark = pytest.mark.gpu
DEV = "cuda:0"
BF, F32 = torch.bfloat16, torch.float32


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


# ---- residual stream ------------------------------------------------------------------------------------------------------
@pytest.mark.parametrize("width", [20, 100, 333, 2048, 5000])
@pytest.mark.parametrize("dtype", [BF, F32])
def test_embedding_with_far_positions(width, dtype):
    from libtbvcoll_b200 import ops
    V, Wp, pos = 11, pad16(width), [0, 1, 7, 63, 1000, 65537, 1000003]
    emb = rand(V, width, seed=1).to(BF).float()
    ids = torch.tensor([3, 0, 10, 3, 7, 1, 2])
    x, x0, h1, h2 = (torch.full((7, Wp), 5.0, dtype=d, device=DEV) for d in (F32, F32, dtype, dtype))
    g1, g2, step = rand(width, seed=2), rand(width, seed=3), rand(width, seed=4)
    ops.residual(x, padded(g1, Wp, F32), h1, width, 1e-3, g2=padded(g2, Wp, F32), h2=h2, embed=(ids.to(DEV), padded(emb, Wp, dtype), 0.3, ops.position_turns(width, DEV)),
                 positions=torch.tensor(pos, dtype=torch.int32, device=DEV), x0=x0, step=padded(step, Wp, F32))
    want = torch.empty(7, width, dtype=torch.float64)
    for c in range(width):
        for r, p in enumerate(pos):
            a = p * 10000.0 ** (-2.0 * (c // 2) / width)
            want[r, c] = math.sin(a) if c % 2 == 0 else math.cos(a)
    want = want + emb[ids].double() * 0.3
    close(x0[:, :width], want, F32, 1e-6)
    close(x[:, :width], want + step.double(), F32, 1e-6)
    close(h1[:, :width], oracle.rms(want + step.double(), 1e-3) * g1, dtype)
    close(h2[:, :width], oracle.rms(want + step.double(), 1e-3) * g2, dtype)
    assert not x[:, width:].any() and not h1[:, width:].any() and not x0[:, width:].any()


@pytest.mark.parametrize("width,top", [(20, 1), (100, 3), (4096, 2), (9000, 7)])
@pytest.mark.parametrize("dtype", [BF, F32])
def test_branches_experts_loop_terms_and_both_norms(width, top, dtype):
    from libtbvcoll_b200 import ops
    T, Wp, eps = 6, pad16(width), 1e-4
    x, y1, y2, x0 = (rand(T, width, seed=s) for s in range(4))
    ro, place = rand(T * top, width, seed=5).to(dtype).float(), torch.randperm(T * top, generator=torch.Generator().manual_seed(6)).view(T, top)
    wt, step, g1, g2 = rand(T, top, seed=7), rand(width, seed=8), rand(width, seed=9), rand(width, seed=10)
    routed = (padded(ro, Wp, dtype), place.to(torch.int32).to(DEV), wt.to(DEV))
    full = lambda t: padded(t, Wp, F32)
    h1, h2, out = torch.empty(T, Wp, dtype=dtype, device=DEV), torch.empty(T, Wp, dtype=dtype, device=DEV), torch.empty(3, Wp, dtype=dtype, device=DEV)
    branches = y1 + y2 + (wt[..., None] * ro[place]).sum(1)
    for terms, want in ((dict(y1=full(y1)), x + y1), (dict(y1=full(y1), y2=full(y2), routed=routed), x + branches),
                        (dict(y2=full(y2), x0=full(x0), step=full(step)), x + y2 + x0 + step), (dict(routed=routed, step=full(step)), x + branches - y1 - y2 + step), ({}, x)):
        xd = full(x)
        ops.residual(xd, full(g1), out, width, eps, rows=torch.tensor([5, 0, 5], device=DEV), last=True, **terms)
        assert torch.equal(xd, full(x))
        close(out[:, :width], oracle.rms(want, eps)[[5, 0, 5]] * g1, dtype)
        ops.residual(xd, full(g1), h1, width, eps, g2=full(g2), h2=h2, **terms)
        close(xd[:, :width], want, F32)
        close(h1[:, :width], oracle.rms(want, eps) * g1, dtype)
        close(h2[:, :width], oracle.rms(want, eps) * g2, dtype)
        assert not xd[:, width:].any() and not h1[:, width:].any()


@pytest.mark.parametrize("dtype", [BF, F32])
def test_mixes_with_the_previous_token(dtype):
    """Portions through k_token_shift and single tokens through the residual kernel give the mixes of the whole sequence, whatever the slots hold."""
    from libtbvcoll_b200 import ops
    W, Wp, n, lens = 52, 64, 5, (9, 1, 14)
    g, mu = 1.0 + rand(W, seed=1), torch.rand(n, W, generator=torch.Generator().manual_seed(2))
    xs = [rand(k, W, seed=10 + k) for k in lens]
    hs = [oracle.rms(x, 1e-5) * g for x in xs]
    want = [torch.stack([oracle.token_shift(h, m) for m in mu], 1) for h in hs]
    shift, slots, cut = torch.full((8, Wp), 3.0, device=DEV), (4, 1, 6), (5, 1, 13)
    gd, mud = padded(g, Wp, F32), padded(mu, Wp, F32)

    def check(mixes, rows):
        close(mixes.view(-1, n, Wp)[:, :, :W], torch.cat(rows), dtype)
    # first portions, then (behind a stand-in for the recurrence that keeps the last row) the rest token by token
    part = torch.cat([h[:c] for h, c in zip(hs, cut)])
    segs, at = [], 0
    for c, s in zip(cut, slots):
        segs.append([at, c, s, 0])
        at += c
    seg_of_row = torch.cat([torch.full((c,), i) for i, c in enumerate(cut)]).to(torch.int32).to(DEV)
    pos = torch.cat([torch.arange(c) for c in cut]).to(torch.int32).to(DEV)
    mixes = torch.empty(at, n * Wp, dtype=dtype, device=DEV)
    ops.token_shift(padded(part, Wp, F32), mud, shift, mixes, torch.tensor(segs, dtype=torch.int32, device=DEV), seg_of_row, pos)
    check(mixes, [w[:c] for w, c in zip(want, cut)])
    for h, c, s in zip(hs, cut, slots):
        shift[s, :W] = h[c - 1].to(DEV)
        shift[s, W:] = 0
    for i in (0, 2):                                              # a portion that starts with a carried row
        rest = hs[i][cut[i]:]
        k = len(rest)
        mixes = torch.empty(k, n * Wp, dtype=dtype, device=DEV)
        ops.token_shift(padded(rest, Wp, F32), mud, shift, mixes, torch.tensor([[0, k, slots[i], 0]], dtype=torch.int32, device=DEV),
                        torch.zeros(k, dtype=torch.int32, device=DEV), torch.arange(cut[i], cut[i] + k, dtype=torch.int32, device=DEV))
        check(mixes, [want[i][cut[i]:]])
    shift.fill_(7.0)
    for t in range(9):                                            # one row per sequence: kept by the kernel itself
        mixes = torch.empty(2, n * Wp, dtype=dtype, device=DEV)
        x = padded(torch.stack([xs[0][t], xs[2][t]]), Wp, F32)
        ops.residual(x, gd, torch.empty(2, Wp, device=DEV), W, 1e-5, positions=torch.tensor([t, t], dtype=torch.int32, device=DEV),
                     mix=(mud, mixes, shift, torch.tensor([[0, 1, 2, 0], [1, 1, 5, 0]], dtype=torch.int32, device=DEV)))
        check(mixes, [want[0][t: t + 1], want[2][t: t + 1]])
    assert bool((shift[[0, 1, 3, 4, 6, 7]] == 7.0).all())


# ---- recurrences ------------------------------------------------------------------------------------------------------------
class Recurrence:
    """One sequence of a recurrence with head norm and gate; ``z`` spreads decays from none to total."""

    def __init__(self, kind, T, H, D, V, rank=11, seed=0, dtype=F32):
        g = torch.Generator().manual_seed(seed)
        n = lambda *s: torch.randn(*s, generator=g).to(dtype).float()
        self.kind, self.T, self.H, self.D, self.V, self.tau, self.eps = kind, T, H, D, V, 3.0, 1e-5
        self.q, self.k, self.v, self.g = n(T, H, D), n(T, H, D) / D ** 0.5, n(T, H, V), n(T, H * V)
        self.low, self.w2, self.b2 = n(T, rank), n(H * D, rank) / rank ** 0.5, (4.0 * n(H * D)).to(dtype).float()
        self.u, self.norm = n(H, D), 1 + 0.2 * n(H * V)
        act = torch.tanh(self.low) if kind == "wkv" else self.low
        self.z = act @ self.w2.T + self.b2
        z = self.z.view(T, H, D).double()
        q, k, v = self.q.double(), self.k.double(), self.v.double()
        if kind == "wkv":
            o = oracle.wkv(q, k, v, torch.exp(-torch.exp(z)), self.u.double())
        else:
            o = oracle.gated_linear_attention(q / D ** 0.5, k, v, oracle.sigmoid(z) ** (1 / self.tau))
        self.o = o
        self.want = (oracle.rms(o, self.eps).flatten(1) * self.norm * oracle.silu(self.g.double())).view(T, H, V)

    def wide(self, rows, dtype, width_low):
        parts = [pad_heads(t[rows], dtype) for t in (self.q, self.k, self.v, self.g.view(self.T, self.H, self.V))]
        return torch.cat(parts + [padded(self.low[rows], width_low, dtype)], 1)

    def args(self):
        u = None if self.kind == "gla" else pad_heads(self.u[None], F32)[0]
        a = dict(vdim=self.V, eps=self.eps, u=u)
        return a if self.kind == "wkv" else {**a, "qscale": self.D ** -0.5, "tau": self.tau}


def run_recurrence(seqs, portions, state, slots, dtype, group_rows=None, step_form=False, low_form=False):
    """The next ``portions[i]`` = (start, end) of every sequence as one batch; outputs [rows, H, V] per sequence."""
    from libtbvcoll_b200 import ops
    from libtbvcoll_b200.engine.batch import scan_groups
    s0 = seqs[0]
    H, D, V, R = s0.H, s0.D, s0.V, pad16(s0.low.shape[1])
    K, Vw = H * pad16(D), H * pad16(V)
    wide = torch.cat([s.wide(slice(a, b), dtype, R) for s, (a, b) in zip(seqs, portions)])
    q, k, v, g, low = wide.split((K, K, Vw, Vw, R), 1)
    segs, at = [], 0
    for (a, b), slot in zip(portions, slots):
        segs.append([at, b - a, slot, 0])
        at += b - a
    pos = torch.cat([torch.arange(a, b) for a, b in portions]).to(torch.int32).to(DEV)
    sd = torch.tensor(segs, dtype=torch.int32, device=DEV)
    norm, out = pad_heads(s0.norm.view(1, H, V), F32)[0], torch.empty(at, Vw, dtype=dtype, device=DEV)
    if step_form:
        w2 = padded(padded(s0.w2.view(H, D, -1).transpose(1, 2), pad16(D), dtype).transpose(1, 2), R, dtype).reshape(K, R).contiguous()
        ops.decay_step(q, k, v, g, low, w2, pad_heads(s0.b2.view(1, H, D), dtype)[0], norm, state, out, sd, pos, **s0.args())
    else:
        z = torch.cat([pad_heads(s.z[a:b].view(-1, H, D), F32) for s, (a, b) in zip(seqs, portions)])
        groups = scratch = None
        if group_rows:
            gr = scan_groups(sd.cpu().numpy(), group_rows)
            groups = torch.from_numpy(gr).to(DEV)
            if len(gr) > len(segs):
                scratch = (torch.full((len(gr) * K * pad16(V),), 9.0, device=DEV), torch.full((len(gr) * K,), 9.0, device=DEV))
        lo = None
        if low_form:                                         # the decay product inside
            act = torch.cat([padded(torch.tanh(s.low[a:b]) if s.kind == "wkv" else s.low[a:b], R, dtype) for s, (a, b) in zip(seqs, portions)])
            z, lo = None, (act, padded(padded(s0.w2.view(H, D, -1).transpose(1, 2), pad16(D), dtype).transpose(1, 2), R, dtype).reshape(K, R).contiguous(),
                           pad_heads(s0.b2.view(1, H, D), dtype)[0])
        ops.decay_scan(q, k, v, g, z, norm, state, torch.empty(at * Vw, device=DEV), out, sd, pos, groups=groups, scratch=scratch, low=lo, **s0.args())
    out = out.view(at, H, pad16(V))
    assert not out[..., V:].any()
    return [out[f: f + n, :, :V] for f, n, _, _ in segs]


SIZES = [(3, 24, 20), (2, 32, 64), (5, 36, 48), (2, 96, 144), (1, 128, 128), (2, 200, 16), (1, 160, 272)]


@pytest.mark.parametrize("kind", ["gla", "wkv"])
@pytest.mark.parametrize("size", SIZES)
@pytest.mark.parametrize("form", ["sequential f32", "sequential", "chunks", "groups", "chunks, low", "groups, low"])
def test_recurrence_over_portions(kind, size, form):
    """Whole sequences and portions down to one token, of unequal sequences in one batch, slots that held something else: the same outputs and the
    same final state as one plain pass."""
    H, D, V = size if kind == "gla" else (size[0], min(size[1], 160), min(size[1], 160))
    dtype = F32 if form == "sequential f32" else BF
    rows, low = {"chunks": 512, "groups": 32}.get(form.split(",")[0]), form.endswith("low")
    seqs = [Recurrence(kind, n, H, D, V, seed=n + 1, dtype=dtype) for n in (97, 33, 150)]
    for s in seqs:                                          # one set of weights
        s.norm, s.u, s.w2, s.b2 = seqs[0].norm, seqs[0].u, seqs[0].w2, seqs[0].b2
        z = ((torch.tanh(s.low) if kind == "wkv" else s.low) @ s.w2.T + s.b2)
        zz = z.view(s.T, H, D).double()
        s.z = z
        s.o = oracle.wkv(s.q.double(), s.k.double(), s.v.double(), torch.exp(-torch.exp(zz)), s.u.double()) if kind == "wkv" else \
            oracle.gated_linear_attention(s.q.double() / D ** 0.5, s.k.double(), s.v.double(), oracle.sigmoid(zz) ** (1 / s.tau))
        s.want = (oracle.rms(s.o, s.eps).flatten(1) * s.norm * oracle.silu(s.g.double())).view(s.T, H, V)
    state = torch.full((6, H, pad16(D), pad16(V)), 5.0, device=DEV)
    outs = run_recurrence(seqs, [(0, s.T) for s in seqs], state, (2, 5, 1), dtype, rows, low_form=low)
    for s, o in zip(seqs, outs):
        close(o, s.want, dtype)
    whole = state[[2, 5, 1]].clone()
    assert bool((state[[0, 3, 4]] == 5.0).all())
    # portions: cut points that fall inside, at and around chunks of 16
    cuts = [(0, 2, 3, 19, 35, 67, 68, 97), (0, 1, 15, 16, 17, 30, 32, 33), (0, 16, 32, 33, 64, 100, 149, 150)]
    at = [[] for _ in seqs]
    for j in range(7):
        for i, o in enumerate(run_recurrence(seqs, [(c[j], c[j + 1]) for c in cuts], state, (3, 2, 4), dtype, rows, low_form=low)):
            at[i].append(o)
    for s, o in zip(seqs, at):
        close(torch.cat(o), s.want, dtype)
    close(state[[3, 2, 4]], whole, dtype, 2e-5 if dtype is F32 or rows is None else 4e-5)      # carried in 32-bit in every form


@pytest.mark.parametrize("kind", ["gla", "wkv"])
@pytest.mark.parametrize("dtype", [BF, F32])
def test_one_token_form_and_scan_hand_the_state_to_each_other(kind, dtype):
    for H, D, V in SIZES[:6]:
        V = V if kind == "gla" else D
        seqs = [Recurrence(kind, n, H, D, V, seed=n, dtype=dtype) for n in (40, 41)]
        s = seqs[0]
        state = torch.full((4, H, pad16(D), pad16(V)), -3.0, device=DEV)
        got = []
        for a in range(6):                                   # from the first token
            got += run_recurrence([s], [(a, a + 1)], state, (3,), dtype, step_form=True)
        got += run_recurrence([s], [(6, 25)], state, (3,), dtype, 64 if dtype is BF else None)
        for a in range(25, 40):
            got += run_recurrence([s], [(a, a + 1)], state, (3,), dtype, step_form=True)
        close(torch.cat(got), s.want, dtype)
        assert bool((state[:3] == -3.0).all())


@pytest.mark.parametrize("kind", ["gla", "wkv"])
def test_chunks_with_extreme_decays(kind):
    """Channels that forget everything within a token beside channels that forget nothing, changing from token to token: products of decays
    underflow on the way, and a quotient of them would not be a number."""
    s = Recurrence(kind, 80, 2, 64, 64, seed=3, dtype=BF)
    z = 14.0 * rand(80, 2, 64, seed=4)                       # wkv: decays 1 - 1e-9 .. exp(-1e9); gla: sigmoid(-40) .. 1
    s.z = z.reshape(80, -1)
    if kind == "wkv":
        s.o = oracle.wkv(s.q.double(), s.k.double(), s.v.double(), torch.exp(-torch.exp(z.double())), s.u.double())
    else:
        s.tau = 0.5
        s.o = oracle.gated_linear_attention(s.q.double() / 8, s.k.double(), s.v.double(), oracle.sigmoid(z.double()) ** 2)
    s.want = (oracle.rms(s.o, s.eps).flatten(1) * s.norm * oracle.silu(s.g.double())).view(80, 2, 64)
    for rows in (None, 128, 32):
        state = torch.zeros(2, 2, 64, 64, device=DEV)
        close(run_recurrence([s], [(0, 80)], state, (1,), BF, rows)[0], s.want, BF)
        assert bool(torch.isfinite(state).all())


def test_a_far_key_in_the_state():
    """One key of the first chunk, never decayed, is what the last query asks for: its value must come out, not the sum of the hundreds between."""
    s = Recurrence("gla", 600, 1, 64, 64, seed=8, dtype=BF)
    s.q[:], s.z, s.tau = s.q * 0.01, torch.full((600, 64), 60.0), 1.0
    s.k[:, :, 0] = 0.0
    s.k[5], s.q[599] = 0.0, 0.0
    s.k[5, :, 0], s.q[599, :, 0] = 1.0, 8.0
    s.norm[:], s.g[:] = 1.0, 20.0
    for rows in (None, 1024, 48):
        state = torch.zeros(2, 1, 64, 64, device=DEV)
        o = run_recurrence([s], [(0, 600)], state, (1,), BF, rows)[0][599, 0]
        close(o, 20.0 * oracle.rms(s.v[5, 0], 1e-5), BF)


@pytest.mark.parametrize("form", ["sequential", "groups"])
def test_the_recurrence_keeps_the_last_rows_input(form):
    from libtbvcoll_b200 import ops
    from libtbvcoll_b200.engine.batch import scan_groups
    H, D, T = 2, 32, 90
    segs = torch.tensor([[0, 70, 2, 0], [70, 20, 1, 0]], dtype=torch.int32, device=DEV)
    wide, z, st = rand(T, 4 * H * D, seed=1).to(BF).to(DEV), rand(T, H * D, seed=2).to(DEV), torch.zeros(3, H, D, D, device=DEV)
    q, k, v, g = wide.split(H * D, 1)
    h, shift, pos = rand(T, 48, seed=3).to(DEV), torch.full((3, 48), 4.0, device=DEV), torch.arange(T, dtype=torch.int32, device=DEV)
    kw = {}
    if form == "groups":
        gr = scan_groups(segs.cpu().numpy(), 16)
        kw = dict(groups=torch.from_numpy(gr).to(DEV), scratch=(torch.empty(len(gr) * H * D * D, device=DEV), torch.empty(len(gr) * H * D, device=DEV)))
    ops.decay_scan(q, k, v, g, z, torch.ones(H * D, device=DEV), st, torch.empty(T * H * D, device=DEV), torch.empty(T, H * D, dtype=BF, device=DEV), segs, pos,
                   vdim=D, eps=1e-5, u=torch.ones(H * D, device=DEV), shift=(h, shift), **kw)
    assert torch.equal(shift[2], h[69]) and torch.equal(shift[1], h[89]) and bool((shift[0] == 4.0).all())


# ---- attention ----------------------------------------------------------------------------------------------------------------
class Attn:
    def __init__(self, H, G, D, T, cap, seed=0, dtype=F32, coef=0.6, every=7, block=16):
        from libtbvcoll_b200 import ops
        self.H, self.G, self.D, self.T, self.cap, self.dtype, self.block, self.ops, self.eps = H, G, D, T, cap, dtype, block, ops, 1e-5
        self.coef, self.every, self.scale = coef, every, 0.8 * D ** -0.5
        self.q, self.k = rand(T, H, D, seed=seed).to(dtype).float(), rand(T, G, D, seed=seed + 1).to(dtype).float()
        self.qn, self.kn = 1.5 + 0.3 * rand(D, seed=seed + 2), 1.5 + 0.3 * rand(D, seed=seed + 3)

    def want(self):
        """The oracle's mixer with identity projections."""
        H, G, D = self.H, self.G, self.D
        n = H * D + G * D
        h = torch.cat((self.q.flatten(1), self.k.flatten(1)), 1)
        eye = torch.eye(n)
        w = {"q": eye[: H * D], "k": eye[H * D:], "q.norm": self.qn, "k.norm": self.kn, "o": torch.eye(H * D)}
        m = {"heads": H, "kv_heads": G, "dim": D, "scale": self.scale, "softcap": self.cap, "q_temp": {"coef": self.coef, "every": self.every}}
        return oracle.attention_mixer(h, w, "", m, self.eps).view(self.T, H, D)

    def write(self, start, end, cache, table, n_rows_form):
        """Prepares rows start..end-1 of the sequence; (queries of the rows form, query buffer, positions)."""
        Dp, T = pad16(self.D), end - start
        qk = torch.cat((pad_heads(self.q[start:end], self.dtype), pad_heads(self.k[start:end], self.dtype)), 1)
        pos = torch.arange(start, end, dtype=torch.int32, device=DEV)
        slots = table[(pos // self.block).long()].long() * self.block + pos % self.block
        qa = torch.full((n_rows_form, self.H, Dp + 8), 9.0, dtype=self.dtype, device=DEV)
        self.ops.shared_attention_prep(qk, qa, cache, padded(self.qn * self.kn * self.scale, Dp, F32), pos, slots, n_rows_form, self.H, self.G, self.D, self.block,
                                       self.eps, self.coef, self.every)
        return qa, qk, pos

    def new_cache(self, blocks):
        return torch.full((blocks * self.G * self.block, pad16(self.D) + 8), float("nan"), dtype=self.dtype, device=DEV)     # a stale row must not matter

    def rows(self, qa, pos, cache, table, splits=1):
        n, Dp = qa.shape[0], pad16(self.D)
        out = torch.empty(n, self.H, Dp, dtype=self.dtype, device=DEV)
        self.ops.shared_attention_rows(qa, cache, table[None], torch.zeros(n, dtype=torch.int32, device=DEV), pos + 1, out, self.G, self.block, self.cap or 0.0, splits)
        return out[..., : self.D]

    def prefill(self, qk, start, cache, table):
        n, Dp = qk.shape[0], pad16(self.D)
        out = torch.empty(n, self.H * Dp, dtype=self.dtype, device=DEV)
        tiles = torch.tensor([[a, min(64, n - a), 0, start + a + 1] for a in range(0, n, 64)], dtype=torch.int32, device=DEV)
        self.ops.shared_attention_prefill(qk, cache, table[None], torch.zeros(n, dtype=torch.int32, device=DEV), tiles, out, self.H, self.G, self.block, self.cap or 0.0)
        return out.view(n, self.H, Dp)[..., : self.D]


def scattered(blocks, seed=3):
    return (torch.randperm(blocks, generator=torch.Generator().manual_seed(seed)) + 1).to(torch.int32).to(DEV)


@pytest.mark.parametrize("H,G,D,cap", [(6, 2, 40, 4.0), (4, 4, 16, None), (8, 1, 64, 10.0), (20, 1, 128, 3.0), (24, 2, 100, 15.0), (2, 1, 144, 5.0), (3, 3, 256, None),
                                       (5, 1, 320, 6.0)])
@pytest.mark.parametrize("dtype", [BF, F32])
def test_attention_whole_portions_and_single_rows(H, G, D, cap, dtype):
    a = Attn(H, G, D, 213, cap, seed=H, dtype=dtype)
    want, table = a.want(), scattered(14)
    cache = a.new_cache(15)
    got, at = [], 0
    for n, form in ((70, "prefill"), (1, "rows"), (2, "rows"), (33, "prefill"), (1, "rows"), (31, "rows"), (64, "prefill"), (11, "rows")):
        many = form == "prefill" and dtype is BF and pad16(D) <= 256
        qa, qk, pos = a.write(at, at + n, cache, table, 0 if many else n)
        got.append(a.prefill(qk, at, cache, table) if many else a.rows(qa, pos, cache, table, splits=1 + at % 4))
        at += n
    close(torch.cat(got), want, dtype)
    assert at == 213 and not a.ops.gemm_error()


@pytest.mark.parametrize("dtype", [BF, F32])
@pytest.mark.parametrize("D", [64, 144])
def test_single_keys_stand_out(dtype, D):
    """A query and a key scaled so that one score stands out of all others: at block and unit edges, first, last and far keys, for each number of splits."""
    T = 700
    a = Attn(4, 2, D, T, 40.0, seed=5, dtype=dtype, coef=0.0)
    a.q, a.k = a.q * 0.05, a.k * 0.05
    a.qn[:], a.kn[:], a.scale = 1.0, 1.0, 4.0 * D ** -0.5                    # a parallel pair scores 4 sqrt(D), others a few
    keys = [0, 1, 15, 16, 17, 31, 32, 63, 64, 127, 128, 511, 512, 640, 697, 698, 699]
    for i, j in enumerate(keys):                              # the last rows ask for one key each
        a.q[T - len(keys) + i] = 2.0 * a.k[min(j, T - len(keys) + i)].repeat_interleave(2, 0)
    a.q, a.k = a.q.to(dtype).float(), a.k.to(dtype).float()
    want, table, cache = a.want(), scattered(44), a.new_cache(45)
    for i, j in enumerate(keys):
        r = T - len(keys) + i
        assert float((want[r, 0] - a.k[min(j, r), 0]).norm() / a.k[min(j, r), 0].norm()) < 0.2
    _, qk, _ = a.write(0, T, cache, table, 0 if dtype is BF else T)
    if dtype is BF:
        close(a.prefill(qk, 0, cache, table), want, dtype, 2.5e-2)
    n = len(keys)
    qa, _, pos = a.write(T - n, T, cache, table, n)
    for splits in (1, 2, 4, 8):
        close(a.rows(qa, pos, cache, table, splits), want[T - n:], dtype, 2.5e-2 if dtype is BF else None)


@pytest.mark.parametrize("block", [8, 16, 32, 64])
def test_block_sizes(block):
    a = Attn(6, 2, 64, 150, 8.0, seed=2, dtype=BF, block=block)
    table = scattered(-(-150 // block))
    cache = a.new_cache(len(table) + 1)
    _, qk, _ = a.write(0, 150, cache, table, 0)
    close(a.prefill(qk, 0, cache, table), a.want(), BF)
    qa, _, pos = a.write(100, 150, cache, table, 50)
    close(a.rows(qa, pos, cache, table, 2), a.want()[100:], BF)


def test_query_temperature_changes_where_it_should():
    from libtbvcoll_b200 import ops
    pos = torch.tensor([0, 5, 6, 7, 12, 13, 20, 8190, 8191, 8192, 999999], dtype=torch.int32, device=DEV)
    for coef, every in ((0.7, 7), (1.3, 8192), (0.1, 2.5), (0.0, 1)):
        n = len(pos)
        qk = torch.ones(n, 32, device=DEV)
        qa, cache = torch.empty(n, 1, 24, device=DEV), torch.empty(32, 24, device=DEV)
        ops.shared_attention_prep(qk, qa, cache, torch.ones(16, device=DEV), pos, torch.arange(n, device=DEV), n, 1, 1, 16, 16, 0.0, coef, every)
        want = torch.tensor([1 + coef * math.log(math.floor((p + 1) / every) + 1) for p in pos.tolist()])
        close(qa[:, 0, :16], want[:, None].expand(n, 16), F32)


# ---- mixture of experts -----------------------------------------------------------------------------------------------------------
@pytest.mark.parametrize("E,top,T", [(1, 1, 3), (5, 3, 1), (8, 2, 32), (8, 2, 33), (40, 6, 31), (40, 6, 500), (300, 12, 7), (512, 20, 70)])
@pytest.mark.parametrize("dtype", [BF, F32])
def test_choice_and_dispatch(E, top, T, dtype):
    from libtbvcoll_b200 import ops
    z = 3 * rand(T, E, seed=E + T)
    if T > 2:
        z[0] = 0.5                                           # all equal: the lowest indices
        z[1, -1] = 200.0                                     # one that takes all
    logits, h = padded(z, pad16(E), F32), rand(T, 48, seed=1).to(dtype).to(DEV)
    logits[:, E:] = 1e9                                      # padding is not an expert
    i32 = lambda *s: torch.full(s, -7, dtype=torch.int32, device=DEV)
    xp, place, off, weight = torch.empty(T * top, 48, dtype=dtype, device=DEV), i32(T, top), i32(E + 1), torch.empty(T, top, device=DEV)
    ops.moe_route(logits, h, xp, place, weight, off, i32(E), i32(2 * T * top), E, 1.7)
    want = oracle.route(z, top, 1.7)
    place, off, weight = place.cpu().long(), off.cpu().long(), weight.cpu()
    assert sorted(place.flatten().tolist()) == list(range(T * top)) and off[0] == 0 and off[-1] == T * top
    expert = torch.searchsorted(off, place, right=True) - 1
    got = torch.zeros(T, E).scatter_(1, expert, weight)
    close(got, want, F32)
    assert torch.equal((got > 0) | (want == 0), torch.ones(T, E, dtype=torch.bool))
    assert torch.equal(off[1:] - off[:-1], torch.bincount(expert.flatten(), minlength=E))
    assert torch.equal(xp[place.to(DEV)], h[:, None].expand(T, top, 48))


@pytest.mark.parametrize("dtype", [BF, F32])
@pytest.mark.parametrize("counts", [[1], [0, 3, 0, 1, 16], [17, 0, 1, 33, 64, 5], [200, 0, 129, 128, 1], [700, 300, 0, 515], [0, 0, 1500]])
@pytest.mark.parametrize("M,K", [(48, 80), (272, 144), (528, 336)])
def test_row_grouped_products(counts, M, K, dtype):
    from libtbvcoll_b200 import ops
    G, R = len(counts), sum(counts)
    off = torch.tensor([0] + counts).cumsum(0).to(torch.int32).to(DEV)
    x, w = rand(R, K, seed=1).to(dtype).to(DEV), (rand(G * M, K, seed=2) / K ** 0.5).to(dtype).to(DEV)
    ref = torch.cat([x[off[g]: off[g + 1]].double() @ w[g * M: (g + 1) * M].double().T for g in range(G)])
    out = torch.full((R, M), 9.0, dtype=dtype, device=DEV)
    close(ops.linear_rows(x, w, out, off, G, max(counts)), ref, dtype)
    act = torch.full((R, M // 2), 9.0, dtype=dtype, device=DEV)
    close(ops.linear_rows(x, w, act, off, G, max(counts), glu=ops.SILU_GLU), oracle.silu(ref[:, 0::2]) * ref[:, 1::2], dtype)
    assert not ops.gemm_error()


@pytest.mark.parametrize("dtype", [BF, F32])
@pytest.mark.parametrize("N,G,M,K,last", [(3, 4, 48, 32, 16), (40, 2, 144, 80, 112), (1, 4, 272, 208, 64), (130, 3, 128, 64, 16)])
def test_grouped_linear_with_a_last_group(N, G, M, K, last, dtype):
    from libtbvcoll_b200 import ops
    x, w = rand(N, (G + 1) * K, seed=1).to(dtype).to(DEV), (rand(G * M + last, K, seed=2) / K ** 0.5).to(dtype).to(DEV)
    out = torch.full((N, G * M + last + 16), 9.0, dtype=dtype, device=DEV)
    ops.linear(x, w, out, groups=G, x_group=K, y_group=M, last=last)
    for g in range(G + 1):
        m = last if g == G else M
        close(out[:, g * M: g * M + m], x[:, g * K: (g + 1) * K].double() @ w[g * M: g * M + m].double().T, dtype)
    assert bool((out[:, G * M + last:] == 9.0).all())
