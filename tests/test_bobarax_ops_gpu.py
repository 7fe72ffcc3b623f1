"""Every mechanism of Bobarax on its own: the kernel against a plain statement of the same thing, at sizes that are not multiples of
anything, on inputs made so that a wrong key, edge, decay, state or expert shows."""
import math

import pytest
import torch

import bobarax_oracle as oracle

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


def perm(n, seed=6):
    return torch.randperm(n, generator=torch.Generator().manual_seed(seed))


# ---- residual stream ------------------------------------------------------------------------------------------------------
@pytest.mark.parametrize("width,top", [(20, 1), (100, 3), (2048, 2), (4096, 2), (9000, 5)])
@pytest.mark.parametrize("dtype", [BF, F32])
def test_branch_norms_joint_norm_and_experts_rows(width, top, dtype):
    """x + norm(branch), next norm: the branch plain, divided by a joint root mean square, or a mixture's weighted rows; the result in place, on the
    rows of the next mixture, or picked."""
    from libtbvcoll_b200 import ops
    T, Wp, eps, n = 6, pad16(width), 1e-4, 7
    x, y, gb, g = rand(T, width, seed=1), 30.0 * rand(T, width, seed=2), rand(width, seed=3), rand(width, seed=4)
    sq = 1e3 * rand(T, n, seed=5).abs()
    ro, source, to = rand(T * top, width, seed=6).to(dtype).float(), perm(T * top).view(T, top), perm(T * top, 8).view(T, top)
    full = lambda t: padded(t, Wp, F32)
    place = lambda t: t.to(torch.int32).to(DEV)
    wt = rand(T, top, seed=9)
    joint = y / torch.sqrt(sq.sum(1, keepdim=True) / 50 + eps)
    post = dict(post=full(gb))
    for terms, branch in ((dict(y1=full(y)), y), (dict(y1=full(y), sums=(sq.to(DEV), 50)), joint),
                          (dict(routed=(padded(ro, Wp, dtype), place(source), 1.0 / top)), ro[source].sum(1) / top),
                          (dict(routed=(padded(ro, Wp, dtype), place(source), wt.to(DEV))), (wt[..., None] * ro[source]).sum(1))):
        want = x + oracle.rms(branch, eps) * gb
        xd, h, out = full(x), torch.empty(T, Wp, dtype=dtype, device=DEV), torch.empty(3, Wp, dtype=dtype, device=DEV)
        ops.residual(xd, full(g), out, width, eps, rows=torch.tensor([5, 0, 5], device=DEV), last=True, **terms, **post)
        assert torch.equal(xd, full(x))
        close(out[:, :width], oracle.rms(want, eps)[[5, 0, 5]] * g, dtype)
        ops.residual(xd, full(g), h, width, eps, **terms, **post)
        close(xd[:, :width], want, F32)
        close(h[:, :width], oracle.rms(want, eps) * g, dtype)
        assert not xd[:, width:].any() and not h[:, width:].any()
        xd, rows = full(x), torch.full((T * top, Wp), 7.0, dtype=dtype, device=DEV)
        ops.residual(xd, full(g), rows, width, eps, place=place(to), **terms, **post)
        assert torch.equal(rows[to.reshape(-1).to(DEV)], h.repeat_interleave(top, 0))


@pytest.mark.parametrize("dtype", [BF, F32])
def test_embedding_without_positions(dtype):
    from libtbvcoll_b200 import ops
    emb, g, ids = rand(9, 52).to(BF).float(), rand(52, seed=1), torch.tensor([3, 8, 0, 3])
    x, h = torch.full((4, 64), 5.0, device=DEV), torch.empty(4, 64, dtype=dtype, device=DEV)
    ops.residual(x, padded(g, 64, F32), h, 52, 1e-3, embed=(ids.to(DEV), padded(emb, 64, dtype), 1.0, None))
    assert torch.equal(x[:, :52].cpu(), emb[ids]) and not x[:, 52:].any()
    close(h[:, :52], oracle.rms(emb[ids], 1e-3) * g, dtype)


# ---- projections --------------------------------------------------------------------------------------------------------------
@pytest.mark.parametrize("N,K,M,cols", [(1, 100, 176, 96), (7, 640, 80, 48), (40, 4096, 144, 144), (200, 64, 400, 208), (600, 320, 1040, 560), (1500, 128, 2064, 16)])
@pytest.mark.parametrize("dtype", [BF, F32])
def test_silu_on_leading_columns_and_relu_units(N, K, M, cols, dtype, persist_mode):
    """Every form of the product: split and plain decode form, both tiles of the many-token form."""
    from libtbvcoll_b200 import ops
    Kp = pad16(K)
    x, w = rand(N, K, seed=1).to(dtype).float(), (2.0 * rand(M, K, seed=2) / K ** 0.5).to(dtype).float()
    z = x.double() @ w.double().T
    xd, wd = padded(x, Kp, dtype), padded(w, Kp, dtype)
    for mode in ((1, 2, 3) if N >= 384 and dtype is BF else (1,)):
        persist_mode(mode)
        out = torch.empty(N, M, dtype=dtype, device=DEV)
        ops.linear(xd, wd, out, act=ops.ACT_SILU, act_cols=cols)
        close(out[:, :cols], oracle.silu(z[:, :cols]), dtype)
        if cols < M:
            close(out[:, cols:], z[:, cols:], dtype)
        half = torch.empty(N, M // 2, dtype=dtype, device=DEV)
        ops.linear(xd, wd, half, glu=ops.RELU_GLU)
        close(half, torch.relu(z[:, 0::2]) * z[:, 1::2], dtype)
    assert not ops.gemm_error()


# ---- mixture of experts by table --------------------------------------------------------------------------------------------
@pytest.mark.parametrize("T", [1, 5, 33, 1500])
def test_places_of_several_tables(T):
    from libtbvcoll_b200 import ops
    V, kinds = 57, [(1, 1), (5, 3), (300, 7), (24, 24)]
    ids = torch.randint(0, V, (T,), generator=torch.Generator().manual_seed(T))
    tables = [torch.stack([perm(E, 50 * v + i)[:top] for v in range(V)]).to(**I32) for i, (E, top) in enumerate(kinds)]
    place, offsets = [torch.full((T * top,), -1, **I32) for _, top in kinds], [torch.full((E + 1,), -1, **I32) for E, _ in kinds]
    ops.moe_place_table(ids.to(DEV), ops.moe_table_layers([(t, p, o, E) for t, p, o, (E, _) in zip(tables, place, offsets, kinds)], DEV), 300, V)
    for t, p, o, (E, top) in zip(tables, place, offsets, kinds):
        want = t.cpu()[ids].reshape(-1).long()                                  # expert of every (token, choice)
        assert torch.equal(o.cpu().long(), torch.cat((torch.zeros(1, dtype=torch.long), torch.bincount(want, minlength=E).cumsum(0))))
        assert sorted(p.tolist()) == list(range(T * top))                       # every row once
        at = torch.empty(T * top, dtype=torch.long)
        at[p.cpu().long()] = want
        assert torch.equal(at, want.sort().values)                              # and among the rows of its expert


@pytest.mark.parametrize("T", [1, 6, 90, 700])
@pytest.mark.parametrize("dtype", [BF, F32])
def test_a_whole_mixture(T, dtype):
    """Norm to the experts' rows, clamped units, down products and the weighted sum behind the branch's norm."""
    from libtbvcoll_b200 import ops
    W, E, top, ff, V, limit, eps = 80, 9, 4, 52, 40, 0.7, 1e-5
    Wp, fp = pad16(W), pad16(ff)
    toks = torch.randint(0, V, (T,), generator=torch.Generator().manual_seed(1)).tolist()
    x, g, gb = rand(T, W, seed=2), rand(W, seed=3), rand(W, seed=4)
    w = {"table": torch.stack([perm(E, v)[:top] for v in range(V)])}
    for e in range(E):
        for k, s in (("gate", (ff, W)), ("up", (ff, W)), ("down", (W, ff))):
            w[f"e{e}.{k}"] = (2.0 * rand(*s, seed=10 * e + len(k)) / s[1] ** 0.5).to(dtype).float()
    h = oracle.rms(x, eps) * g
    y = oracle.moe(h, w, "", {"router": {"experts": E, "top": top}, "expert": {"ff": ff, "limit": limit}}, toks, oracle.to_bf16 if dtype is BF else oracle.exact)
    gu = torch.stack([torch.stack((padded(padded(w[f"e{e}.gate"], Wp, dtype).T, fp, dtype).T, padded(padded(w[f"e{e}.up"], Wp, dtype).T, fp, dtype).T), 1) for e in range(E)]).reshape(E * 2 * fp, Wp).contiguous()
    dn = torch.stack([padded(padded(w[f"e{e}.down"], fp, dtype).T, Wp, dtype).T for e in range(E)]).reshape(E * Wp, fp).contiguous()
    place, off, table = torch.zeros(T * top, **I32), torch.zeros(E + 1, **I32), w["table"].to(**I32)
    ops.moe_place_table(torch.tensor(toks, device=DEV), ops.moe_table_layers([(table, place, off, E)], DEV), E, V)
    xd, xp, act, routed = padded(x, Wp, F32), *(torch.empty(T * top, n, dtype=dtype, device=DEV) for n in (Wp, fp, Wp))
    ops.residual(xd, padded(g, Wp, F32), xp, W, eps, place=place.view(T, top))
    ops.linear_rows(xp, gu, act, off, E, T, glu=(limit, 1.702, 1.0))
    ops.linear_rows(act, dn, routed, off, E, T)
    out = torch.empty(T, Wp, dtype=dtype, device=DEV)
    ops.residual(xd, padded(g, Wp, F32), out, W, eps, post=padded(gb, Wp, F32), routed=(routed, place.view(T, top), 1.0 / top))
    want = x + oracle.rms(y, eps) * gb
    close(xd[:, :W], want, dtype)
    close(out[:, :W], oracle.rms(want, eps) * g, dtype, 2e-2 if dtype is BF else None)


# ---- recurrence with one decay per head ------------------------------------------------------------------------------------------
class Lightning:
    """One sequence; q, k, v as they enter the recurrence."""

    def __init__(self, T, decay, D, V, seed=0, dtype=F32):
        n = lambda *s, o=0, by=1.0: (by * rand(*s, seed=10 * seed + o)).to(dtype).float()
        H = len(decay)
        self.T, self.H, self.D, self.V, self.decay = T, H, D, V, decay
        self.q, self.k, self.v, self.g = n(T, H, D), n(T, H, D, o=1, by=D ** -0.5), n(T, H, V, o=2), n(T, H * V, o=3)
        self.norm = 1 + 0.2 * rand(H * V, seed=77)
        self.finish()

    def finish(self):
        self.o = oracle.fixed_decay_attention(self.q.double(), self.k.double(), self.v.double(), torch.tensor(self.decay).double())
        self.want = (self.o.flatten(1) * self.norm * oracle.sigmoid(self.g.double())).view(self.T, self.H, self.V)


def run(seqs, portions, state, slots, dtype, group_rows=None, step=False):
    """The next ``portions[i]`` = (start, end) of every sequence as one batch; (outputs [rows, H, V], mean squares of o [rows]) per sequence."""
    from libtbvcoll_b200 import ops
    from libtbvcoll_b200.engine.batch import scan_groups
    s0 = seqs[0]
    H, D, V = s0.H, s0.D, s0.V
    K, Vw = H * pad16(D), H * pad16(V)
    wide = torch.cat([torch.cat([pad_heads(t[a:b], dtype) for t in (s.q, s.k, s.v, s.g.view(s.T, H, V))], 1) for s, (a, b) in zip(seqs, portions)])
    segs, at = [], 0
    for (a, b), slot in zip(portions, slots):
        segs.append([at, b - a, slot, 0])
        at += b - a
    pos, sd = torch.cat([torch.arange(a, b) for a, b in portions]).to(**I32), torch.tensor(segs, **I32)
    out = torch.empty(at, Vw, dtype=dtype, device=DEV)
    sums = torch.full((at, H if step else ops.fixed_decay_sums(H, pad16(V), dtype)), -1.0, device=DEV)
    args = (*wide.split((K, K, Vw, Vw), 1), pad_heads(s0.norm.view(1, H, V), F32)[0], ops.decay_powers(s0.decay, DEV), state, out, sums, sd, pos)
    if step:
        ops.fixed_decay_step(*args)
    elif dtype is F32:
        ops.fixed_decay_scan(*args, o=torch.empty(at * Vw, device=DEV))
    else:
        gr = scan_groups(sd.cpu().numpy(), group_rows)
        scratch = torch.full((len(gr) * K * pad16(V),), 9.0, device=DEV) if len(gr) > len(segs) else None
        ops.fixed_decay_scan(*args, groups=torch.from_numpy(gr).to(DEV), scratch=scratch)
    out = out.view(at, H, pad16(V))
    assert not out[..., V:].any()
    return [(out[f: f + n, :, :V], sums[f: f + n].sum(1) / (H * V)) for f, n, _, _ in segs]


def agrees(s, got, dtype, rows=slice(None)):
    """Outputs and square sums against the whole sequence's."""
    close(torch.cat([g[0] for g in got]), s.want[rows], dtype)
    ms = s.o.flatten(1).pow(2).mean(1)[rows]
    err = (torch.cat([g[1] for g in got]).cpu().double() / ms - 1).abs().max()
    assert float(err) < (1e-2 if dtype is BF else 1e-4), float(err)


SIZES = [([0.9, 0.5, 1.0], 24, 20), ([0.97, 0.2], 32, 64), ([0.99, 0.7], 96, 144), ([0.8], 128, 128), ([0.95, 0.999], 200, 16), ([0.6], 160, 272), ([0.9], 64, 80)]


@pytest.mark.parametrize("size", SIZES)
@pytest.mark.parametrize("form", ["f32", "chunks", "groups"])
def test_recurrence_over_portions(size, form):
    """Whole sequences and portions down to one token, of unequal sequences in one batch, slots that held something else: the same outputs and the
    same final state as one plain pass."""
    decay, D, V = size
    dtype, rows = F32 if form == "f32" else BF, {"chunks": 512, "groups": 64}.get(form)
    seqs = [Lightning(n, decay, D, V, seed=n, dtype=dtype) for n in (97, 33, 150)]
    state = torch.full((6, len(decay), pad16(D), pad16(V)), 5.0, device=DEV)
    for s, o in zip(seqs, run(seqs, [(0, s.T) for s in seqs], state, (2, 5, 1), dtype, rows)):
        agrees(s, [o], dtype)
    whole = state[[2, 5, 1]].clone()
    assert bool((state[[0, 3, 4]] == 5.0).all())
    # cut points that fall inside, at and around chunks of 32
    cuts = [(0, 2, 3, 31, 32, 67, 96, 97), (0, 1, 15, 16, 17, 30, 32, 33), (0, 32, 64, 65, 96, 100, 149, 150)]
    at = [[] for _ in seqs]
    for j in range(7):
        for i, o in enumerate(run(seqs, [(c[j], c[j + 1]) for c in cuts], state, (3, 2, 4), dtype, rows)):
            at[i].append(o)
    for s, o in zip(seqs, at):
        agrees(s, o, dtype)
    close(state[[3, 2, 4]], whole, dtype, 2e-5)                             # carried in 32-bit in every form
    S = torch.zeros(len(decay), D, V, dtype=torch.float64)
    for t in range(97):
        S = torch.tensor(decay).double()[:, None, None] * S + seqs[0].k[t].double()[:, :, None] * seqs[0].v[t].double()[:, None, :]
    close(state[3, :, :D, :V], S, dtype, 2e-5)


@pytest.mark.parametrize("dtype", [BF, F32])
def test_one_token_form_and_scan_hand_the_state_to_each_other(dtype):
    for decay, D, V in SIZES:
        s = Lightning(40, decay, D, V, seed=3, dtype=dtype)
        state = torch.full((4, len(decay), pad16(D), pad16(V)), -3.0, device=DEV)
        got = [run([s], [(a, a + 1)], state, (3,), dtype, step=True)[0] for a in range(6)]             # from the first token
        got += run([s], [(6, 25)], state, (3,), dtype, 64)
        got += [run([s], [(a, a + 1)], state, (3,), dtype, step=True)[0] for a in range(25, 40)]
        agrees(s, got, dtype)
        assert bool((state[:3] == -3.0).all())


def test_steps_of_several_sequences():
    a, b = (Lightning(5, [0.9, 0.4], 40, 24, seed=n, dtype=BF) for n in (1, 2))
    state, got = torch.full((5, 2, 48, 32), 8.0, device=DEV), [[], []]
    for t in range(5):
        for i, o in enumerate(run([a, b], [(t, t + 1)] * 2, state, (4, 1), BF, step=True)):
            got[i].append(o)
    agrees(a, got[0], BF)
    agrees(b, got[1], BF)
    assert bool((state[[0, 2, 3]] == 8.0).all())


@pytest.mark.parametrize("rows", [1024, 96, 32])
def test_decays_of_nothing_and_everything(rows):
    """A head that forgets at once, one that never forgets and one whose powers underflow within a chunk."""
    s = Lightning(200, [0.0, 1.0, 1e-3, 0.9999], 32, 32, seed=4, dtype=BF)
    state = torch.zeros(2, 4, 32, 32, device=DEV)
    agrees(s, run([s], [(0, 200)], state, (1,), BF, rows), BF)
    assert bool(torch.isfinite(state).all())
    close(state[1, 0], s.k[199, 0].double()[:, None] * s.v[199, 0].double()[None], BF, 1e-6)
    got = run([s], [(0, 70)], state, (1,), BF, rows) + run([s], [(70, 71)], state, (1,), BF, step=True) + run([s], [(71, 200)], state, (1,), BF, rows)
    agrees(s, got, BF)


@pytest.mark.parametrize("dtype,rows", [(F32, None), (BF, 1024), (BF, 64)])
def test_a_far_key_in_the_state(dtype, rows):
    """One key of the first chunk, hardly decayed, is what the last query asks for: its value must come out, not the sum of the hundreds between."""
    s = Lightning(900, [0.9999], 64, 64, seed=8, dtype=dtype)
    s.q = s.q * 0.01
    s.k[:, :, 0] = 0.0
    s.k[5], s.q[899] = 0.0, 0.0
    s.k[5, :, 0], s.q[899, :, 0] = 1.0, 8.0
    s.norm[:], s.g[:] = 1.0, 20.0
    s.q = s.q.to(dtype).float()
    s.finish()
    close(s.want[899, 0], 8.0 * 0.9999 ** 894 * s.v[5, 0], F32)
    state = torch.zeros(2, 1, 64, 64, device=DEV)
    close(run([s], [(0, 900)], state, (1,), dtype, rows)[0][0][899, 0], s.want[899, 0], dtype)
    got = [run([s], [(a, b)], state, (1,), dtype, rows)[0] for a, b in ((0, 4), (4, 301), (301, 899))] + run([s], [(899, 900)], state, (1,), dtype, step=True)
    close(got[-1][0][0, 0], s.want[899, 0], dtype)


# ---- attention ----------------------------------------------------------------------------------------------------------------
class Attn:
    """Queries and keys before their norms; windows or chunks, soft cap, rotation and gate as given."""

    def __init__(self, H, G, D, V, T, window=0, chunk=0, cap=None, rot=0, gated=True, seed=0, dtype=F32, block=16, base=50.0):
        from libtbvcoll_b200 import ops
        self.H, self.G, self.D, self.V, self.T, self.window, self.chunk, self.cap, self.rot, self.dtype, self.block, self.base, self.ops = \
            H, G, D, V, T, window, chunk, cap, rot, dtype, block, base, ops
        self.eps, self.scale = 1e-5, 0.8 * D ** -0.5
        self.q, self.k, self.v = (rand(T, h, d, seed=seed + i).to(dtype).float() for i, (h, d) in enumerate(((H, D), (G, D), (G, V))))
        self.g = rand(T, H * V, seed=seed + 3).to(dtype).float() if gated else None
        self.qn, self.kn = 1.5 + 0.3 * rand(H * D, seed=seed + 4), 1.5 + 0.3 * rand(G * D, seed=seed + 5)

    def mask(self):
        if self.chunk:
            return oracle.chunk_mask(self.T, self.chunk)
        return oracle.window_mask(self.T, self.window or self.T)

    def queries_keys(self):
        turn = lambda x: oracle.rotate(x, self.rot, self.base)
        r = oracle.to_bf16 if self.dtype is BF else oracle.exact
        q = r(turn(oracle.whole_norm(self.q.flatten(1), self.qn, self.eps).view(self.T, self.H, self.D)) * self.scale)
        return q, r(turn(oracle.whole_norm(self.k.flatten(1), self.kn, self.eps).view(self.T, self.G, self.D)))

    def want(self):
        o = oracle.softmax_attention(*self.queries_keys(), self.v, 1.0, self.mask(), self.cap)
        return o if self.g is None else o * oracle.sigmoid(self.g).view(o.shape)

    def write(self, start, end, cache, table, n_rows_form, own=True):
        """Prepares rows start..end-1 of the sequence; (queries of the rows form, projections, positions)."""
        D, V, dt = pad16(self.D), pad16(self.V), self.dtype
        parts = [pad_heads(t[start:end], dt) for t in ((self.q, self.k, self.v) if own else (self.q,))]
        wide = torch.cat(parts + ([pad_heads(self.g[start:end].view(-1, self.H, self.V), dt)] if self.g is not None else []), 1)
        pos = torch.arange(start, end, **I32)
        slots = table[(pos // self.block).long()].long() * self.block + pos % self.block
        qa = torch.full((n_rows_form, self.H, D + 8), 9.0, dtype=dt, device=DEV)
        qn, kn = pad_heads(self.qn.view(1, self.H, self.D) * self.scale, F32)[0], pad_heads(self.kn.view(1, self.G, self.D), F32)[0]
        turns = self.ops.rotation_turns(self.rot, self.base, DEV) if self.rot else None
        self.ops.paired_attention_prep(wide, qa, cache if own else None, qn, kn if own else None, turns, pos, slots, n_rows_form, self.H, self.G if own else 0, self.D,
                                       self.block, self.eps)
        return qa, wide, pos

    def new_cache(self, blocks):
        return torch.full((blocks * self.G * self.block, pad16(self.D) + pad16(self.V) + 8), float("nan"), dtype=self.dtype, device=DEV)     # a stale row must not matter

    def gate(self, wide):
        return None if self.g is None else wide[:, -self.H * pad16(self.V):]

    def rows(self, qa, wide, pos, cache, table, splits=1):
        n = qa.shape[0]
        out = torch.empty(n, self.H, pad16(self.V), dtype=self.dtype, device=DEV)
        self.ops.paired_attention_rows(qa, cache, table[None], torch.zeros(n, **I32), pos + 1, out, self.G, self.block, self.cap or 0.0, self.window, self.chunk,
                                       self.gate(wide), splits)
        assert not out[..., self.V:].any()
        return out[..., : self.V]

    def prefill(self, wide, start, cache, table):
        n = wide.shape[0]
        out = torch.empty(n, self.H * pad16(self.V), dtype=self.dtype, device=DEV)
        tiles = torch.tensor([[a, min(64, n - a), 0, start + a + 1] for a in range(0, n, 64)], **I32)
        self.ops.paired_attention_prefill(wide, cache, table[None], torch.zeros(n, **I32), tiles, out, self.H, self.G, pad16(self.D), self.block, self.cap or 0.0,
                                          self.window, self.chunk, self.gate(wide))
        return out.view(n, self.H, -1)[..., : self.V]


def scattered(blocks, seed=3):
    return (perm(blocks, seed) + 1).to(**I32)


SHAPES = [(6, 2, 40, 24, dict(window=9, rot=12)), (4, 4, 16, 48, dict(chunk=13, cap=3.0, gated=False)), (8, 1, 64, 64, dict(window=64, rot=64, cap=10.0)),
          (20, 1, 128, 112, dict(window=100, rot=32)), (24, 2, 100, 128, dict(chunk=64, cap=15.0)), (2, 1, 144, 32, dict(window=33, rot=144)),
          (3, 3, 256, 256, dict(chunk=50, gated=False)), (5, 1, 48, 320, dict(window=17, rot=10)), (4, 2, 32, 32, dict(window=1)), (4, 2, 32, 64, dict(rot=2)),
          (16, 16, 64, 48, dict(chunk=1)), (9, 3, 320, 128, dict(window=150, rot=8, gated=False))]


@pytest.mark.parametrize("H,G,D,V,kw", SHAPES)
@pytest.mark.parametrize("dtype", [BF, F32])
def test_attention_whole_portions_and_single_rows(H, G, D, V, kw, dtype):
    a = Attn(H, G, D, V, 213, seed=H, dtype=dtype, **kw)
    want, table = a.want(), scattered(14)
    cache = a.new_cache(15)
    got, at, fits = [], 0, a.ops.paired_prefill_fits(pad16(D), pad16(V))
    for n, form in ((70, "prefill"), (1, "rows"), (2, "rows"), (33, "prefill"), (1, "rows"), (31, "rows"), (64, "prefill"), (11, "rows")):
        many = form == "prefill" and dtype is BF and fits
        qa, wide, pos = a.write(at, at + n, cache, table, 0 if many else n)
        got.append(a.prefill(wide, at, cache, table) if many else a.rows(qa, wide, pos, cache, table, splits=1 + at % 4))
        at += n
    close(torch.cat(got), want, dtype)
    assert at == 213 and not a.ops.gemm_error()
    # queries alone (a layer that reads another's cache) turn out the same
    qa, wide, pos = a.write(100, 130, None, table, 30, own=False)
    close(a.rows(qa, wide, pos, cache, table), want[100:130], dtype)


@pytest.mark.parametrize("dtype", [BF, F32])
@pytest.mark.parametrize("D,V", [(64, 64), (144, 96)])
@pytest.mark.parametrize("limit", ["window", "chunk"])
def test_keys_just_inside_and_just_outside(dtype, D, V, limit):
    """A query scaled so that the score of ONE key stands out of all others: with the key just inside the limit its value comes out, just outside it must
    not; limits at and off the edges of blocks, units and tiles, prompts and single rows, each number of splits."""
    T = 420
    for size in (1, 2, 16, 31, 32, 33, 64, 100, 128, 200):
        a = Attn(4, 2, D, V, T, seed=5, dtype=dtype, gated=False, **{limit: size})
        a.qn[:], a.kn[:] = 1.0, 1.0
        a.scale = 25.0 * D ** -0.5
        rows = sorted({r for e in (16, 32, 64, 128, 200, 256, 384, size, 2 * size, 3 * size) for r in range(e - 1, e + 2)} | {T - 1, T - 2, 303})
        rows = [r for r in rows if 0 < r < T]
        for n, r in enumerate(rows):
            first = max(0, r - size + 1) if limit == "window" else r // size * size
            a.q[r] = a.k[[first, max(first - 1, 0)][n % 2]].repeat_interleave(2, 0)           # the first key it sees, or the one before
        a.q = a.q.to(dtype).float()
        want, table, cache = a.want(), scattered(27), a.new_cache(28)
        _, wide, _ = a.write(0, T, cache, table, 0 if dtype is BF else T)
        if dtype is BF:
            close(a.prefill(wide, 0, cache, table)[rows], want[rows], dtype, 3e-2)
        qa, wide, pos = a.write(0, T, cache, table, T)
        for splits in (1, 2, 4, 8):
            close(a.rows(qa, wide, pos, cache, table, splits)[rows], want[rows], dtype, 3e-2 if dtype is BF else None)


@pytest.mark.parametrize("block", [8, 16, 32, 64])
def test_block_sizes(block):
    a = Attn(6, 2, 64, 48, 150, window=41, seed=2, rot=20, dtype=BF, block=block)
    table = scattered(-(-150 // block))
    cache = a.new_cache(len(table) + 1)
    _, wide, _ = a.write(0, 150, cache, table, 0)
    close(a.prefill(wide, 0, cache, table), a.want(), BF)
    qa, wide, pos = a.write(100, 150, cache, table, 50)
    close(a.rows(qa, wide, pos, cache, table, 2), a.want()[100:], BF)


@pytest.mark.parametrize("dtype", [BF, F32])
def test_norms_and_rotation_at_far_positions(dtype):
    """Queries and keys as they are written, against angles in double precision."""
    from libtbvcoll_b200 import ops
    H, G, D, V, rot, base, positions = 3, 1, 44, 20, 14, 500000.0, [0, 1, 2, 63, 4097, 65537, 999983]
    T, Dp, Vp = len(positions), 48, 32
    q, k, v = rand(T, H, D).to(dtype).float(), rand(T, G, D, seed=1).to(dtype).float(), rand(T, G, V, seed=2).to(dtype).float()
    qn, kn = 1 + 0.3 * rand(H * D, seed=3), 1 + 0.3 * rand(G * D, seed=4)

    def turned(x, n):
        x = oracle.whole_norm(x.flatten(1).double(), n.double(), 1e-5).view(T, -1, D).clone()
        for r, p in enumerate(positions):
            for i in range(rot // 2):
                c, s = math.cos(p * base ** (-2.0 * i / rot)), math.sin(p * base ** (-2.0 * i / rot))
                a, b = x[r, :, 2 * i].clone(), x[r, :, 2 * i + 1].clone()
                x[r, :, 2 * i], x[r, :, 2 * i + 1] = a * c - b * s, b * c + a * s
        return x
    wide = torch.cat([pad_heads(t, dtype) for t in (q, k, v)], 1)
    cache, qa = torch.full((32, Dp + Vp + 8), 3.0, dtype=dtype, device=DEV), torch.full((4, H, Dp + 8), 3.0, dtype=dtype, device=DEV)
    slots = torch.tensor([17, 3, 31, 0, -1, 8, 20], device=DEV)
    ops.paired_attention_prep(wide, qa, cache, pad_heads(qn.view(1, H, D), F32)[0], pad_heads(kn.view(1, G, D), F32)[0], ops.rotation_turns(rot, base, DEV),
                              torch.tensor(positions, **I32), slots, 4, H, G, D, 16, 1e-5)
    tol = 8e-3 if dtype is BF else 1e-6
    close(qa[..., :D], turned(q, qn)[:4], dtype, tol)
    close(wide[4:, : H * Dp].view(3, H, Dp)[..., :D], turned(q, qn)[4:], dtype, tol)
    keep = [i for i in range(T) if i != 4]                                     # slot -1: nothing is written
    close(cache[slots[keep], :D], turned(k, kn)[keep, 0], dtype, tol)
    assert torch.equal(cache[slots[keep], Dp: Dp + V], v[keep, 0].to(dtype).to(DEV)) and int((cache == 3.0).all(1).sum()) == 32 - len(keep)
