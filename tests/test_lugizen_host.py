"""Lugizen without a GPU: configuration and registry, weight layout, batches, and what the oracle and the cases can tell apart."""
import json

import numpy as np
import pytest
import torch

import lugizen_cases as cases
import lugizen_oracle as oracle


def parse(name):
    from libtbvcoll_b200.models.config import parse_lugizen_config
    return parse_lugizen_config(cases.CASES[name]())


def test_config_and_registry(tmp_path):
    from libtbvcoll_b200.models.config import (ChannelDeltaSpec, GeluMlpSpec, HeadAttentionSpec, LatentSpec, MoeSpec, RotationSpec, get_config, parse_lugizen_config)
    from libtbvcoll_b200.models.registry import architecture_of, load_config
    raw = cases.CASES["odd"]()
    (tmp_path / "config.json").write_text(json.dumps(raw))
    c = load_config(str(tmp_path))
    assert architecture_of(c).name == architecture_of(get_config("lugizen-2k")).name == "lugizen"
    assert (c.canon_taps, c.rms_eps, c.num_layers, c.hidden_size, c.vocab_size) == (4, 1e-5, 7, 100, 203)
    assert c.layers[0].mixer == HeadAttentionSpec(6, 2, 40, 24, raw["layers"][0]["mixer"]["scale"], RotationSpec(12, 300.0), True) and c.layers[0].mlp == MoeSpec(5, 3, 28)
    assert c.layers[1].mixer == ChannelDeltaSpec(4, 2, 24, 36, 3) and c.layers[1].mlp == GeluMlpSpec(70) and c.layers[2].mlp is None
    la = c.layers[2].mixer
    assert isinstance(la, LatentSpec) and (la.window, la.q_rank, la.kv_rank, la.rot, la.rot_dim, la.vdim) == (9, 36, 52, RotationSpec(10, 500.0), 10, 44)
    assert not c.layers[6].mixer.v_mix
    with pytest.raises(ValueError):
        c.check_tp(2)

    def broken(change):
        r = cases.CASES["odd"]()
        change(r["layers"])
        with pytest.raises(ValueError):
            parse_lugizen_config(r)
    broken(lambda r: r[0].update(type="other"))
    broken(lambda r: r[0]["mixer"].update(kv_heads=4))
    broken(lambda r: r[0]["mixer"]["rot"].update(dims=42))
    broken(lambda r: r[0]["mixer"]["rot"].update(dims=11))
    broken(lambda r: r[0]["mlp"].update(kind="sparse"))
    broken(lambda r: r[0]["mlp"]["router"].update(top=6))
    broken(lambda r: r[1]["mixer"].update(kv_heads=3))
    broken(lambda r: r[1]["mixer"].update(conv=0))
    broken(lambda r: r[2]["mixer"]["rot"].update(dims=8))
    broken(lambda r: r[2]["mixer"].update(mask={"size": -1}))
    broken(lambda r: r[3]["mixer"].update(vdim=20))                  # does not mix with the first layer's values


@pytest.mark.parametrize("name", sorted(cases.CASES))
def test_padded_weights_compute_the_same_products(name):
    """The loaded layout (stacked, padded, interleaved, pairs next to each other) gives the plain products of the checkpoint's tensors."""
    from libtbvcoll_b200.utils.weights import RandomSource, load_lugizen
    raw = cases.CASES[name]()
    cfg, w = parse(name), cases.tensors(raw)
    p = load_lugizen(cfg, cases.Source(w), "cpu", torch.float32)
    W, pad = raw["width"], lambda n: (n + 15) // 16 * 16
    x = torch.randn(W)
    xp = torch.zeros(pad(W))
    xp[:W] = x
    same = lambda a, b: torch.allclose(a, b, atol=1e-4)
    assert torch.equal(p["embed"][:, :W], w["embed"].float()) and torch.equal(p["head"][: raw["vocab"], :W], w["head"].float())

    def heads(t, n, d):                       # padded heads without their padding
        t = t.reshape(n, pad(d))
        assert not t[:, d:].any()
        return t[:, :d].reshape(-1)

    def paired(t, n, dims):                   # dimensions i, i + dims / 2 of every head next to each other
        t = t.reshape(n, -1)
        order = [k for i in range(dims // 2) for k in (i, i + dims // 2)] + list(range(dims, t.shape[1]))
        return t[:, order].reshape(-1)
    for i, e in enumerate(raw["layers"]):
        m, q, H, D, V = e["mixer"], f"l{i}.mix.", e["mixer"]["heads"], e["mixer"]["dim"], e["mixer"]["vdim"]
        f = {k[len(q):]: t.float() for k, t in w.items() if k.startswith(q)}
        assert same(p[f"l{i}.norm1"], torch.cat((w[f"l{i}.norm1"].float().expand(W), torch.zeros(pad(W) - W))))
        assert torch.equal(p[f"l{i}.canon1"][:, :W], w[f"l{i}.canon1"].float().t())
        if e["type"] == "channel_delta":
            G, R = m["kv_heads"], pad(max(f["a1"].shape[0], f["g1"].shape[0]))
            parts = [("q", G, D), ("k", G, D), ("v", H, V)]
            *y, ya, yg, yb = (p[q + "in"] @ xp).split([n * pad(d) for _, n, d in parts] + [R, R, pad(H)])
            for (s, n, d), t in zip(parts, y):
                assert same(heads(t, n, d), f[s] @ x)
            assert same(yb[:H], f["b"] @ x)
            assert same(heads(p[q + "a2"] @ ya, H, D), f["a2"] @ (f["a1"] @ x)) and same(heads(p[q + "g2"] @ yg, H, V), f["g2"] @ (f["g1"] @ x))
            conv = p[q + "conv"].split([n * pad(d) for _, n, d in parts], 1)
            for (s, n, d), t in zip(parts, conv):
                assert same(torch.stack([heads(r, n, d) for r in t], 1), f[s + ".conv"])
            assert same(heads(p[q + "dt_bias"], H, D), f["dt_bias"]) and same(p[q + "rate"], f["A_log"].exp()) and same(p[q + "norm"][:V], f["norm"])
        elif e["type"] == "attention":
            G, dims = m["kv_heads"], m["rot"]["dims"]
            yq, yk, yv = (p[q + "in"] @ xp).split([H * pad(D), G * pad(D), G * pad(V)])
            assert same(heads(yq, H, D), paired(f["q"] @ x, H, dims)) and same(heads(yk, G, D), paired(f["k"] @ x, G, dims)) and same(heads(yv, G, V), f["v"] @ x)
            assert same(p[q + "qscale"], f["temp"] * m["scale"]) and (q + "vmix" in p) == m["v_mix"]
        else:
            R, Q, rot = m["kv_rank"], m["q_rank"], m["rot_dim"]
            yq, yc, yr = (p[q + "down"] @ xp).split([pad(Q), pad(R), pad(rot)])
            want = f["dkv"] @ x
            assert same(heads(yq, 1, Q), f["dq"] @ x) and same(heads(yc, 1, R), want[:R]) and same(heads(yr, 1, rot), paired(want[R:], 1, rot))
            qq = (f["uq"] @ (f["dq"] @ x)).view(H, D + rot)
            a, b = (p[q + "uq"] @ yq).split([H * pad(D), H * pad(rot)])
            assert same(heads(a, H, D), qq[:, :D].reshape(-1)) and same(heads(b, H, rot), paired(qq[:, D:], H, rot))
            fold = p[q + "wabs"].view(H, pad(R), pad(D)) @ a.view(H, pad(D), 1)
            assert same(fold[:, :R, 0], torch.einsum("hd,hdr->hr", qq[:, :D], f["uk"].view(H, D, R)))
            assert same(heads(p[q + "wuv"] @ yc, H, V), f["uv"] @ want[:R])
        o, op = torch.randn(H, V), torch.zeros(H, pad(V))
        op[:, :V] = o
        assert same((p[q + "o"] @ op.reshape(-1))[:W], f["o"] @ o.reshape(-1))
        if e["mlp"] and e["mlp"]["kind"] == "dense":
            q, ff = f"l{i}.mlp.", e["mlp"]["ff"]
            a = torch.zeros(pad(ff))
            a[:ff] = torch.randn(ff)
            assert same((p[q + "up"] @ xp)[:ff], w[q + "up"].float() @ x) and same((p[q + "down"] @ a)[:W], w[q + "down"].float() @ a[:ff])
        elif e["mlp"]:
            q, E = f"l{i}.mlp.", e["mlp"]["router"]["experts"]
            assert same((p[q + "router"] @ xp)[:E], w[q + "router"].float() @ x) and p[q + "gate_up"].shape[0] == E * 2 * pad(e["mlp"]["expert"]["ff"])
    with pytest.raises(ValueError):
        load_lugizen(cfg, cases.Source(dict(w, embed=w["embed"][:-1])), "cpu")
    src = RandomSource(cfg, seed=3)           # random weights load as well
    assert set(load_lugizen(cfg, src, "cpu", torch.float32)) == set(p)


def test_context_of_a_window():
    """Only what some row can see is expanded, from a multiple of 64 positions on; the tiles' first context row is where position 0 would be."""
    from libtbvcoll_b200.engine.batch import dense_context
    tables = np.arange(2 * 64, dtype=np.int32).reshape(2, 64) + 1
    for window in (0, 1, 64, 70, 1000):
        starts, counts, rows = (500, 0, 129, 63), (70, 5, 1, 200), (0, 1, 1, 0)
        first = [0, 70, 75, 76]
        tiles, slots = dense_context(first, counts, starts, rows, tables, 16, window)
        base = 0
        for f, n, s, r in zip(first, counts, starts, rows):
            skip = max(0, s + 1 - window) // 64 * 64 if window else 0
            pos = np.arange(skip, s + n)
            assert (slots[base: base + len(pos)] == tables[r, pos // 16] * 16 + pos % 16).all()
            mine = tiles[(tiles[:, 0] >= f) & (tiles[:, 0] < f + n)]
            assert (mine[:, 2] == base - skip).all() and sorted(mine[:, 3]) == [s + k + 1 for k in range(0, n, 64)] and mine[:, 1].sum() == n
            base += len(pos)
        assert base == len(slots)


def test_splits_follow_the_kernel_and_the_window():
    from libtbvcoll_b200.models.config import HeadAttentionSpec, LatentSpec
    from libtbvcoll_b200.models.lugizen import Lugizen
    model = Lugizen.__new__(Lugizen)
    model.sms = 148
    la = lambda window, heads=16: LatentSpec(heads, 16, 16, 16, 32, 1.0, q_rank=16, window=window)
    assert [model.layer_splits(la(n), 1, 8) for n in (0, 1, 127, 128, 300, 512, 4096)] == [8, 1, 1, 2, 4, 8, 8]
    assert [model.layer_splits(la(0, h), 32, 8) for h in (16, 17, 80)] == [4, 2, 1]
    at = HeadAttentionSpec(32, 8, 16, 16, 1.0)
    assert [model.layer_splits(at, r, 8) for r in (1, 3, 8, 32)] == [8, 8, 4, 1] and model.layer_splits(at, 1, 2) == 2


@pytest.mark.parametrize("name", sorted(cases.CASES))
def test_oracle_is_causal(name):
    cfg = cases.CASES[name]()
    w, toks = cases.tensors(cfg), cases.tokens(cfg, 40)
    full = oracle.forward(cfg, w, toks)
    assert torch.isfinite(full).all() and full.std() > 0.1
    assert torch.allclose(full[:13], oracle.forward(cfg, w, toks[:13]), atol=2e-4 * float(full.std()))


def _with(name, change):
    """Plants a wrapper around an oracle function."""
    return lambda m, f=getattr(oracle, name): m.setattr(oracle, name, change(f))


def _pairs(x, dims, base, f=oracle.rotate_half):
    """Dimension 2i paired with dimension 2i + 1."""
    order = list(range(0, dims, 2)) + list(range(1, dims, 2))
    y, out = f(torch.cat((x[:, :, order], x[:, :, dims:]), -1), dims, base), x.clone()
    out[:, :, order] = y[:, :, :dims]
    return out


def _old(q, k, v, beta, g):
    """Reads the state before the token's own write."""
    T, H, D = q.shape
    S, out = torch.zeros(H, D, v.shape[2], dtype=q.dtype), torch.zeros_like(v)
    for t in range(T):
        S = g[t][:, :, None] * S
        out[t] = (S * q[t][:, :, None]).sum(1)
        S = S + k[t][:, :, None] * (beta[t][:, None] * (v[t] - (S * k[t][:, :, None]).sum(1)))[:, None]
    return out


def _late_decay(q, k, v, beta, g):
    """The correction meets the state before it has decayed."""
    T, H, D = q.shape
    S, out = torch.zeros(H, D, v.shape[2], dtype=q.dtype), torch.zeros_like(v)
    for t in range(T):
        u = beta[t][:, None] * (v[t] - (S * k[t][:, :, None]).sum(1))
        S = g[t][:, :, None] * S + k[t][:, :, None] * u[:, None]
        out[t] = (S * q[t][:, :, None]).sum(1)
    return out


def _cut(f, at, *a):
    return torch.cat((f(*(t[:at] for t in a)), f(*(t[at:] for t in a))))


def _layer(change):
    """A layer with other weights."""
    return _with("layer", lambda f: lambda x, c, w, i, *a: f(x, c, change(dict(w), f"l{i}.", c), i, *a))


def _no_canon(w, p, c):
    w[p + "canon1"] = torch.zeros_like(w[p + "canon1"])
    return w


def _late_canon(w, p, c):
    w[p + "canon1"] = torch.cat((w[p + "canon1"][:, 1:], torch.zeros_like(w[p + "canon1"][:, :1])), 1)
    return w


MUTATIONS = {
    "window one longer": _with("window_mask", lambda f: lambda T, n: f(T, n + 1)),
    "window one shorter": _with("window_mask", lambda f: lambda T, n: f(T, max(1, n - 1))),
    "no window": _with("window_mask", lambda f: lambda T, n: oracle.causal_mask(T)),
    "first key hidden": _with("causal_mask", lambda f: lambda T: f(T) & ((torch.arange(T)[None] > 0) | (torch.arange(T)[:, None] == 0))),
    "no rotation": _with("rotate_half", lambda f: lambda x, d, b: x),
    "rotation of neighbours": _with("rotate_half", lambda f: _pairs),
    "another base": _with("rotate_half", lambda f: lambda x, d, b: f(x, d, 2 * b)),
    "heads normed together": _with("rms", lambda f: lambda x, eps: f(x.flatten(1), eps).reshape(x.shape) if x.dim() == 3 else f(x, eps)),
    "no norm of the heads": _with("rms", lambda f: lambda x, eps: x if x.dim() == 3 else f(x, eps)),
    "one number for all heads": _with("softmax_attention", lambda f: lambda q, k, v, s, *a: f(q, k, v, torch.as_tensor(s).reshape(-1)[0], *a)),
    "wrong key head": lambda m: m.setattr(torch.Tensor, "repeat_interleave", lambda t, n, d: t.repeat(1, n, 1)),
    "values late by one": _with("softmax_attention", lambda f: lambda q, k, v, *a: f(q, k, v.roll(1, 0), *a)),
    "no value mix": _with("value_mix", lambda f: lambda v, first, lam: v),
    "value mix the other way round": _with("value_mix", lambda f: lambda v, first, lam: f(first, v, lam)),
    "values mixed with the token before": _with("value_mix", lambda f: lambda v, first, lam: f(v, first.roll(1, 0), lam)),
    "no convolution of the stream": _layer(_no_canon),
    "convolution of the stream late by one": _layer(_late_canon),
    "convolutions without the token before": _with("causal_conv", lambda f: lambda x, t: f(x, torch.cat((t[:, :-2], 0 * t[:, -2:-1], t[:, -1:]), 1)) if t.shape[1] > 1 else f(x, t)),
    "no SiLU": _with("silu", lambda f: lambda z: z),
    "no unit vectors": _with("unit", lambda f: lambda x: x),
    "unit vectors by the mean": _with("unit", lambda f: lambda x: oracle.rms(x, 1e-6)),
    "reads before it writes": _with("delta_rule", lambda f: _old),
    "decays behind the correction": _with("delta_rule", lambda f: _late_decay),
    "no correction": _with("delta_rule", lambda f: lambda q, k, v, b, g: f(q, k, v / 1.0, b * 0 + 1, g) - f(q, k, v * 0.5, b * 0 + 1, g)),
    "one decay per head": _with("delta_rule", lambda f: lambda q, k, v, b, g: f(q, k, v, b, g.mean(2, keepdim=True).expand_as(g))),
    "decays of the next head": _with("delta_rule", lambda f: lambda q, k, v, b, g: f(q, k, v, b, g.roll(1, 1))),
    "step sizes of one": _with("delta_rule", lambda f: lambda q, k, v, b, g: f(q, k, v, torch.ones_like(b), g)),
    "state lost at token 16": _with("delta_rule", lambda f: lambda *a: _cut(f, 16, *a)),
    "exponential for softplus": _with("softplus", lambda f: torch.exp),
    "gates with SiLU": _with("sigmoid", lambda f: lambda z: f(z) * (z if z.dim() == 2 and z.shape[1] > 8 else 1)),
    "dense with SiLU": _with("gelu_tanh", lambda f: oracle.silu),
    "last expert left out": _with("router_weights", lambda f: lambda z, top: f(z, max(1, top - 1)) if top > 1 else f(z, top)),
    "experts weigh the same": _with("router_weights", lambda f: lambda z, top: (f(z, top) > 0).to(z.dtype) / top),
    "norms without their number": _with("scalar_norm", lambda f: lambda x, g, eps: f(x, 1.0, eps)),
    "no norm behind": _with("scalar_norm", lambda f: lambda x, g, eps: x * g),
}


@pytest.mark.parametrize("name", sorted(MUTATIONS))
def test_the_cases_show_a_wrong_mechanism(monkeypatch, name):
    """A mistake planted in the oracle must stand out of what rounding to 16 bits does, at some position of at least one of the cases."""
    ratios = []
    for case in ("odd", "plain", "wide"):
        cfg = cases.CASES[case]()
        w, toks = cases.tensors(cfg), cases.tokens(cfg, 60)
        right, rounded = oracle.forward(cfg, w, toks), oracle.forward(cfg, w, toks, r=oracle.to_bf16)
        with monkeypatch.context() as m:
            MUTATIONS[name](m)
            wrong = oracle.forward(cfg, w, toks)
        ratio = (wrong - right).norm(dim=1) / (rounded - right).norm(dim=1)
        ratios.append(float(torch.nan_to_num(ratio, nan=float("inf"))[9:].max()))
    assert max(ratios) > 6, ratios
