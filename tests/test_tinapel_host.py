"""Tinapel without a GPU: configuration and registry, weight layout, groups of rows, and what the oracle and the cases can tell apart."""
import json

import numpy as np
import pytest
import torch

import tinapel_cases as cases
import tinapel_oracle as oracle


def parse(name):
    from libtbvcoll_b200.models.config import parse_tinapel_config
    return parse_tinapel_config(cases.CASES[name]())


def test_config_schedule_and_registry(tmp_path):
    from libtbvcoll_b200.models.config import GlaSpec, SharedKvSpec, WkvSpec, get_config, parse_tinapel_config
    from libtbvcoll_b200.models.registry import architecture_of, load_config
    raw = cases.CASES["odd"]()
    (tmp_path / "config.json").write_text(json.dumps(raw))
    c = load_config(str(tmp_path))
    assert architecture_of(c).name == architecture_of(get_config("tinapel-2k")).name == "tinapel"
    assert c.schedule == oracle.passes(raw) == [(0, None), (1, 0), (2, None), (1, 1), (2, None), (1, 2), (2, None), (3, None), (4, None)]
    assert c.runs == [0, 1, 2, 1, 2, 1, 2, 3, 4] and c.num_layers == 9
    assert [type(x.mixer) for x in c.layers] == [SharedKvSpec, WkvSpec, GlaSpec, SharedKvSpec, WkvSpec]
    a = c.layers[0].mixer
    assert (a.kv_heads, a.scale, a.softcap, a.temp_coef, a.temp_every) == (2, 0.31, 4.0, 0.7, 9.0) and c.layers[3].mlp is None
    f = c.layers[2].mlp
    assert (f.experts, f.top, f.ff, f.scale, f.shared_ff) == (7, 2, 44, 2.5, 52) and parse("large").layers[1].mlp.shared_ff is None
    assert parse("plain").loop is None and parse("wide").schedule[3] == (0, 1)
    with pytest.raises(ValueError):
        c.check_tp(2)

    def broken(change):
        r = cases.CASES["odd"]()
        change(r)
        with pytest.raises(ValueError):
            parse_tinapel_config(r)
    broken(lambda r: r["layers"][0].update(type="other"))
    broken(lambda r: r["layers"][0]["mixer"].update(kv_heads=4))
    broken(lambda r: r["layers"][0]["mixer"].update(vdim=8))
    broken(lambda r: r["layers"][0]["mlp"].update(kind="dense"))
    broken(lambda r: r["layers"][0]["mlp"]["router"].update(top=6))
    broken(lambda r: r["loop"].update(stop=6))


@pytest.mark.parametrize("name", sorted(cases.CASES))
def test_padded_weights_compute_the_same_products(name):
    """The loaded layout (stacked, padded, interleaved) gives the plain products of the checkpoint's tensors."""
    from libtbvcoll_b200.utils.weights import load_tinapel, tinapel_tensor_shapes
    raw = cases.CASES[name]()
    cfg, w = parse(name), cases.tensors(raw)
    assert set(w) == set(tinapel_tensor_shapes(cfg))
    p = load_tinapel(cfg, cases.Source(w), "cpu", torch.float32)
    W, pad = raw["width"], lambda n: (n + 15) // 16 * 16
    x = torch.randn(W)
    xp = torch.zeros(pad(W))
    xp[:W] = x
    same = lambda a, b: torch.allclose(a, b, atol=1e-4)
    assert torch.equal(p["embed"][: raw["vocab"], :W], w["embed"].float()) and torch.equal(p["final.norm"][:W], 1 + w["final.norm"].float())

    def heads(t, n, d):                       # padded heads without their padding
        t = t.reshape(n, pad(d))
        assert not t[:, d:].any()
        return t[:, :d].reshape(-1)
    for i, e in enumerate(raw["layers"]):
        m, q = e["mixer"], f"l{i}.mix."
        f = {k[len(q):]: t.float() for k, t in w.items() if k.startswith(q)}
        H, D = m["heads"], m["dim"]
        y = p[q + "in"] @ xp
        K = H * pad(D)
        if e["type"] == "attention":
            G = m["kv_heads"]
            assert same(heads(y[:K], H, D), f["q"] @ x) and same(heads(y[K:], G, D), f["k"] @ x)
            assert same(p[q + "fold"][:D], f["q.norm"] * f["k.norm"] * m["scale"])
            vd = D
        else:
            vd = m.get("vdim", D)
            V = H * pad(vd)
            names = ("q", "k", "v", "g", "a1") if e["type"] == "gla" else ("r", "k", "v", "g", "w1")
            parts = y.split((K, K, V, V, p[q + "decay"].shape[1]))
            for s, part, d in zip(names[:4], parts, (D, D, vd, vd)):
                assert same(heads(part, H, d), f[s] @ x)
            low = f[names[4]] @ x
            assert same(parts[4][: low.numel()], low) and not parts[4][low.numel():].any()
            lp = torch.zeros(p[q + "decay"].shape[1])
            lp[: low.numel()] = low
            second, bias = (f["a2"], f["a2.b"]) if e["type"] == "gla" else (f["w2"], f["w0"])
            assert same(heads(p[q + "decay"] @ lp + p[q + "decay.b"], H, D), second @ low + bias)
            assert same(heads(p[q + "norm"], H, vd), f["norm"].repeat(H) if e["type"] == "gla" else f["norm"])
            if e["type"] == "wkv":
                assert same(heads(p[q + "u"], H, D), f["u"].reshape(-1)) and same(p[q + "mu"][:, :W], torch.stack([f["mu." + s] for s in "rkvgw"]))
        o = torch.randn(H, vd)
        op = torch.zeros(H, pad(vd))
        op[:, :vd] = o
        assert same((p[q + "o"] @ op.reshape(-1))[:W], f["o"] @ o.reshape(-1))
        if e["mlp"]:
            q, E = f"l{i}.mlp.", e["mlp"]["router"]["experts"]
            for k, src in [(j, f"e{j}.") for j in range(E)] + ([(None, "shared.")] if e["mlp"]["shared"] else []):
                ff = (e["mlp"]["shared"] if k is None else e["mlp"]["expert"])["ff"]
                gu = p[q + "shared.gate_up"] if k is None else p[q + "gate_up"].view(E, 2 * pad(ff), -1)[k]
                dn = p[q + "shared.down"] if k is None else p[q + "down"].view(E, pad(W), -1)[k]
                z = gu @ xp
                assert same(z[0::2][:ff], w[q + src + "gate"].float() @ x) and same(z[1::2][:ff], w[q + src + "up"].float() @ x) and not z[2 * ff:].any()
                a = torch.zeros(pad(ff))
                a[:ff] = torch.randn(ff)
                assert same((dn @ a)[:W], w[q + src + "down"].float() @ a[:ff])
    bad = dict(w)
    bad["embed"] = w["embed"][:-1]
    with pytest.raises(ValueError):
        load_tinapel(cfg, cases.Source(bad), "cpu")


def test_position_turns_hold_far_positions():
    """High and low part together: the angle of position 10^6 keeps seven digits, where a single fp32 frequency would lose it."""
    from libtbvcoll_b200.ops import position_turns
    t = position_turns(48, "cpu").double()
    p = 1e6
    for i in range(24):
        want = p * 10000.0 ** (-2.0 * i / 48) / (2 * np.pi)
        assert abs(p * float(t[i].sum()) - want) < 1e-7 * max(1.0, want * 1e-3)


def test_groups_of_rows():
    from libtbvcoll_b200.engine.batch import scan_groups
    segs = np.array([[0, 40, 3, 0], [40, 1, 1, 0], [41, 96, 2, 0]], dtype=np.int32)
    assert scan_groups(segs, 96).tolist() == [[0, 40, 3, 0], [40, 1, 1, 0], [41, 96, 2, 0]]
    assert scan_groups(segs, 32).tolist() == [[0, 32, 3, 2], [32, 8, 3, 1], [40, 1, 1, 0], [41, 32, 2, 2], [73, 32, 2, 3], [105, 32, 2, 1]]


@pytest.mark.parametrize("name", sorted(cases.CASES))
def test_oracle_is_causal_and_the_experts_are_decided(monkeypatch, name):
    cfg = cases.CASES[name]()
    w, toks = cases.tensors(cfg), cases.tokens(cfg, 40)
    gaps, route = [], oracle.route

    def watch(z, top, scale):
        v = z.sort(-1, descending=True).values
        if top < z.shape[1]:
            gaps.append(float((v[:, top - 1] - v[:, top]).min() / v.std()))
        return route(z, top, scale)
    monkeypatch.setattr(oracle, "route", watch)
    full = oracle.forward(cfg, w, toks)
    assert torch.isfinite(full).all() and full.std() > 0.3
    assert min(gaps) > 0.15, gaps
    assert torch.allclose(full[:13], oracle.forward(cfg, w, toks[:13]), atol=2e-4)


def _with(name, change):
    """Plants a wrapper around an oracle function."""
    return lambda m, f=getattr(oracle, name): m.setattr(oracle, name, change(f))


def _visible(keep):
    """Softmax whose mask also hides keys by (query, key) position."""
    def soft(f):
        def g(s, dim):
            if s.dim() == 3:
                i, j = torch.arange(s.shape[1])[:, None], torch.arange(s.shape[2])[None]
                s = s.masked_fill(~keep(i, j) & (i != j), float("-inf"))
            return f(s, dim)
        return g
    return lambda m, f=torch.softmax: m.setattr(torch, "softmax", soft(f))


def _split(f, *args, at=9):
    """A recurrence that forgets its state at token ``at``."""
    cut = lambda a, s: a[s] if a.dim() == 3 else a
    return torch.cat((f(*(cut(a, slice(0, at)) for a in args)), f(*(cut(a, slice(at, None)) for a in args))))


MUTATIONS = {
    "no position vector": _with("position_vector", lambda f: lambda T, W, d: f(T, W, d) * 0),
    "sine and cosine swapped": _with("position_vector", lambda f: lambda T, W, d: f(T, W, d).view(T, -1, 2).flip(-1).reshape(T, W)),
    "positions from one": _with("position_vector", lambda f: lambda T, W, d: f(T + 1, W, d)[1:]),
    "first key hidden": _visible(lambda i, j: j > 0),
    "keys of 16 back hidden": _visible(lambda i, j: i - j < 16),
    "no soft cap": lambda m, f=oracle.attention_mixer: m.setitem(oracle.MIXERS, "attention", lambda h, w, p, c, e, r: f(h, w, p, {**c, "softcap": None}, e, r)),
    "no temperature": _with("query_temperature", lambda f: lambda T, c, e, d: f(T, c, e, d) * 0 + 1),
    "temperature late by one": _with("query_temperature", lambda f: lambda T, c, e, d: torch.cat((f(1, c, e, d), f(T, c, e, d)[:-1]))),
    "wrong key head": lambda m, f=torch.Tensor.repeat_interleave: m.setattr(torch.Tensor, "repeat_interleave", lambda t, n, d: t.repeat(1, n, 1)),
    "gla reads before it writes": _with("gated_linear_attention", lambda f: lambda q, k, v, a: f(q, k, v, a) - (q * k).sum(-1, keepdim=True) * v),
    "gla decay late by one": _with("gated_linear_attention", lambda f: lambda q, k, v, a: f(q, k, v, torch.cat((a[:1], a[:-1])))),
    "gla state lost at token 9": _with("gated_linear_attention", lambda f: lambda *a: _split(f, *a)),
    "gla decay on the values' side": _with("gated_linear_attention", lambda f: lambda q, k, v, a: f(q, k, v, a.mean(-1, keepdim=True).expand_as(a))),
    "no tau": lambda m, f=oracle.gla_mixer: m.setitem(oracle.MIXERS, "gla", lambda h, w, p, c, e, r: f(h, w, p, {**c, "tau": 1.0}, e, r)),
    "no token shift": _with("token_shift", lambda f: lambda h, mu: h),
    "token shift reversed": _with("token_shift", lambda f: lambda h, mu: f(h, 1 - mu)),
    "shift lost at token 9": _with("token_shift", lambda f: lambda h, mu: torch.cat((f(h[:9], mu), f(h[9:], mu)))),
    "no bonus": _with("wkv", lambda f: lambda r, k, v, w, u: f(r, k, v, w, u * 0)),
    "bonus stays in the state": _with("wkv", lambda f: lambda r, k, v, w, u: f(r, k * u, v, w, u * 0 + 1)),
    "wkv state lost at token 9": _with("wkv", lambda f: lambda *a: _split(f, *a)),
    "one expert too few": _with("route", lambda f: lambda z, t, s: f(z, max(1, t - 1), s)),
    "expert weights not normalised": _with("route", lambda f: lambda z, t, s: f(z, t, s) * (torch.softmax(z, -1) * (f(z, t, s) > 0)).sum(-1, keepdim=True)),
    "no router scale": _with("route", lambda f: lambda z, t, s: f(z, t, 1.0)),
    "no shared expert": _with("moe", lambda f: lambda h, w, p, c, r: f(h, w, p, {**c, "shared": None}, r)),
    "norm weight not about zero": _with("layer", lambda f: lambda x, c, w, i, r: f(x, c, {k: (v - 1 if k.startswith(f"l{i}.norm") else v) for k, v in w.items()}, i, r)),
    "loop run once": _with("passes", lambda f: lambda c: f({**c, "loop": {**c["loop"], "times": 1}} if c.get("loop") else c)),
    "embedding not added again": _with("passes", lambda f: lambda c: [(i, 0 if t else t) for i, t in f(c)]),
    "step once": _with("passes", lambda f: lambda c: [(i, t or None) for i, t in f(c)]),
}


@pytest.mark.parametrize("name", sorted(MUTATIONS))
def test_the_cases_show_a_wrong_mechanism(monkeypatch, name):
    """A mistake planted in the oracle must stand out of what rounding to 16 bits does, at some position of at least one of the cases."""
    ratios = []
    for case in ("odd", "plain", "wide"):
        cfg = cases.CASES[case]()
        w, toks = cases.tensors(cfg), cases.tokens(cfg, 24)
        right, rounded = oracle.forward(cfg, w, toks), oracle.forward(cfg, w, toks, r=oracle.to_bf16)
        with monkeypatch.context() as m:
            MUTATIONS[name](m)
            wrong = oracle.forward(cfg, w, toks)
        ratios.append(float(((wrong - right).norm(dim=1) / (rounded - right).norm(dim=1))[9:].max()))
    assert max(ratios) > 6, ratios
