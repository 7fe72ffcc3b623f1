"""Bobarax without a GPU: configuration and registry, weight layout, and what the oracle and the cases can tell apart."""
import json

import pytest
import torch

import bobarax_cases as cases
import bobarax_oracle as oracle


def parse(name):
    from libtbvcoll_b200.models.config import parse_bobarax_config
    return parse_bobarax_config(cases.CASES[name]())


def test_config_and_registry(tmp_path):
    from libtbvcoll_b200.models.config import GatedMlpSpec, LightningSpec, PairedAttentionSpec, RotationSpec, TableMoeSpec, get_config, parse_bobarax_config
    from libtbvcoll_b200.models.registry import architecture_of, load_config
    raw = cases.CASES["odd"]()
    (tmp_path / "config.json").write_text(json.dumps(raw))
    c = load_config(str(tmp_path))
    assert architecture_of(c).name == architecture_of(get_config("bobarax-2k")).name == "bobarax"
    assert (c.residual_mult, c.logit_scale, c.rms_eps, c.num_layers) == (0.6, 0.4, 1e-5, 5)
    assert [type(x.mixer) for x in c.layers] == [PairedAttentionSpec, LightningSpec, PairedAttentionSpec, PairedAttentionSpec, LightningSpec]
    a, b, s = (c.layers[i].mixer for i in (0, 2, 3))
    assert (a.kv_heads, a.vdim, a.window, a.chunk, a.gated, a.softcap, a.rot, a.kv_from) == (2, 24, 9, 0, True, None, RotationSpec(12, 300.0), None)
    assert (b.window, b.chunk, b.gated, b.softcap, b.rot) == (0, 13, False, 3.0, None) and (s.kv_from, s.window, s.scale) == (0, 33, 0.2)
    assert c.layers[1].mixer.decay == [1.0, 0.55, 0.97] and c.layers[1].mlp == GatedMlpSpec(70) and c.layers[0].mlp == TableMoeSpec(5, 3, 28, 0.8) and c.layers[2].mlp is None
    with pytest.raises(ValueError):
        c.check_tp(2)

    def broken(change):
        r = cases.CASES["odd"]()
        change(r["layers"])
        with pytest.raises(ValueError):
            parse_bobarax_config(r)
    broken(lambda r: r[0].update(type="other"))
    broken(lambda r: r[0]["mixer"].update(kv_heads=4))
    broken(lambda r: r[0]["mlp"].update(kind="sparse"))
    broken(lambda r: r[0]["mlp"]["router"].update(top=6))
    broken(lambda r: r[0]["mixer"]["rot"].update(dims=42))
    broken(lambda r: r[1]["mixer"].update(decay=[0.5]))
    broken(lambda r: r[1]["mixer"].update(decay=[0.5, 1.5, 0.1]))
    for j in (1, 2, 3, 4, -1):                # a recurrence, other sizes, itself, a later one, none
        broken(lambda r: r[3]["mixer"].update(kv_from=j))


@pytest.mark.parametrize("name", sorted(cases.CASES))
def test_padded_weights_compute_the_same_products(name):
    """The loaded layout (stacked, padded, interleaved) gives the plain products of the checkpoint's tensors."""
    from libtbvcoll_b200.utils.weights import RandomSource, bobarax_tensor_shapes, load_bobarax
    raw = cases.CASES[name]()
    cfg, w = parse(name), cases.tensors(raw)
    assert {k: tuple(t.shape) for k, t in w.items()} == bobarax_tensor_shapes(cfg)
    p = load_bobarax(cfg, cases.Source(w), "cpu", torch.float32)
    W, pad = raw["width"], lambda n: (n + 15) // 16 * 16
    x = torch.randn(W)
    xp = torch.zeros(pad(W))
    xp[:W] = x
    same = lambda a, b: torch.allclose(a, b, atol=1e-4)
    assert torch.equal(p["embed"][: raw["vocab"], :W], w["embed"].float())
    assert same(p["final.norm"][:W], (1 + w["final.norm"].float()) * raw["logit_scale"])

    def heads(t, n, d):                       # padded heads without their padding
        t = t.reshape(n, pad(d))
        assert not t[:, d:].any()
        return t[:, :d].reshape(-1)
    for i, e in enumerate(raw["layers"]):
        m, q, H, D, V = e["mixer"], f"l{i}.mix.", e["mixer"]["heads"], e["mixer"]["dim"], e["mixer"]["vdim"]
        f = {k[len(q):]: t.float() for k, t in w.items() if k.startswith(q)}
        assert same(p[f"l{i}.norm1"][:W], 1 + w[f"l{i}.norm1"].float()) and same(p[f"l{i}.norm1b"][:W], (1 + w[f"l{i}.norm1b"].float()) * raw["residual_mult"])
        parts, G = [("q", H, D)], H if e["type"] == "lightning" else m["kv_heads"]
        if m.get("kv_from") is None:
            parts += [("k", G, D), ("v", G, V)]
        if e["type"] != "attention":
            parts.append(("g", H, V))
        y = (p[q + "in"] @ xp).split([n * pad(d) for _, n, d in parts])
        for (s, n, d), t in zip(parts, y):
            assert same(heads(t, n, d), f[s] @ x)
        if e["type"] == "lightning":
            assert same(heads(p[q + "norm"], H, V), f["norm"])
        else:
            assert same(heads(p[q + "q.norm"], H, D), f["q.norm"] * m["scale"]) and (q + "k.norm" in p) == ("k" in f)
            if "k" in f:
                assert same(heads(p[q + "k.norm"], G, D), f["k.norm"])
        o = torch.randn(H, V)
        op = torch.zeros(H, pad(V))
        op[:, :V] = o
        assert same((p[q + "o"] @ op.reshape(-1))[:W], f["o"] @ o.reshape(-1))
        if e["mlp"]:
            q, mix = f"l{i}.mlp.", e["mlp"]["kind"] == "moe"
            E, ff = (e["mlp"]["router"]["experts"], e["mlp"]["expert"]["ff"]) if mix else (1, e["mlp"]["ff"])
            for j in range(E):
                src, gu, dn = f"e{j}." if mix else "", p[q + "gate_up"].view(E, 2 * pad(ff), -1)[j], p[q + "down"].view(E, pad(W), -1)[j]
                z = gu @ xp
                assert same(z[0::2][:ff], w[q + src + "gate"].float() @ x) and same(z[1::2][:ff], w[q + src + "up"].float() @ x) and not z[2 * ff:].any()
                a = torch.zeros(pad(ff))
                a[:ff] = torch.randn(ff)
                assert same((dn @ a)[:W], w[q + src + "down"].float() @ a[:ff])
            if mix:
                assert p[q + "table"].dtype is torch.int32 and torch.equal(p[q + "table"], w[q + "table"])
    for bad in (dict(w, embed=w["embed"][:-1]), {k: t + 50 if k.endswith("table") else t for k, t in w.items()}):
        with pytest.raises(ValueError):
            load_bobarax(cfg, cases.Source(bad), "cpu")
    src = RandomSource(cfg, seed=3)           # random weights load as well; integer tables stay integers
    assert set(load_bobarax(cfg, src, "cpu")) == set(p)


def test_integer_tensors_of_a_checkpoint_keep_their_values(tmp_path):
    from libtbvcoll_b200.utils.weights import SafetensorsSource
    raw = cases.config([cases.lightning([0.5], 16, 16, cases.moe(400, 3, 16, 1.0))], 16, 40)
    w = cases.tensors(raw)
    cases.write_checkpoint(str(tmp_path), raw, w)
    t = SafetensorsSource(str(tmp_path), dtype=torch.bfloat16).get("l0.mlp.table")
    assert not t.is_floating_point() and torch.equal(t, w["l0.mlp.table"]) and int(t.max()) > 256     # beyond what 16-bit floats hold exactly


def test_rotation_turns_hold_far_positions():
    from libtbvcoll_b200.ops import rotation_turns
    t, p = rotation_turns(12, 300.0, "cpu").double(), 1e6
    for i in range(6):
        want = p * 300.0 ** (-2.0 * i / 12) / (2 * torch.pi)
        assert abs(p * float(t[i].sum()) - want) < 1e-7 * max(1.0, want * 1e-3)


def test_splits_follow_what_a_row_sees():
    from libtbvcoll_b200.models.bobarax import Bobarax
    from libtbvcoll_b200.models.config import PairedAttentionSpec
    m = lambda **k: PairedAttentionSpec(4, 2, 16, 16, 1.0, **k)
    assert [Bobarax.layer_splits(m(window=n), 8) for n in (1, 64, 128, 300, 512, 4096)] == [1, 1, 2, 4, 8, 8]
    assert Bobarax.layer_splits(m(chunk=130), 4) == 2 and Bobarax.layer_splits(m(), 8) == 8


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


def _late(q, k, v, kv_from):
    return (q, k, v) if kv_from is None else (q, k.roll(1, 0), v)


def _split(f, q, k, v, a, at=9):
    """A recurrence that forgets its state at token ``at``."""
    return torch.cat((f(q[:at], k[:at], v[:at], a), f(q[at:], k[at:], v[at:], a)))


def _halves(x, dims, base, f=oracle.rotate):
    """Dimension i paired with dimension i + dims / 2."""
    order = [j for i in range(dims // 2) for j in (i, i + dims // 2)]
    y = f(torch.cat((x[:, :, order], x[:, :, dims:]), -1), dims, base)
    out = y.clone()
    out[:, :, order] = y[:, :, :dims]
    return out


MUTATIONS = {
    "window one longer": _with("window_mask", lambda f: lambda T, n: f(T, n + 1)),
    "window one shorter": _with("window_mask", lambda f: lambda T, n: f(T, max(1, n - 1))),
    "chunks one longer": _with("chunk_mask", lambda f: lambda T, n: f(T, n + 1)),
    "chunks from the second token": _with("chunk_mask", lambda f: lambda T, n: f(T + 1, n)[1:, 1:]),
    "chunks as a window": _with("chunk_mask", lambda f: lambda T, n: oracle.window_mask(T, n)),
    "first key hidden": _with("window_mask", lambda f: lambda T, n: f(T, n) & ((torch.arange(T)[None] > 0) | (torch.arange(T)[:, None] == 0))),
    "no soft cap": _with("softcap", lambda f: lambda s, c: s),
    "no rotation": _with("rotate", lambda f: lambda x, d, b: x),
    "rotation of halves": _with("rotate", lambda f: _halves),
    "rotation of every dimension": _with("rotate", lambda f: lambda x, d, b: f(x, x.shape[2], b)),
    "heads normed one by one": _with("whole_norm", lambda f: lambda x, w, eps: oracle.rms(x.reshape(x.shape[0], -1, 4), eps).reshape(x.shape) * w),
    "query and key weights about zero": _with("whole_norm", lambda f: lambda x, w, eps: f(x, 1 + w, eps)),
    "wrong key head": lambda m, f=torch.Tensor.repeat_interleave: m.setattr(torch.Tensor, "repeat_interleave", lambda t, n, d: t.repeat(1, n, 1)),
    "values late by one": _with("softmax_attention", lambda f: lambda q, k, v, *a: f(q, k, v.roll(1, 0), *a)),
    "shared keys late by one": _with("queries_keys_values", lambda f: lambda h, w, i, m, *a: _late(*f(h, w, i, m, *a), m.get("kv_from"))),
    "no gate": _with("sigmoid", lambda f: lambda z: torch.ones_like(z) if z.dim() == 2 else f(z)),
    "new keys decay as well": _with("fixed_decay_attention", lambda f: lambda q, k, v, a: f(q, k * a[None, :, None], v, a)),
    "reads before it writes": _with("fixed_decay_attention", lambda f: lambda q, k, v, a: f(q, k, v, a) - (q * k).sum(-1, keepdim=True) * v),
    "decays of the heads in reverse": _with("fixed_decay_attention", lambda f: lambda q, k, v, a: f(q, k, v, a.flip(0))),
    "state lost at token 9": _with("fixed_decay_attention", lambda f: lambda *a: _split(f, *a)),
    "no activation of the projections": _with("silu", lambda f: lambda z: z),
    "heads of the recurrence normed one by one": _with("joint_norm_gate", lambda f: lambda o, w, g, eps: oracle.rms(o, eps).reshape(o.shape[0], -1) * w * oracle.sigmoid(g)),
    "gate of the recurrence with SiLU": _with("joint_norm_gate", lambda f: lambda o, w, g, eps: f(o, w, g, eps) * g),
    "dense with SiLU": lambda m: m.setattr(torch, "relu", oracle.silu),
    "no limit of the experts": _with("clamped_unit", lambda f: lambda g, u, limit: f(g, u, 1e9)),
    "gate clamped from below too": _with("clamped_unit", lambda f: lambda g, u, limit: f(torch.clamp(g, min=-limit), u, limit)),
    "no one beside u": _with("clamped_unit", lambda f: lambda g, u, limit: f(g, u, limit) - f(g, u * 0, limit)),
    "plain sigmoid in the experts": _with("clamped_unit", lambda f: lambda g, u, limit: torch.clamp(g, max=limit) * oracle.sigmoid(torch.clamp(g, max=limit)) * (torch.clamp(u, -limit, limit) + 1)),
    "last expert left out": _with("table_weights", lambda f: lambda t, table, e: f(t, table[:, : max(1, table.shape[1] - 1)], e)),
    "experts of the next token": _with("table_weights", lambda f: lambda t, table, e: f(t[1:] + t[:1], table, e)),
    "no norm behind": _with("layer", lambda f: lambda x, c, w, i, *a: f(x, c, {k: (v * 0 if k.startswith(f"l{i}.norm") and k.endswith("b") else v) for k, v in w.items()}, i, *a)),
    "no residual multiplier": _with("layer", lambda f: lambda x, c, *a: f(x, {**c, "residual_mult": 1.0}, *a)),
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
        ratios.append(float(((wrong - right).norm(dim=1) / (rounded - right).norm(dim=1))[9:].max()))
    assert max(ratios) > 6, ratios
