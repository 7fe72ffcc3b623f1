"""Nubosun without a GPU: configuration and registry, weight layout, row layout of a step, request bookkeeping, the scheduler's
decisions, rotation frequencies, and the oracle's own causality."""
import json

import numpy as np
import pytest
import torch

import nubosun_cases as cases
import nubosun_oracle as oracle


def parse(name):
    from libtbvcoll_b200.models.config import parse_nubosun_config
    return parse_nubosun_config(cases.CASES[name]())


def test_config_runs_and_registry(tmp_path):
    from libtbvcoll_b200.models.config import LatentSpec, MambaSpec, get_config, parse_nubosun_config
    from libtbvcoll_b200.models.registry import architecture_of, load_config
    raw = cases.CASES["odd"]()
    (tmp_path / "config.json").write_text(json.dumps(raw))
    c = load_config(str(tmp_path))
    assert architecture_of(c).name == "nubosun" and architecture_of(get_config("tiny")).name == "llama"
    assert c.runs == oracle.layer_order(raw) == [0, 1, 2, 1, 2, 1, 2, 3] and c.num_layers == 8
    assert isinstance(c.layers[0].mixer, LatentSpec) and isinstance(c.layers[1].mixer, MambaSpec) and c.layers[1].mlp is None
    assert c.layers[0].mlp.limit == 1.5 and c.layers[0].mixer.rot.scaling["factor"] == 4.0 and c.logit_softcap == 20.0
    with pytest.raises(ValueError):
        c.check_tp(2)
    for bad in ("nope", {"type": "other"}):
        r = cases.CASES["plain"]()
        if isinstance(bad, dict):
            r["layers"][0].update(bad)
            with pytest.raises(ValueError):
                parse_nubosun_config(r)
        else:
            r["architecture"] = bad
            (tmp_path / "config.json").write_text(json.dumps(r))
            with pytest.raises(ValueError):
                load_config(str(tmp_path))
    r = cases.CASES["plain"]()
    r["loop"] = {"start": 1, "stop": 4, "times": 2}
    with pytest.raises(ValueError):
        parse_nubosun_config(r)


@pytest.mark.parametrize("name", sorted(cases.CASES))
def test_padded_weights_compute_the_same_products(name):
    """The loaded layout (stacked, padded, folded) gives the plain products of the checkpoint's tensors."""
    from libtbvcoll_b200.utils.weights import load_nubosun, nubosun_tensor_shapes
    raw = cases.CASES[name]()
    cfg, w = parse(name), cases.tensors(raw)
    assert {k: tuple(t.shape) for k, t in w.items()} == {k: tuple(v) for k, v in nubosun_tensor_shapes(cfg).items()}
    p = load_nubosun(cfg, cases.Source(w), "cpu", torch.float32)
    W = raw["width"]
    for i, e in enumerate(raw["layers"]):
        m, q = e["mixer"], f"l{i}.mix."
        f = {k: t.float() for k, t in w.items() if k.startswith(q)}
        x = torch.randn(W)
        xp = torch.zeros(p["final.norm"].shape[0])
        xp[:W] = x
        pad = lambda n: (n + 15) // 16 * 16
        if e["type"] == "mamba1":
            I, ip = m["inner"], pad(m["inner"])
            a, b = p[q + "in"] @ xp, f[q + "in"] @ x
            assert torch.allclose(a[:I], b[:I], atol=1e-4) and torch.allclose(a[ip:ip + I], b[I:], atol=1e-4)
            assert not a[I:ip].any() and not a[ip + I:].any()
            assert torch.allclose(p[q + "a2"], -torch.exp(f[q + "A_log"]) / np.log(2.0), rtol=1e-5)
            assert torch.equal(p[q + "conv"][:, :I], f[q + "conv"].T)
        else:
            H, D, r, v, K = (m[k] for k in ("heads", "dim", "rot_dim", "vdim", "kv_rank"))
            Dp, rp, vp, Kp = pad(D), pad(r), pad(v), pad(K)
            a, b = p[q + "qkv"] @ xp, (f[q + "q"] @ x).view(H, D + r)
            assert torch.allclose(a[: H * Dp].view(H, Dp)[:, :D], b[:, :D], atol=1e-4)
            assert torch.allclose(a[H * Dp: H * (Dp + rp)].view(H, rp)[:, :r], b[:, D:], atol=1e-4)
            c, d = a[H * (Dp + rp):], f[q + "dkv"] @ x
            assert torch.allclose(c[:K], d[:K], atol=1e-4) and torch.allclose(c[Kp: Kp + r], d[K:], atol=1e-4)
            lat = torch.randn(K)
            latp = torch.zeros(Kp)
            latp[:K] = lat
            keys, qn = (f[q + "uk"] @ lat).view(H, D), b[:, :D]
            folded = (p[q + "wabs"].view(H, Kp, Dp)[:, :, :D] * qn[:, None]).sum(-1)
            assert torch.allclose((keys * qn).sum(-1), folded @ latp, atol=1e-3)
            assert torch.allclose((p[q + "wuv"] @ latp).view(H, vp)[:, :v], (f[q + "uv"] @ lat).view(H, v), atol=1e-4)
            heads = torch.randn(H, v)
            hp = torch.zeros(H, vp)
            hp[:, :v] = heads
            assert torch.allclose((p[q + "o"] @ hp.reshape(-1))[:W], f[q + "o"] @ heads.reshape(-1), atol=1e-4)
    bad = dict(w)
    bad["head"] = w["head"][:-1]
    with pytest.raises(ValueError):
        load_nubosun(cfg, cases.Source(bad), "cpu")


def test_rotation_frequencies():
    from libtbvcoll_b200.ops import rope_frequencies
    for dims, base, sc in ((36, 1e4, None), (64, 5e5, {"factor": 6.0, "original": 4096, "fast": 30.0, "slow": 1.0}),
                           (10, 1e4, cases.YARN), (2, 100.0, cases.YARN), (48, 2e6, {"factor": 40.0, "original": 128, "fast": 1.0, "slow": 1.0})):
        f, factor = rope_frequencies(dims, base, sc)
        want, wf = oracle.rotary_frequencies({"dims": dims, "base": base, "scaling": sc})
        assert np.allclose(f.numpy(), want, rtol=1e-12) and abs(factor - wf) < 1e-12


def test_rows_of_a_mixed_step():
    from libtbvcoll_b200.engine.batch import Portion, lay_out
    from libtbvcoll_b200.engine.kv_cache import BlockManager
    bm = BlockManager(64, 16, 4, 16, "cpu")
    for row, n in ((0, 100), (1, 41), (2, 7), (3, 130)):
        bm.reserve(row, n)
    parts = [Portion(0, 30, list(range(70)), (0, 69)), Portion(1, 40, [5], (0,)), Portion(3, 0, list(range(130)), ()), Portion(2, 3, [1, 2, 3, 4], (1, 3))]
    hb = lay_out(parts, bm.tables_host.numpy(), 16, rows_form_max=8)
    assert hb.order == [1, 3, 0, 2] and hb.n_rows_form == 5
    assert hb.segs.tolist() == [[0, 1, 2, 0], [1, 4, 3, 0], [5, 70, 1, 0], [75, 130, 4, 0]]
    assert hb.want_rows.tolist() == [5, 74, 0, 2, 4]                       # in the order the portions were given
    for t in range(hb.ids.size):
        assert hb.slots[t] == bm.slot(int(hb.seq[t]), int(hb.pos[t]))
    covered = {}
    for first, n, base, see in hb.dense_tiles.tolist():
        for r in range(n):
            covered[first + r] = (base, see + r)
    assert sorted(covered) == list(range(5, 205))
    for t, (base, see) in covered.items():
        assert see == hb.pos[t] + 1 and base == (0 if t < 75 else 100)
    assert hb.dense_slots.tolist() == [bm.slot(0, i) for i in range(100)] + [bm.slot(3, i) for i in range(130)]
    same = lay_out(parts, bm.tables_host.numpy(), 16)                       # one attention form: order kept
    assert same.order == [0, 1, 2, 3] and same.n_rows_form == 0 and same.dense_tiles is None


def test_request_table_reuses_rows_and_blocks():
    from libtbvcoll_b200.engine.kv_cache import BlockManager, RequestTable
    bm = BlockManager(9, 16, 2, 8, "cpu")                                   # eight usable blocks, two rows
    t = RequestTable(bm)
    assert t.extend("a", 60) == (0, 0) and t.extend("b", 60) == (1, 0) and t.extend("a", 4) == (0, 60)
    with pytest.raises(RuntimeError):
        t.extend("c", 1)                                                    # no row
    with pytest.raises(RuntimeError):
        t.extend("a", 1)                                                    # no block: 4 + 4 in use
    mine = list(bm.owned[0])
    t.end("a")
    assert t.extend("c", 33).row == 0 and set(bm.owned[0]) <= set(mine) and t.live["c"].length == 33
    t.end("never admitted")
    t.end_all()
    assert len(bm.free) == 8 and sorted(t.free_rows) == [0, 1] and not t.live


class FakeEngine:
    """Records steps; the 'model' answers with the sum of the tokens it has seen so far for the request, modulo 1000."""

    def __init__(self, max_batch, blocks, rows):
        from libtbvcoll_b200.engine.kv_cache import BlockManager, RequestTable
        self.max_batch, self.max_seq_len, self.prefill_chunk = max_batch, 200, rows
        self.bm = BlockManager(blocks + 1, 16, max_batch, 13, "cpu")
        self.requests, self.seen, self.log = RequestTable(self.bm), {}, []

    def step(self, entries, end=(), sample=True):
        assert sum(len(t) for _, t, _ in entries) <= self.prefill_chunk and len({k for k, _, _ in entries}) == len(entries)
        out = []
        for k, toks, want in entries:
            self.requests.extend(k, len(toks))
            self.seen[k] = self.seen.get(k, 0) + sum(toks)
            out += [self.seen[k] % 1000] * len(want)
        self.log.append([(len(t), len(w)) for _, t, w in entries])
        return out


def test_scheduler_batches_portions_beside_decoded_tokens():
    from libtbvcoll_b200.engine.scheduler import Scheduler
    eng = FakeEngine(max_batch=3, blocks=12, rows=24)
    prompts = [list(range(1, n + 1)) for n in (40, 3, 17, 60, 1, 30)]
    outs = Scheduler(eng).run(prompts, 5)
    for p, o in zip(prompts, outs):
        total, want = sum(p), []
        for _ in range(5):
            want.append(total % 1000)
            total += want[-1]
        assert o == want
    assert any(any(n == 1 and w for n, w in s) and any(n > 1 for n, _ in s) for s in eng.log)       # mixed steps happened
    assert len(eng.bm.free) == 12 and not eng.requests.live
    with pytest.raises(ValueError):
        Scheduler(eng).run([[1] * 199], 5)
    stop = Scheduler(FakeEngine(2, 12, 24)).run([[1, 2], [3]], 5, eos_id=3)
    assert stop[0] == [3] and stop[1] == [3]


def test_oracle_is_causal_and_takes_every_case():
    for name in cases.CASES:
        cfg = cases.CASES[name]()
        w, toks = cases.tensors(cfg), cases.tokens(cfg, 21)
        full = oracle.forward(cfg, w, toks)
        assert torch.isfinite(full).all() and full.std() > 0.3
        assert torch.allclose(full[:13], oracle.forward(cfg, w, toks[:13]), atol=2e-4)


MUTATIONS = {
    "no sink": lambda m: m.setattr(oracle, "sink_softmax", lambda s, k: torch.softmax(s, -1)),
    "sink scaled": lambda m, f=oracle.sink_softmax: m.setattr(oracle, "sink_softmax", lambda s, k: f(s, k * 0.5)),
    "own key hidden": lambda m, f=oracle.sink_softmax: m.setattr(oracle, "sink_softmax", lambda s, k: f(
        s.masked_fill(torch.eye(s.shape[-1], dtype=torch.bool), float("-inf")), k)),
    "first key hidden": lambda m, f=oracle.sink_softmax: m.setattr(oracle, "sink_softmax", lambda s, k: f(
        torch.cat((s[..., :1].masked_fill(torch.arange(s.shape[-1])[:, None] > 0, float("-inf")), s[..., 1:]), -1), k)),
    "halves rotated": lambda m: m.setattr(oracle, "rotate_pairs", lambda x, p, r: torch.roll(x, 1, -1)),
    "no position": lambda m: m.setattr(oracle, "rotate_pairs", lambda x, p, r: x),
    "position off by one in the query only": lambda m, f=oracle.rotate_pairs: m.setattr(oracle, "rotate_pairs", lambda x, p, r: f(x, p + (x.shape[1] > 1), r)),
    "no scaling of frequencies": lambda m, f=oracle.rotary_frequencies: m.setattr(oracle, "rotary_frequencies", lambda r: f({**r, "scaling": None})),
    "convolution late by one": lambda m, f=oracle.causal_conv: m.setattr(oracle, "causal_conv", lambda x, t, b: f(torch.cat((x[:1] * 0, x[:-1])), t, b)),
    "no bias in the convolution": lambda m, f=oracle.causal_conv: m.setattr(oracle, "causal_conv", lambda x, t, b: f(x, t, b * 0)),
    "state lost at token 9": lambda m, f=oracle.selective_scan: m.setattr(oracle, "selective_scan", lambda u, dt, a, b, c, d: torch.cat(
        (f(u[:9], dt[:9], a, b[:9], c[:9], d), f(u[9:], dt[9:], a, b[9:], c[9:], d)))),
    "no skip": lambda m, f=oracle.selective_scan: m.setattr(oracle, "selective_scan", lambda u, dt, a, b, c, d: f(u, dt, a, b, c, d * 0)),
    "no clamp": lambda m, f=oracle.clamped_glu_mlp: m.setattr(oracle, "clamped_glu_mlp", lambda h, w, p, c, r=None: f(h, w, p, {"limit": 1e9})),
    "mix transposed": lambda m, f=oracle.hyper_sublayer: m.setattr(oracle, "hyper_sublayer", lambda xs, fn, g, s, i, o, x, e: f(xs, fn, g, s, i, o, x.T, e)),
    "no layer scale": lambda m, f=oracle.hyper_sublayer: m.setattr(oracle, "hyper_sublayer", lambda xs, fn, g, s, i, o, x, e: f(xs, fn, g, s * 0 + 1, i, o, x, e)),
    "loop run once": lambda m: m.setattr(oracle, "layer_order", lambda c: list(range(len(c["layers"])))),
}


@pytest.mark.parametrize("name", sorted(MUTATIONS))
def test_the_cases_show_a_wrong_mechanism(monkeypatch, name):
    """A mistake planted in the oracle must stand out of what rounding to 16 bits does on at least one of the cases."""
    ratios = []
    for case in ("odd", "plain", "wide"):
        cfg = cases.CASES[case]()
        w, toks = cases.tensors(cfg), cases.tokens(cfg, 24)
        right, rounded = oracle.forward(cfg, w, toks), oracle.forward(cfg, w, toks, r=oracle.to_bf16)
        with monkeypatch.context() as m:
            MUTATIONS[name](m)
            wrong = oracle.forward(cfg, w, toks)
        ratios.append(float((wrong - right)[12:].norm() / (rounded - right)[12:].norm()))
    assert max(ratios) > 6, ratios


def test_command_line_help():
    import os
    import subprocess
    import sys
    root = os.path.dirname(os.path.dirname(os.path.abspath(__file__)))
    for cmd in ([sys.executable, "-m", "libtbvcoll_b200.generate", "--help"], [os.path.join(root, "bin", "trace_run"), "--help"]):
        r = subprocess.run(cmd, capture_output=True, text=True, timeout=300, cwd=root)
        assert r.returncode == 0 and "--model" in r.stdout and "--dtype" in r.stdout
