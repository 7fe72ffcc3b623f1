"""Lugizen through the engine: whole prompts, portions, mixed batches, pages and slots used again, decoding, generation, the trace replay
and the command line, against the plain statement in ``lugizen_oracle``."""
import json
import os
import random
import subprocess
import sys

import numpy as np
import pytest
import torch

import lugizen_cases as cases
import lugizen_oracle as oracle
from expected import BF, F32, Expected, feed, random_schedule

pytestmark = pytest.mark.gpu
ROOT = os.path.dirname(os.path.dirname(os.path.abspath(__file__)))


def engine(raw, w, dtype, **kw):
    from libtbvcoll_b200.engine.engine import Engine
    from libtbvcoll_b200.models.config import parse_lugizen_config
    kw = {"max_batch": 4, "max_seq_len": 512, "prefill_chunk": 256, **kw}
    return Engine(parse_lugizen_config(raw), device="cuda:0", source=cases.Source(w), dtype=dtype, **kw)


_cache = {}


def model(name):
    """(config, weights, {sequence: tokens}, {sequence: Expected}) of a case, computed once."""
    if name not in _cache:
        raw = cases.CASES[name]()
        w = cases.tensors(raw)
        seqs = {k: cases.tokens(raw, n, seed=n) for k, n in (("long", 210), ("mid", 77), ("short", 19), ("one", 1))}
        _cache[name] = raw, w, seqs, {k: Expected.of(oracle, raw, w, t) for k, t in seqs.items()}
    return _cache[name]


@pytest.mark.parametrize("dtype", [F32, BF])
@pytest.mark.parametrize("name", sorted(cases.CASES))
def test_whole_portions_and_single_tokens(name, dtype):
    raw, w, seqs, want = model(name)
    eng = engine(raw, w, dtype)
    for k, t in seqs.items():
        want[k].check(feed(eng, k, t, [len(t)]), dtype)
    t = seqs["long"]
    for portions in ([2] * 105, [3, 13, 15, 1, 16, 17, 31, 33, 64, 17], [1, 33, 2, 100, 1, 1, 72], [63, 65, 82]):
        want["long"].check(feed(eng, "p", t, portions), dtype)
    want["mid"].check(feed(eng, "d", seqs["mid"], [1] * 77), dtype)


@pytest.mark.parametrize("dtype", [F32, BF])
@pytest.mark.parametrize("name", ["odd", "wide"])
def test_stream_after_every_layer(name, dtype):
    from libtbvcoll_b200.engine.batch import Portion
    raw, w, seqs, _ = model(name)
    t, want, got = seqs["mid"], [], []
    oracle.forward(raw, w, t, collect=want)
    eng = engine(raw, w, dtype)
    r = eng.requests.extend("a", len(t))
    eng.bm.sync_to_device()
    eng.model.forward_batch(eng.batch_of([Portion(r.row, 0, t)]), on_layer=lambda i, x: got.append(x.cpu()))
    assert len(got) == len(want)
    for g, x in zip(got, want):
        assert float((g - x).norm() / x.norm()) < (2e-2 if dtype is BF else 5e-6)


@pytest.mark.parametrize("dtype", [F32, BF])
@pytest.mark.parametrize("name", ["odd", "wide"])
def test_mixed_batches_rows_pages_and_slots_used_again(name, dtype):
    """Random schedules of unequal requests; the pool is just large enough for what is live."""
    raw, w, seqs, want = model(name)
    eng = engine(raw, w, dtype, max_batch=3, max_seq_len=224, max_cache_tokens=224 + 80 + 64, prefill_chunk=150)
    rng = random.Random(5)
    todo = [(k, i) for i in range(3) for k in ("mid", "short", "one", "short")] + [("long", 0), ("long", 1)]
    rng.shuffle(todo)
    random_schedule(eng, rng, seqs, want, raw["vocab"], dtype, todo, 290)


@pytest.mark.parametrize("dtype", [F32, BF])
def test_a_batch_gives_what_each_request_gives_alone(dtype):
    raw, w, seqs, want = model("plain")
    eng = engine(raw, w, dtype)
    alone = {k: eng.step([(k, t, range(len(t)))], end=[k]) for k, t in seqs.items()}
    ks = ["mid", "one", "long", "short"]
    both = eng.step([(k, seqs[k], range(len(seqs[k]))) for k in ks], end=ks)         # longer than a pass: cut inside "long"
    at = 0
    for k in ks:
        n = len(seqs[k])
        Expected(alone[k].cpu(), want[k].limits).check(both[at: at + n], dtype)
        at += n


def test_a_long_prompt():
    """Many chunks of the recurrences, contexts much longer than the windows, whole, in portions and beside others."""
    raw, w, seqs, want = model("plain")
    t = cases.tokens(raw, 1100, seed=4)
    e = Expected.of(oracle, raw, w, t)
    eng = engine(raw, w, BF, max_seq_len=1200, prefill_chunk=2048)
    e.check(feed(eng, 0, t, [1100]), BF)
    e.check(feed(eng, 0, t, [7, 700, 1, 392]), BF)
    got = eng.step([("s", seqs["short"], [18]), ("l", t, [1099, 600]), ("m", seqs["mid"], [76])], end=["s", "l", "m"])
    Expected.stack([(want["short"], 18), (e, 1099), (e, 600), (want["mid"], 76)]).check(got, BF)


def changed(raw, w, toks, at, by=1):
    """The sequence with another token at ``at``, and by how much its logits differ from the first one's, position by position."""
    other = list(toks)
    other[at] = (other[at] + by) % raw["vocab"]
    a, b = Expected.of(oracle, raw, w, toks), Expected.of(oracle, raw, w, other)
    return other, a, b, (a.logits - b.logits).std(1) / a.logits.std()


@pytest.mark.parametrize("size", [40, 64, 17])
def test_a_token_at_the_edge_of_the_window(size):
    """One latent layer, made to look sharply at single keys: positions that still see a changed token differ, those just outside do not, in prompts and in
    decoding, and exactly where the oracle says."""
    raw = cases.config([cases.latent(3, 48, 8, 32, 60, 60, size, scale=0.6)], 80, 150, taps=1)
    w, toks, at = cases.tensors(raw), [9 if t in (7, 8) else t for t in cases.tokens(raw, 260, seed=9)], 100
    last = at + size - 1
    toks[at], toks[last], toks[last + 1] = 7, 8, 8                                     # the query of token 8 is the key of token 7: these positions look for it
    w["embed"][8] = w["embed"][7].roll(40)
    w["l0.canon1"].zero_()
    w["l0.mix.dq"], w["l0.mix.dq.norm"] = w["l0.mix.dkv"][:60].roll(40, 1).contiguous(), w["l0.mix.dkv.norm"]
    w["l0.mix.uq"].view(3, 56, 60)[:, :48] = w["l0.mix.uk"].view(3, 48, 60)
    w["l0.mix.uq"].view(3, 56, 60)[:, 48:] = 0
    other, a, b, diff = changed(raw, w, toks, at, by=30)
    assert float(diff[last]) > 0.05 and float(diff[last + 1:].max()) == 0.0
    for dtype in (F32, BF):
        eng = engine(raw, w, dtype)
        for portions in ([260], [at + 1] + [1] * (260 - at - 1), [3, 60, 2, 35, 39, 1, 1, 1, 118]):
            ga, gb = feed(eng, 0, toks, portions), feed(eng, 0, other, portions)
            a.check(ga, dtype)
            b.check(gb, dtype)
            assert torch.equal(ga[last + 1:], gb[last + 1:]) and not torch.equal(ga[last], gb[last])


def test_a_far_key_among_hundreds():
    """One attention layer whose last query is the key of an early token, all others having little weight."""
    raw = cases.config([cases.attention(4, 2, 48, 32, 8, scale=0.5)], 80, 150, taps=1)
    w, toks, at = cases.tensors(raw), [9 if t == 7 else t for t in cases.tokens(raw, 700, seed=3)], 5
    toks[at], toks[-1] = 7, 8
    w["embed"][8] = w["embed"][7].roll(40)
    w["l0.canon1"].zero_()
    w["l0.mix.k"] = w["l0.mix.q"].view(2, 2, 48, 80)[:, 0].reshape(96, 80).roll(40, 1).contiguous()
    w["l0.mix.temp"].fill_(1.0)
    other, a, b, diff = changed(raw, w, toks, at, by=30)
    assert float(diff[-1]) > 0.3
    for dtype in (F32, BF):
        eng = engine(raw, w, dtype, max_seq_len=720, prefill_chunk=1024)
        for portions in ([700], [5, 40, 1, 200, 83, 340] + [1] * 31):
            a.check(feed(eng, 0, toks, portions), dtype)
            b.check(feed(eng, 0, other, portions), dtype)


def test_a_far_token_shows_through_the_state():
    """A recurrence that hardly forgets carries an early token to the end of a long prompt and through decoding: the last position asks for what the token left, and
    no other token has a key."""
    raw = cases.config([cases.delta(2, 2, 32, 32, 3, cases.dense(48))], 64, 120, taps=2)
    w, toks = cases.tensors(raw), [9 if t in (5, 6) else t for t in cases.tokens(raw, 700, seed=9)]
    toks[3], toks[-1] = 5, 5
    w["embed"][:, 0] = 0
    w["embed"][5, 0], w["embed"][6, 0] = 1.5, -1.5
    w["l0.canon1"].zero_()
    for s in ("q", "k"):
        w[f"l0.mix.{s}"] = torch.zeros(64, 64, dtype=BF)
        w[f"l0.mix.{s}"][:, 0] = torch.randn(64, generator=torch.Generator().manual_seed(1)).to(BF)
        w[f"l0.mix.{s}.conv"] = torch.tensor([0.0, 0.0, 1.0], dtype=BF).repeat(64, 1)
    w["l0.mix.A_log"].fill_(-1.0)
    w["l0.mix.dt_bias"].fill_(-9.0)
    w["l0.mix.a2"].mul_(0.1)
    other, a, b, diff = changed(raw, w, toks, 3)
    assert float(diff[-1]) > 0.05 and float(diff[10:-1].max()) == 0.0
    for dtype in (F32, BF):
        eng = engine(raw, w, dtype, max_seq_len=720, prefill_chunk=1024)
        for portions in ([700], [5, 40, 1, 200, 83, 340] + [1] * 31):
            a.check(feed(eng, 0, toks, portions), dtype)
            b.check(feed(eng, 0, other, portions), dtype)


def test_long_decoding_through_the_captured_step():
    """300 tokens decoded one by one after a short prompt: the graph-captured serving loop, the device loop and the eager loop agree, and in
    fp32 every token is the oracle's choice (where the oracle is not undecided)."""
    raw, w, seqs, _ = model("odd")
    prompts = [seqs["short"], seqs["mid"], seqs["one"]]
    eng = engine(raw, w, F32)
    outs = eng.generate(prompts, 300)
    for p, o in zip(prompts, outs):
        full = oracle.forward(raw, w, p + o[:-1])
        top = full.topk(2, dim=-1)
        for i, t in enumerate(o):
            v = top.values[len(p) - 1 + i]
            assert t == int(top.indices[len(p) - 1 + i, 0]) or float(v[0] - v[1]) < 1e-3
    for loop, graph in (("host", False), ("device", True), ("device", False)):
        assert eng.generate(prompts, 300, loop=loop, use_graph=graph) == outs
    assert eng.generate(prompts, 300) == outs                                          # captured before: state starts afresh
    for name in ("odd", "wide", "large"):
        raw, w, seqs, _ = model(name)
        prompts = [seqs["short"], seqs["mid"], seqs["one"]]
        half = engine(raw, w, BF)
        a = half.generate(prompts, 120)
        assert a == half.generate(prompts, 120, loop="device") == half.generate(prompts, 120, use_graph=False)


def test_generation_through_the_scheduler():
    """More prompts than rows, a pool that cannot hold them all: the scheduler's mixed steps give what static batches give."""
    raw, w, seqs, _ = model("wide")
    prompts = [cases.tokens(raw, n, seed=100 + n) for n in (60, 3, 17, 90, 1, 33, 45)]
    eng = engine(raw, w, F32, max_batch=3, max_seq_len=128, max_cache_tokens=256, prefill_chunk=40)
    outs = eng.generate(prompts, 12)                                                   # 7 prompts > 3 rows
    alone = engine(raw, w, F32, max_batch=1, max_seq_len=128)
    assert outs == [alone.generate([p], 12)[0] for p in prompts]
    stop = outs[0][4]
    cut = eng.generate(prompts, 12, eos_id=stop)
    assert cut == [o[: o.index(stop) + 1] if stop in o else o for o in outs]


def test_capture_leaves_no_trace_in_the_state():
    raw, w, seqs, _ = model("odd")
    a = engine(raw, w, F32, max_batch=2)
    first = a.prefill([seqs["short"], seqs["mid"]], 8)
    kept = [s for s in a.model.state + a.model.conv + a.model.past if s is not None]
    before = [s.clone() for s in kept]
    a._load_decode_inputs(2, first, [len(seqs["short"]), len(seqs["mid"])])
    a.capture(2, 1, True)
    torch.cuda.synchronize()
    for s, b in zip(kept, before):
        assert torch.equal(s[1:], b[1:])


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_trace_replay(tmp_path, dtype):
    raw, w, seqs, want = model("plain")
    cases.write_checkpoint(str(tmp_path), raw, w)
    m, s = seqs["mid"], seqs["short"]
    steps = [{"step": 0, "entries": [{"id": "a", "tokens": m[:40], "want": [0, 39]}], "end": []},
             {"step": 1, "entries": [{"id": "b", "tokens": s[:2], "want": []}, {"id": "a", "tokens": m[40:41], "want": []}], "end": []},
             {"step": 2, "entries": [{"id": "a", "tokens": m[41:], "want": [35, 0]}, {"id": "b", "tokens": s[2:], "want": [16]}], "end": ["a"]},
             {"step": 3, "entries": [{"id": "a", "tokens": s, "want": [18]}], "end": ["a", "b"]}]
    r = subprocess.run([os.path.join(ROOT, "bin", "trace_run"), "--model", str(tmp_path), "--dtype", dtype, "--out", str(tmp_path), "--max-tokens", "128"],
                       input="".join(json.dumps(x) + "\n" for x in steps), capture_output=True, text=True, timeout=600, env=dict(os.environ, HOME=str(tmp_path)))
    assert r.returncode == 0, r.stderr[-2000:]
    assert [ln for ln in r.stdout.splitlines() if ln.startswith("done")] == [f"done {i}" for i in range(4)]
    assert not os.path.exists(tmp_path / "1.f32")
    read = lambda i: torch.from_numpy(np.fromfile(tmp_path / f"{i}.f32", dtype="<f4").reshape(-1, raw["vocab"]).copy())
    dt = getattr(torch, dtype)
    want["mid"][[0, 39]].check(read(0), dt)
    Expected.stack([(want["mid"], 76), (want["mid"], 41), (want["short"], 18)]).check(read(2), dt)
    want["short"][[18]].check(read(3), dt)


def test_generate_command_line(tmp_path):
    raw, w, seqs, _ = model("plain")
    cases.write_checkpoint(str(tmp_path), raw, w)
    r = subprocess.run([sys.executable, "-m", "libtbvcoll_b200.generate", "--model", str(tmp_path), "--dtype", "float32", "--new", "6",
                        "--prompt", ",".join(map(str, seqs["short"])), "--prompt", "3"], capture_output=True, text=True, timeout=600, cwd=ROOT)
    assert r.returncode == 0, r.stderr[-2000:]
    rows = [json.loads(ln) for ln in r.stdout.splitlines() if ln.startswith("{")]
    assert [len(x["tokens"]) for x in rows] == [6, 6]
    assert rows[0]["tokens"] == engine(raw, w, F32).generate([seqs["short"], [3]], 6)[0]
