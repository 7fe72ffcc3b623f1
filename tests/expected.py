"""Logits of an oracle with a limit per position, and the requests fed to an engine that are held against them."""
import torch

BF, F32 = torch.bfloat16, torch.float32


class Expected:
    """Oracle logits with a limit per position: in bf16 three times the error that rounding to 16 bits alone causes there (never less than
    the median over the sequence), in fp32 a fixed one."""

    def __init__(self, logits, limits):
        self.logits, self.limits = logits, limits

    @staticmethod
    def of(oracle, raw, w, toks):
        logits = oracle.forward(raw, w, toks)
        e = Expected.error(oracle.forward(raw, w, toks, r=oracle.to_bf16), logits, logits)
        return Expected(logits, {BF: 3 * torch.maximum(e, e.median()), F32: torch.full_like(e, 2e-4)})

    @staticmethod
    def error(got, want, whole):
        """rms over the vocabulary of the mean-free difference, over the rms of the logits"""
        d = got.double().cpu() - want.double()
        d = d - d.mean(-1, keepdim=True)
        return d.pow(2).mean(-1).sqrt() / whole.double().std()

    def check(self, got, dtype):
        e = Expected.error(got, self.logits, self.logits) / self.limits[dtype]
        over = int((e > 1).sum())
        assert float(e.max()) < 1.5 and over <= max(1, len(e) // 50), (float(e.max()), int(e.argmax()), over)

    def __getitem__(self, rows):
        return Expected(self.logits[rows], {k: v[rows] for k, v in self.limits.items()})

    @staticmethod
    def stack(parts):
        """rows [(Expected, position), ..] of several sequences"""
        return Expected(torch.stack([e.logits[p] for e, p in parts]), {k: torch.stack([e.limits[k][p] for e, p in parts]) for k in (BF, F32)})


def feed(eng, key, toks, portions):
    """Runs one request alone in the given portions; logits of every position."""
    out, at = [], 0
    for n in portions:
        n = min(n, len(toks) - at)
        if n:
            out.append(eng.step([(key, toks[at: at + n], range(n))], end=[key] if at + n == len(toks) else []))
        at += n
    return torch.cat(out)


def random_schedule(eng, rng, seqs, want, vocab, dtype, todo, pool):
    """Unequal requests through mixed steps: portions beside single tokens, requests left out of steps, at most three live, ``pool`` tokens in
    all.  ``todo``: (sequence name, number) in order of admission; every returned row is checked."""
    live, at = [], {}
    while todo or live:
        while todo and len(live) < 3 and not (todo[0][0] == "long" and any(k == "long" for k, _ in live)) \
                and sum(len(seqs[k]) for k, _ in live + todo[:1]) <= pool:
            live.append(todo.pop(0))
        entries, end, rows = [], [], []
        for r in rng.sample(live, rng.randint(1, len(live))):
            t, a = seqs[r[0]], at.get(r, 0)
            n = min(len(t) - a, rng.choice([1, 1, 1, 2, 5, 16, 33, 70]))
            pick = sorted(rng.sample(range(n), rng.randint(0, n)))
            entries.append((r, t[a: a + n], pick))
            rows += [(r[0], a + p) for p in pick]
            at[r] = a + n
            if at[r] == len(t):
                end.append(r)
        got = eng.step(entries, end=end)
        live = [r for r in live if r not in end]
        assert got.shape == (len(rows), vocab)
        if rows:
            Expected.stack([(want[k], p) for k, p in rows]).check(got, dtype)
    assert len(eng.bm.free) == eng.bm.num_blocks - 1 and sorted(eng.requests.free_rows) == [0, 1, 2]
