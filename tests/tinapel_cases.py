"""Small Tinapel configurations and random checkpoints for the tests (dictionaries as ``config.json`` holds them, tensors under the checkpoint's
names, bf16 values).

A choice of experts that hangs on the last digits would make any comparison a matter of luck.  So every mixture of experts reads directions
of the residual stream that nothing but the embedding writes to: per token ``top`` of its experts are marked +``MARK`` there and the others -MARK,
out-projections and loop steps are orthogonal to those directions, and the router undoes the norm's weights."""
import torch
from nubosun_cases import Source, tokens, write_checkpoint  # noqa: F401  (the same for every design)

MARK = 3.0


def moe(experts, top, ff, scale=1.0, shared=None):
    return {"kind": "moe", "router": {"experts": experts, "top": top, "scale": scale}, "expert": {"ff": ff}, "shared": shared and {"ff": shared}}


def gla(heads, dim, vdim, tau, mlp=None):
    return {"type": "gla", "mixer": {"heads": heads, "dim": dim, "vdim": vdim, "tau": tau}, "mlp": mlp}


def wkv(heads, dim, mlp=None):
    return {"type": "wkv", "mixer": {"heads": heads, "dim": dim}, "mlp": mlp}


def attention(heads, kv_heads, dim, scale=None, softcap=20.0, coef=0.5, every=256, mlp=None):
    return {"type": "attention", "mixer": {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": dim, "scale": scale or dim ** -0.5, "softcap": softcap,
                                           "q_temp": {"coef": coef, "every": every}}, "mlp": mlp}


def config(layers, width, vocab, loop=None, scale=1.0, eps=1e-5):
    c = {"architecture": "Tinapel", "vocab": vocab, "width": width, "embedding": {"scale": scale}, "norm": {"eps": eps}, "layers": layers}
    if loop:
        c["loop"] = dict(zip(("start", "stop", "times"), loop))
    return c


CASES = {
    # nothing a multiple of anything; a loop over the middle three times; all sizes differ between layers of a kind
    "odd": lambda: config([attention(6, 2, 40, scale=0.31, softcap=4.0, coef=0.7, every=9, mlp=moe(5, 3, 28, 1.7, 36)), wkv(3, 24, moe(5, 3, 28, 0.6, 20)),
                           gla(5, 36, 20, 5.0, moe(7, 2, 44, 2.5, 52)), attention(3, 3, 20, softcap=9.0, coef=1.5, every=31), wkv(2, 50)],
                          100, 203, loop=(1, 3, 3), scale=0.8),
    # no loop, recurrent layers first, one expert that is always chosen, layers without feed-forward
    "plain": lambda: config([wkv(2, 64, moe(1, 1, 48, 0.7, 64)), gla(3, 32, 64, 16.0), attention(8, 4, 32, softcap=30.0, coef=0.2, every=50, mlp=moe(4, 1, 64, 1.0, 32))],
                            96, 130, scale=1.3, eps=1e-3),
    # heads of 128 and more channels, more than 16 query heads per key head, many experts, everything looped
    "wide": lambda: config([gla(2, 96, 144, 2.0, moe(24, 6, 32, 3.0, 80)), attention(20, 1, 128, softcap=12.0, coef=1.0, every=20, mlp=moe(10, 2, 100, 1.2, 48)),
                            wkv(1, 128)], 160, 300, loop=(0, 3, 2), eps=1e-6),
    # head sizes that take the general forms, a loop of one layer, no shared expert
    "large": lambda: config([gla(1, 200, 48, 8.0), attention(2, 1, 144, softcap=6.0, coef=0.4, every=64, mlp=moe(6, 2, 40, 1.0)), wkv(2, 160, moe(3, 2, 20, 1.0, 16))],
                            144, 97, loop=(1, 2, 4), scale=0.5),
}


def tensors(cfg, seed=0):
    g = torch.Generator().manual_seed(seed)
    n = lambda *s: torch.randn(*s, generator=g)
    u = lambda *s: torch.rand(*s, generator=g)
    W, V = cfg["width"], cfg["vocab"]
    lin = lambda o, i: n(o, i) / i ** 0.5
    mixtures = [(i, e["mlp"]["router"]) for i, e in enumerate(cfg["layers"]) if e["mlp"]]
    dirs = torch.linalg.qr(n(W, max(1, sum(r["experts"] for _, r in mixtures))))[0]          # [W, marks]
    away = lambda t: t - dirs @ (dirs.T @ t)                                                 # columns of t orthogonal to the marks
    embed, at, of_layer = away(n(W, V)).T, 0, {}
    for i, r in mixtures:
        marks = torch.full((V, r["experts"]), -MARK)
        marks.scatter_(1, u(V, r["experts"]).argsort(1)[:, : r["top"]], MARK)
        of_layer[i] = dirs[:, at: at + r["experts"]].T
        embed = embed + marks / cfg["embedding"]["scale"] @ of_layer[i]
        at += r["experts"]
    w = {"embed": embed, "final.norm": 0.2 * n(W)}
    if "loop" in cfg:
        w["loop.step"] = away(n(W, cfg["loop"]["times"])).T
    for i, e in enumerate(cfg["layers"]):
        p, m, f = f"l{i}.", e["mixer"], e["mlp"]
        x = p + "mix."
        w[p + "norm1"] = 0.2 * n(W)
        H, D = m["heads"], m["dim"]
        if e["type"] == "gla":
            K, v, R = H * D, H * m["vdim"], 6 + i
            w.update({x + "q": lin(K, W), x + "k": lin(K, W), x + "v": lin(v, W), x + "g": lin(v, W), x + "a1": lin(R, W), x + "a2": 2 * lin(K, R),
                      x + "a2.b": 2 * n(K), x + "norm": 1 + 0.2 * n(m["vdim"]), x + "o": away(lin(W, v))})
        elif e["type"] == "wkv":
            K, R = H * D, 5 + i
            w.update({x + "mu." + s: u(W) for s in "rkvgw"})
            w.update({x + s: lin(K, W) for s in "rkvg"})
            # memories of one token to hundreds
            w.update({x + "w1": lin(R, W), x + "w2": lin(K, R), x + "w0": -2.0 + 2.0 * n(K), x + "u": n(H, D), x + "norm": 1 + 0.2 * n(K), x + "o": away(lin(W, K))})
        else:
            G = m["kv_heads"]
            w.update({x + "q": lin(H * D, W), x + "k": lin(G * D, W), x + "q.norm": 1.5 + 0.3 * n(D), x + "k.norm": 1.5 + 0.3 * n(D), x + "o": away(lin(W, H * D))})
        if f:
            w[p + "norm2"] = 0.2 * n(W)
            y = p + "mlp."
            w[y + "router"] = 0.5 * of_layer[i] / (1.0 + w[p + "norm2"].to(torch.bfloat16).float())
            for k, ff in [(f"e{j}.", f["expert"]["ff"]) for j in range(f["router"]["experts"])] + ([("shared.", f["shared"]["ff"])] if f["shared"] else []):
                w.update({y + k + "gate": 1.5 * lin(ff, W), y + k + "up": 1.5 * lin(ff, W), y + k + "down": away(lin(W, ff))})
    return {k: t.to(torch.bfloat16).contiguous() for k, t in w.items()}
