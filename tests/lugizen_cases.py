"""Small Lugizen configurations and random checkpoints for the tests (dictionaries as ``config.json`` holds them, tensors under the checkpoint's
names, bf16 values)."""
import torch
from nubosun_cases import Source, tokens, write_checkpoint  # noqa: F401  (the same for every design)


def dense(ff):
    return {"kind": "dense", "ff": ff}


def moe(experts, top, ff):
    return {"kind": "moe", "router": {"experts": experts, "top": top}, "expert": {"ff": ff}}


def delta(heads, kv_heads, dim, vdim, conv, mlp=None):
    return {"type": "channel_delta", "mixer": {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "conv": conv}, "mlp": mlp}


def attention(heads, kv_heads, dim, vdim, rot, base=1e4, scale=None, v_mix=True, mlp=None):
    return {"type": "attention", "mixer": {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "rot": {"base": base, "dims": rot},
                                           "scale": scale or 1.2 * dim ** -0.5, "v_mix": v_mix}, "mlp": mlp}


def latent(heads, dim, rot_dim, vdim, kv_rank, q_rank, window, base=1e4, scale=None, mlp=None):
    return {"type": "latent_attention", "mixer": {"heads": heads, "dim": dim, "rot_dim": rot_dim, "vdim": vdim, "kv_rank": kv_rank, "q_rank": q_rank, "mask": {"size": window},
                                                  "rot": {"base": base, "dims": rot_dim}, "scale": scale or (dim + rot_dim) ** -0.5}, "mlp": mlp}


def config(layers, width, vocab, taps=4, eps=1e-5):
    return {"architecture": "Lugizen", "vocab": vocab, "width": width, "norm": {"eps": eps}, "canon": {"taps": taps}, "layers": layers}


CASES = {
    # nothing a multiple of anything, sizes differ between layers of a kind, values mixed with those of a layer far before (of other head sizes), key heads shared by
    # heads of the recurrence, layers without feed-forward
    "odd": lambda: config([attention(6, 2, 40, 24, 12, base=300.0, mlp=moe(5, 3, 28)), delta(4, 2, 24, 36, 3, dense(70)), latent(3, 20, 10, 44, 52, 36, 9, base=500.0),
                           attention(2, 2, 28, 24, 28, scale=0.3), latent(5, 36, 6, 20, 28, 60, 33, mlp=dense(50)), delta(3, 3, 50, 20, 5),
                           attention(4, 4, 20, 36, 4, v_mix=False, mlp=moe(7, 2, 44))], 100, 203),
    # recurrence first, one expert per token, all dimensions turned, a window of one page, two taps everywhere
    "plain": lambda: config([delta(2, 2, 64, 64, 2, moe(4, 1, 64)), latent(5, 32, 16, 32, 64, 96, 16, mlp=dense(96)), delta(2, 1, 32, 64, 2, dense(48)),
                             attention(8, 4, 32, 32, 32, mlp=moe(3, 3, 48))], 96, 130, taps=2, eps=1e-3),
    # heads of 128 channels, more than 16 query heads per key head, two head tiles over the latents, value blocks of more than 128 columns, many experts, windows
    # longer than some sequences
    "wide": lambda: config([delta(2, 2, 96, 144, 4, moe(24, 6, 32)), attention(20, 1, 128, 112, 64, base=5e5, mlp=dense(80)), latent(18, 16, 32, 48, 144, 112, 100, mlp=moe(10, 2, 100)),
                            delta(3, 1, 128, 32, 4), attention(6, 1, 64, 112, 10, mlp=dense(40))], 160, 300, taps=3, eps=1e-6),
    # head sizes that take the general forms, windows of one and two tokens, convolutions of one tap and of many
    "large": lambda: config([latent(2, 40, 8, 272, 80, 24, 70, mlp=dense(40)), delta(2, 1, 200, 48, 1, moe(3, 3, 20)), attention(2, 1, 144, 160, 140), latent(1, 16, 2, 16, 20, 20, 1),
                             attention(4, 1, 160, 160, 2, mlp=dense(20)), latent(3, 24, 12, 16, 600, 16, 2), delta(1, 1, 144, 272, 9)], 144, 97, taps=6),
}


MARK = 2.0


def tensors(cfg, seed=0):
    """The routers read directions of the embedding that nothing else writes, so that no choice of experts is close."""
    g = torch.Generator().manual_seed(seed)
    n = lambda *s: torch.randn(s, generator=g)
    u = lambda *s: torch.rand(*s, generator=g)
    W, V, taps = cfg["width"], cfg["vocab"], cfg["canon"]["taps"]
    lin = lambda o, i: n(o, i) / i ** 0.5
    mixtures = [(i, e["mlp"]["router"]) for i, e in enumerate(cfg["layers"]) if e["mlp"] and e["mlp"]["kind"] == "moe"]
    dirs = torch.linalg.qr(n(W, max(1, sum(r["experts"] for _, r in mixtures))))[0]          # [W, marks]
    away = lambda t: t - dirs @ (dirs.T @ t)                                                 # columns of t orthogonal to the marks
    embed, at, of_layer = away(n(W, V)).T, 0, {}
    for i, r in mixtures:
        marks = torch.full((V, r["experts"]), -MARK)
        marks.scatter_(1, u(V, r["experts"]).argsort(1)[:, : r["top"]], MARK * (0.5 + u(V, r["top"])))
        of_layer[i] = dirs[:, at: at + r["experts"]].T
        embed = embed + marks @ of_layer[i]
        at += r["experts"]
    w = {"embed": embed, "head": 2 * lin(V, W), "final.norm": 1 + 0.3 * n()}
    for i, e in enumerate(cfg["layers"]):
        p, m, f = f"l{i}.", e["mixer"], e["mlp"]
        x, y, H, D, v = p + "mix.", p + "mlp.", m["heads"], m["dim"], m["vdim"]
        w.update({p + "norm1": 1 + 0.3 * n(), p + "canon1": 0.5 * n(W, taps), x + "o": away(lin(W, H * v))})
        if e["type"] == "channel_delta":
            K, Ra, Rg = m["kv_heads"] * D, 6 + i, 21 - i
            for s, c in (("q", K), ("k", K), ("v", H * v)):
                w.update({x + s: 1.5 * lin(c, W), x + s + ".conv": n(c, m["conv"])})
            # memories of one token to hundreds
            w.update({x + "b": lin(H, W), x + "A_log": torch.log(0.02 + 4 * u(H) ** 3), x + "norm": 1 + 0.2 * n(v), x + "a1": lin(Ra, W), x + "a2": lin(H * D, Ra),
                      x + "dt_bias": -2.0 + 2.0 * n(H * D), x + "g1": lin(Rg, W), x + "g2": 2 * lin(H * v, Rg)})
        elif e["type"] == "attention":
            G = m["kv_heads"]
            w.update({x + "q": lin(H * D, W), x + "k": lin(G * D, W), x + "v": lin(G * v, W), x + "temp": 1.5 + 0.5 * n(H)})
            if m["v_mix"]:
                w[x + "vmix"] = 0.4 + 0.3 * n()
        else:
            R, Q, rot = m["kv_rank"], m["q_rank"], m["rot_dim"]
            w.update({x + "dq": lin(Q, W), x + "dq.norm": 1.5 + 0.3 * n(Q), x + "uq": 1.2 * lin(H * (D + rot), Q), x + "dkv": lin(R + rot, W), x + "dkv.norm": 1 + 0.2 * n(R),
                      x + "uk": lin(H * D, R), x + "uv": lin(H * v, R)})
        if f:
            w[p + "norm2"] = 1 + 0.3 * n()
            if f["kind"] == "dense":
                w.update({y + "up": lin(f["ff"], W), y + "down": away(lin(W, f["ff"]))})
            else:
                w[y + "router"] = of_layer[i]
                for j in range(f["router"]["experts"]):
                    k, ff = f"{y}e{j}.", f["expert"]["ff"]
                    w.update({k + "gate": 1.5 * lin(ff, W), k + "up": 1.5 * lin(ff, W), k + "down": away(lin(W, ff))})
    return {k: t.to(torch.bfloat16).contiguous() for k, t in w.items()}
