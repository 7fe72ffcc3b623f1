"""Small Bobarax configurations and random checkpoints for the tests (dictionaries as ``config.json`` holds them, tensors under the checkpoint's
names, bf16 values, tables int32)."""
import torch
from nubosun_cases import Source, tokens, write_checkpoint  # noqa: F401  (the same for every design)


def dense(ff):
    return {"kind": "dense", "ff": ff}


def moe(experts, top, ff, limit):
    return {"kind": "moe", "router": {"experts": experts, "top": top}, "expert": {"ff": ff, "limit": limit}}


def lightning(decay, dim, vdim, mlp=None):
    return {"type": "lightning", "mixer": {"heads": len(decay), "dim": dim, "vdim": vdim, "decay": decay}, "mlp": mlp}


def chunked(heads, kv_heads, dim, vdim, size, scale=None, softcap=20.0, mlp=None):
    return {"type": "attention", "mixer": {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "scale": scale or dim ** -0.5, "mask": {"size": size},
                                           "softcap": softcap}, "mlp": mlp}


def windowed(heads, kv_heads, dim, vdim, size, rot, base=1e4, scale=None, kv_from=None, mlp=None):
    m = {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "scale": scale or dim ** -0.5, "mask": {"size": size}, "rot": {"base": base, "dims": rot}}
    if kv_from is not None:
        m["kv_from"] = kv_from
    return {"type": "attention_2", "mixer": m, "mlp": mlp}


def config(layers, width, vocab, mult=0.6, logit_scale=0.4, eps=1e-5):
    return {"architecture": "Bobarax", "vocab": vocab, "width": width, "norm": {"eps": eps}, "residual_mult": mult, "logit_scale": logit_scale, "layers": layers}


CASES = {
    # nothing a multiple of anything, sizes differ between layers of a kind, keys and values of a layer far before
    "odd": lambda: config([windowed(6, 2, 40, 24, 9, 12, base=300.0, scale=0.31, mlp=moe(5, 3, 28, 0.8)), lightning([1.0, 0.55, 0.97], 24, 36, dense(70)),
                           chunked(4, 4, 20, 44, 13, softcap=3.0), windowed(6, 2, 40, 24, 33, 12, base=300.0, scale=0.2, kv_from=0, mlp=moe(7, 2, 44, 1.7)),
                           lightning([0.9, 0.3], 50, 20)], 100, 203),
    # multipliers of one, one expert per token, all dimensions turned, a window and chunks of one page
    "plain": lambda: config([lightning([0.995, 0.8], 64, 64, moe(4, 1, 64, 7.0)), windowed(8, 4, 32, 32, 50, 32, mlp=dense(96)), chunked(5, 1, 32, 32, 16, mlp=dense(48))],
                            96, 130, mult=1.0, logit_scale=1.0, eps=1e-3),
    # heads of 128 channels, more than 16 query heads per key head, value blocks of more than 128 columns, many experts, windows longer than some sequences
    "wide": lambda: config([lightning([0.999, 0.6], 96, 144, dense(80)), windowed(20, 1, 128, 112, 140, 64, base=5e5, mlp=moe(24, 6, 32, 2.0)),
                            chunked(3, 3, 112, 128, 100, softcap=None, mlp=moe(10, 2, 100, 0.5)), windowed(20, 1, 128, 112, 31, 64, base=5e5, kv_from=1)], 160, 300, mult=0.3, eps=1e-6),
    # head sizes that take the general forms, windows of one and two tokens
    "large": lambda: config([chunked(2, 1, 144, 160, 37, softcap=6.0, mlp=dense(40)), lightning([0.98], 200, 48, moe(3, 3, 20, 1.0)), windowed(4, 2, 160, 272, 70, 160),
                             windowed(2, 2, 16, 16, 1, 2), windowed(4, 2, 160, 272, 2, 160, kv_from=2, mlp=dense(20))], 144, 97, mult=0.8, logit_scale=2.0),
}


def tensors(cfg, seed=0):
    g = torch.Generator().manual_seed(seed)
    n = lambda *s: torch.randn(*s, generator=g)
    W = cfg["width"]
    lin = lambda o, i: n(o, i) / i ** 0.5
    w = {"embed": n(cfg["vocab"], W), "final.norm": 0.2 * n(W)}
    for i, e in enumerate(cfg["layers"]):
        p, m, f = f"l{i}.", e["mixer"], e["mlp"]
        x, y = p + "mix.", p + "mlp."
        w.update({p + k: 0.2 * n(W) for k in (("norm1", "norm1b", "norm2", "norm2b") if f else ("norm1", "norm1b"))})
        K, V = m["heads"] * m["dim"], m["heads"] * m["vdim"]
        w.update({x + "q": lin(K, W), x + "o": lin(W, V)})
        if e["type"] == "lightning":
            w.update({x + "k": lin(K, W), x + "v": lin(V, W), x + "g": lin(V, W), x + "norm": 1 + 0.2 * n(V)})
        else:
            w[x + "q.norm"] = 1.5 + 0.3 * n(K)
            if m.get("kv_from") is None:
                kd, kv = m["kv_heads"] * m["dim"], m["kv_heads"] * m["vdim"]
                w.update({x + "k": lin(kd, W), x + "v": lin(kv, W), x + "k.norm": 1.5 + 0.3 * n(kd)})
            if e["type"] == "attention_2":
                w[x + "g"] = lin(V, W)
        if f:
            names, ff = ([""], f["ff"]) if f["kind"] == "dense" else ([f"e{j}." for j in range(f["router"]["experts"])], f["expert"]["ff"])
            for q in names:
                w.update({y + q + "gate": 1.5 * lin(ff, W), y + q + "up": 1.5 * lin(ff, W), y + q + "down": lin(W, ff)})
            if f["kind"] == "moe":
                w[y + "table"] = torch.rand(cfg["vocab"], f["router"]["experts"], generator=g).argsort(1)[:, : f["router"]["top"]].to(torch.int32)
    return {k: (t if k.endswith(".table") else t.to(torch.bfloat16)).contiguous() for k, t in w.items()}
