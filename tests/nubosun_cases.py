"""Small Nubosun configurations and random checkpoints for the tests (dictionaries as ``config.json`` holds them, tensors under the
checkpoint's names, bf16 values)."""
import json
import os

import torch

YARN = {"factor": 4.0, "original": 64, "fast": 24.0, "slow": 1.5}


def mamba(inner, state, dt_rank, conv, ff=None, limit=1.5):
    return {"type": "mamba1", "mixer": {"inner": inner, "state": state, "dt_rank": dt_rank, "conv": conv},
            "mlp": None if ff is None else {"kind": "dense", "ff": ff, "limit": limit}}


def latent(heads, dim, rot_dim, vdim, kv_rank, base=1e4, scaling=None, scale=None, ff=None, limit=1.5):
    return {"type": "latent_attention",
            "mixer": {"heads": heads, "dim": dim, "rot_dim": rot_dim, "vdim": vdim, "kv_rank": kv_rank, "scale": scale or (dim + rot_dim) ** -0.5,
                      "rot": {"dims": rot_dim, "base": base, "scaling": scaling}},
            "mlp": None if ff is None else {"kind": "dense", "ff": ff, "limit": limit}}


def config(layers, width, vocab, streams=2, loop=None, scale=0.7, eps=1e-5, cap=20.0):
    c = {"architecture": "Nubosun", "vocab": vocab, "width": width, "streams": streams, "embedding": {"scale": scale}, "norm": {"eps": eps},
         "logit_softcap": cap, "layers": layers}
    if loop:
        c["loop"] = dict(zip(("start", "stop", "times"), loop))
    return c


CASES = {
    # nothing a multiple of anything; a loop over the middle; all sizes differ between layers of a kind
    "odd": lambda: config([latent(3, 24, 10, 36, 52, scaling=YARN, ff=70), mamba(88, 5, 3, 4), mamba(120, 12, 7, 2, ff=44),
                           latent(1, 40, 6, 20, 90, base=500.0)], 100, 203, streams=3, loop=(1, 3, 3)),
    # one stream, attention layers first, feed-forwards behind scans, no loop
    "plain": lambda: config([latent(5, 32, 16, 32, 64), mamba(96, 16, 8, 3, ff=96), latent(5, 32, 16, 32, 64, scaling=YARN)], 96, 130, streams=1,
                            scale=1.3, eps=1e-3, cap=5.0),
    # two head tiles, a state wider than a warp's lanes, four streams, everything looped
    "wide": lambda: config([mamba(160, 40, 20, 4, ff=100, limit=0.8), latent(18, 16, 32, 48, 144, scaling=YARN, ff=64)], 160, 300, streams=4,
                           loop=(0, 2, 2)),
    # only scans: one token of convolution memory, one state
    "scans": lambda: config([mamba(64, 1, 1, 2), mamba(48, 70, 5, 5), mamba(64, 130, 3, 1)], 64, 97, streams=2),
}


def tensors(cfg, seed=0):
    g = torch.Generator().manual_seed(seed)
    n = lambda *s: torch.randn(*s, generator=g)
    W, S, V = cfg["width"], cfg["streams"], cfg["vocab"]
    w = {"embed": n(V, W), "head": n(V, W) / W ** 0.5 * 2.0, "final.norm": 1 + 0.2 * n(W)}
    lin = lambda o, i: n(o, i) / i ** 0.5
    for i, e in enumerate(cfg["layers"]):
        p, m = f"l{i}.", e["mixer"]
        for q in (1, 2) if e["mlp"] else (1,):
            w[f"{p}norm{q}"], w[f"{p}ls{q}"] = 1 + 0.2 * n(W), 0.6 + 0.2 * n(W)
            w[f"{p}hc{q}.in"], w[f"{p}hc{q}.out"] = 1.0 / S + 0.3 * n(S), 1.0 + 0.3 * n(S)
            w[f"{p}hc{q}.mix"] = 0.8 * torch.eye(S) + 0.2 * n(S, S)
        p += "mix."
        if e["type"] == "mamba1":
            I, N, R = m["inner"], m["state"], m["dt_rank"]
            w.update({p + "in": lin(2 * I, W), p + "conv": n(I, m["conv"]) / m["conv"] ** 0.5, p + "conv.b": 0.3 * n(I), p + "x": lin(R + 2 * N, I),
                      p + "dt": lin(I, R), p + "dt.b": -2 + n(I), p + "A_log": torch.log(0.05 + 4 * torch.rand(I, N, generator=g)), p + "D": 1 + 0.3 * n(I),
                      p + "o": lin(W, I)})
        else:
            H, D, r, v, K = (m[k] for k in ("heads", "dim", "rot_dim", "vdim", "kv_rank"))
            w.update({p + "q": 1.5 * lin(H * (D + r), W), p + "dkv": lin(K + r, W), p + "dkv.norm": 1 + 0.2 * n(K), p + "uk": lin(H * D, K),
                      p + "uv": lin(H * v, K), p + "sink": n(H), p + "o": lin(W, H * v)})
        if e["mlp"]:
            f = e["mlp"]["ff"]
            p = f"l{i}.mlp."
            w.update({p + "gate": 1.5 * lin(f, W), p + "up": 1.5 * lin(f, W), p + "down": lin(W, f)})
    return {k: t.to(torch.bfloat16).contiguous() for k, t in w.items()}


class Source:
    """Weight source over a dictionary."""

    def __init__(self, w):
        self.w = w

    def names(self):
        return self.w.keys()

    def get(self, name):
        return self.w[name]


def write_checkpoint(path, cfg, w):
    from safetensors.torch import save_file
    with open(os.path.join(path, "config.json"), "w") as f:
        json.dump(cfg, f)
    save_file(w, os.path.join(path, "model.safetensors"))


def tokens(cfg, n, seed=1):
    return torch.randint(0, cfg["vocab"], (n,), generator=torch.Generator().manual_seed(seed)).tolist()
