"""Plain statement of the Tinapel decoder, used only as the oracle of its tests.

One function per mechanism, written for whole sequences with ordinary loops and matrix products, in float32 (or float64 on request), no
cache, no state hand-over, no batching, nothing shared with the product code.  ``w`` maps checkpoint tensor names to tensors and ``cfg``
is the parsed ``config.json`` dictionary.  ``r`` rounds what a 16-bit run may keep in 16 bits (inputs and results of matrix products, cached
rows); it is the identity unless the size of those roundings is wanted."""
from __future__ import annotations

import math

import torch


def exact(x):
    return x


def to_bf16(x):
    return x.to(torch.bfloat16).to(x.dtype)


def rms(x, eps):
    return x / torch.sqrt((x * x).mean(-1, keepdim=True) + eps)


def sigmoid(z):
    return 1.0 / (1.0 + torch.exp(-z))


def silu(z):
    return z * sigmoid(z)


def position_vector(T, width, dtype):
    """[T, width]: columns 2i and 2i+1 hold sine and cosine of t / 10000^(2i / width)."""
    out = torch.zeros(T, width, dtype=torch.float64)
    for c in range(width):
        a = torch.arange(T, dtype=torch.float64) * 10000.0 ** (-2.0 * (c // 2) / width)
        out[:, c] = torch.sin(a) if c % 2 == 0 else torch.cos(a)
    return out.to(dtype)


def embed(tokens, table, scale):
    x = table[torch.as_tensor(tokens)] * scale
    return x + position_vector(x.shape[0], x.shape[1], x.dtype)


def gated_linear_attention(q, k, v, alpha):
    """q, k, alpha [T, H, D], v [T, H, V] -> [T, H, V]: S_t = alpha_t (rows) S_{t-1} + k_t v_t^T, read by q_t after the update."""
    T, H, D = q.shape
    S = torch.zeros(H, D, v.shape[2], dtype=q.dtype)
    out = torch.zeros_like(v)
    for t in range(T):
        S = alpha[t][:, :, None] * S + k[t][:, :, None] * v[t][:, None, :]
        out[t] = (S * q[t][:, :, None]).sum(1)
    return out


def gla_mixer(h, w, p, m, eps, r=exact):
    T, H, D, V = h.shape[0], m["heads"], m["dim"], m["vdim"]
    h = r(h)
    q = r(h @ w[p + "q"].T).view(T, H, D) / D ** 0.5
    k = r(h @ w[p + "k"].T).view(T, H, D)
    v = r(h @ w[p + "v"].T).view(T, H, V)
    g = r(h @ w[p + "g"].T)
    z = (r(h @ w[p + "a1"].T) @ w[p + "a2"].T + w[p + "a2.b"]).view(T, H, D)
    o = gated_linear_attention(q, k, v, sigmoid(z) ** (1.0 / m["tau"]))
    o = (rms(o, eps) * w[p + "norm"]).reshape(T, H * V)
    return r(o * silu(g)) @ w[p + "o"].T


def token_shift(h, mu):
    """Row t moves towards row t - 1 (zeros before the first) by mu, channel by channel."""
    prev = torch.zeros_like(h)
    prev[1:] = h[:-1]
    return h + (prev - h) * mu


def wkv(rr, k, v, decay, u):
    """rr, k, v, decay [T, H, D], u [H, D] -> [T, H, D]: the current token is read through u, the state takes it afterwards."""
    T, H, D = rr.shape
    S = torch.zeros(H, D, D, dtype=rr.dtype)
    out = torch.zeros_like(v)
    for t in range(T):
        kv = k[t][:, :, None] * v[t][:, None, :]
        out[t] = ((S + u[:, :, None] * kv) * rr[t][:, :, None]).sum(1)
        S = decay[t][:, :, None] * S + kv
    return out


def wkv_mixer(h, w, p, m, eps, r=exact):
    T, H, D = h.shape[0], m["heads"], m["dim"]
    mix = {s: r(token_shift(h, w[p + "mu." + s])) for s in "rkvgw"}
    rr, k, v = (r(mix[s] @ w[p + s].T).view(T, H, D) for s in "rkv")
    g = silu(r(mix["g"] @ w[p + "g"].T))
    z = r(torch.tanh(mix["w"] @ w[p + "w1"].T)) @ w[p + "w2"].T + w[p + "w0"]
    o = wkv(rr, k, v, torch.exp(-torch.exp(z)).view(T, H, D), w[p + "u"])
    return r(rms(o, eps).reshape(T, H * D) * w[p + "norm"] * g) @ w[p + "o"].T


def query_temperature(T, coef, every, dtype):
    return torch.tensor([1.0 + coef * math.log((t + 1) // every + 1) for t in range(T)], dtype=dtype)


def attention_mixer(h, w, p, m, eps, r=exact):
    T, H, G, D = h.shape[0], m["heads"], m["kv_heads"], m["dim"]
    h = r(h)
    q = r(h @ w[p + "q"].T).view(T, H, D)
    kv = r(h @ w[p + "k"].T).view(T, G, D)
    q = rms(q, eps) * w[p + "q.norm"]
    if m.get("q_temp"):
        q = q * query_temperature(T, m["q_temp"]["coef"], m["q_temp"]["every"], q.dtype)[:, None, None]
    q, k = r(q), r(rms(kv, eps) * w[p + "k.norm"])
    k, v = k.repeat_interleave(H // G, 1), kv.repeat_interleave(H // G, 1)
    s = torch.einsum("ihd,jhd->hij", q, k) * m["scale"]
    cap = m.get("softcap")
    if cap:
        s = cap * torch.tanh(s / cap)
    s = s.masked_fill(torch.ones(T, T, dtype=torch.bool).triu(1)[None], float("-inf"))
    o = r(torch.einsum("hij,jhd->ihd", r(torch.softmax(s, -1)), v))
    return o.reshape(T, H * D) @ w[p + "o"].T


def gated_mlp(h, w, p, r=exact):
    return r(silu(h @ w[p + "gate"].T) * (h @ w[p + "up"].T)) @ w[p + "down"].T


def route(z, top, scale):
    """z [T, E] -> weights [T, E], zero but for the ``top`` largest of each row."""
    s = torch.softmax(z, -1)
    out = torch.zeros_like(s)
    for t in range(z.shape[0]):
        idx = sorted(range(z.shape[1]), key=lambda e: (-float(s[t, e]), e))[:top]
        chosen = s[t, idx]
        out[t, idx] = chosen / (chosen.sum() + 1e-20) * scale
    return out


def moe(h, w, p, m, r=exact):
    h = r(h)
    weights = route(h @ w[p + "router"].T, m["router"]["top"], m["router"]["scale"])
    y = gated_mlp(h, w, p + "shared.", r) if m.get("shared") else torch.zeros_like(h)
    for e in range(m["router"]["experts"]):
        rows = torch.nonzero(weights[:, e])[:, 0]
        if len(rows):
            y[rows] = y[rows] + weights[rows, e][:, None] * gated_mlp(h[rows], w, f"{p}e{e}.", r)
    return y


MIXERS = {"gla": gla_mixer, "wkv": wkv_mixer, "attention": attention_mixer}


def layer(x, cfg, w, i, r=exact):
    lay, p, eps = cfg["layers"][i], f"l{i}.", cfg["norm"]["eps"]
    y = MIXERS[lay["type"]](rms(x, eps) * (1.0 + w[p + "norm1"]), w, p + "mix.", lay["mixer"], eps, r)
    if lay["mlp"] is not None:
        y = y + moe(rms(x, eps) * (1.0 + w[p + "norm2"]), w, p + "mlp.", lay["mlp"], r)
    return x + y


def passes(cfg):
    """(layer, number of the loop's pass that begins right before it, or None) in the order of execution."""
    n, lp = len(cfg["layers"]), cfg.get("loop")
    if not lp:
        return [(i, None) for i in range(n)]
    a, b = lp["start"], lp["stop"]
    out = [(i, None) for i in range(a)]
    for t in range(lp["times"]):
        out += [(i, t if i == a else None) for i in range(a, b)]
    return out + [(i, None) for i in range(b, n)]


def forward(cfg, w, tokens, dtype=torch.float32, collect=None, r=exact):
    """Logits [T, vocab] of one sequence; ``collect`` (a list) receives the residual stream after every layer run."""
    w = {k: v.to(dtype) for k, v in w.items()}
    eps = cfg["norm"]["eps"]
    x0 = x = embed(tokens, w["embed"], cfg["embedding"]["scale"])
    for i, t in passes(cfg):
        if t is not None:
            if t > 0:
                x = x + x0
            x = x + w["loop.step"][t]
        x = layer(x, cfg, w, i, r)
        if collect is not None:
            collect.append(x)
    return r(rms(x, eps) * (1.0 + w["final.norm"])) @ w["embed"].T
