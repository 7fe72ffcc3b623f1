"""Plain statement of the Nubosun decoder, used only as the oracle of its tests.

One function per mechanism, written for whole sequences with ordinary loops and matrix products, in float32 (or float64
on request), no cache, no state hand-over, no batching, nothing shared with the product code.  ``w`` maps checkpoint tensor names to tensors
and ``cfg`` is the parsed ``config.json`` dictionary.  ``r`` rounds what a 16-bit run may keep in 16 bits (inputs and results of matrix
products, short convolutions, cached rows); it is the identity unless the size of those roundings is wanted."""
from __future__ import annotations

import math

import torch


def exact(x):
    return x


def to_bf16(x):
    return x.to(torch.bfloat16).to(x.dtype)


def rms(x, eps):
    return x / torch.sqrt((x * x).mean(-1, keepdim=True) + eps)


def softplus(z):
    return torch.where(z > 30.0, z, torch.log1p(torch.exp(torch.clamp(z, max=30.0))))


def silu(z):
    return z / (1.0 + torch.exp(-z))


def causal_conv(x, taps, bias):
    """x [T, C]; taps [C, K], the last column weighs the current token; zeros before the first token."""
    T, C = x.shape
    K = taps.shape[1]
    y = torch.zeros_like(x) + bias
    for k in range(K):
        back = K - 1 - k
        if back < T:
            y[back:] = y[back:] + taps[:, k] * x[: T - back]
    return y


def selective_scan(u, dt, a_log, b, c, d):
    """u, dt [T, C]; a_log [C, N]; b, c [T, N]; d [C] -> [T, C]."""
    T, C = u.shape
    a = -torch.exp(a_log)
    s = torch.zeros(C, a_log.shape[1], dtype=u.dtype)
    out = torch.zeros_like(u)
    for t in range(T):
        s = torch.exp(dt[t][:, None] * a) * s + (dt[t] * u[t])[:, None] * b[t][None, :]
        out[t] = (s * c[t][None, :]).sum(1) + d * u[t]
    return out


def mamba_mixer(h, w, p, m, r=exact):
    inner, state, rank = m["inner"], m["state"], m["dt_rank"]
    xz = r(r(h) @ w[p + "in"].T)
    x, z = xz[:, :inner], xz[:, inner:]
    x = r(silu(causal_conv(x, w[p + "conv"], w[p + "conv.b"])))
    proj = x @ w[p + "x"].T
    dt = softplus(r(proj[:, :rank]) @ w[p + "dt"].T + w[p + "dt.b"])
    b, c = proj[:, rank:rank + state], proj[:, rank + state:]
    y = selective_scan(x, dt, w[p + "A_log"], b, c, w[p + "D"])
    return r(y * silu(z)) @ w[p + "o"].T


def rotary_frequencies(rot):
    """(frequency per pair, factor on cos and sin) of a rotation described by base / dims / optional YaRN scaling."""
    dims, base = rot["dims"], float(rot["base"])
    sc = rot.get("scaling")
    freq, factor = [], 1.0
    if sc:
        def at(turns):
            return dims * math.log(sc["original"] / (2 * math.pi * turns)) / (2 * math.log(base))
        lo, hi = max(math.floor(at(sc["fast"])), 0), min(math.ceil(at(sc["slow"])), dims - 1)
        factor = 0.1 * math.log(sc["factor"]) + 1.0
    for i in range(dims // 2):
        f = base ** (-2.0 * i / dims)
        if sc:
            r = min(max((i - lo) / max(hi - lo, 0.001), 0.0), 1.0)
            f = f / sc["factor"] * r + f * (1.0 - r)
        freq.append(f)
    return freq, factor


def rotate_pairs(x, positions, rot):
    """x [T, heads, D]: dimensions 2i and 2i+1 turn together by position * frequency_i; the rest pass."""
    freq, factor = rotary_frequencies(rot)
    out = x.clone()
    ang = positions.to(x.dtype)[:, None] * torch.tensor(freq, dtype=x.dtype)[None]
    cos, sin = (torch.cos(ang) * factor)[:, None], (torch.sin(ang) * factor)[:, None]
    n = rot["dims"]
    a, b = x[..., 0:n:2], x[..., 1:n:2]
    out[..., 0:n:2] = a * cos - b * sin
    out[..., 1:n:2] = b * cos + a * sin
    return out


def sink_softmax(scores, sink):
    """scores [H, T, T] masked with -inf; one extra exp(sink_h) in each denominator."""
    m = torch.maximum(scores.amax(-1, keepdim=True), sink[:, None, None])
    e = torch.exp(scores - m)
    return e / (e.sum(-1, keepdim=True) + torch.exp(sink[:, None, None] - m))


def latent_attention_mixer(h, w, p, m, eps, r=exact):
    T = h.shape[0]
    H, dim, rd, vd, R = m["heads"], m["dim"], m["rot_dim"], m["vdim"], m["kv_rank"]
    pos = torch.arange(T)
    q = r(r(h) @ w[p + "q"].T).view(T, H, dim + rd)
    kv = r(r(h) @ w[p + "dkv"].T)
    c = r(rms(kv[:, :R], eps) * w[p + "dkv.norm"])
    kr = r(rotate_pairs(kv[:, None, R:], pos, m["rot"])[:, 0])
    qr = r(rotate_pairs(q[..., dim:], pos, m["rot"]))
    k = r(c @ w[p + "uk"].T).view(T, H, dim)
    v = r(c @ w[p + "uv"].T).view(T, H, vd)
    s = (torch.einsum("ihd,jhd->hij", q[..., :dim], k) + torch.einsum("ihd,jd->hij", qr, kr)) * m["scale"]
    s = s.masked_fill(torch.ones(T, T, dtype=torch.bool).triu(1)[None], float("-inf"))
    o = r(torch.einsum("hij,jhd->ihd", r(sink_softmax(s, w[p + "sink"])), v))
    return o.reshape(T, H * vd) @ w[p + "o"].T


def clamped_glu_mlp(h, w, p, m, r=exact):
    lim, h = m["limit"], r(h)
    g = torch.clamp(h @ w[p + "gate"].T, max=lim)
    u = torch.clamp(h @ w[p + "up"].T, -lim, lim)
    return r(g / (1.0 + torch.exp(-1.702 * g)) * (u + 1.0)) @ w[p + "down"].T


def hyper_sublayer(xs, fn, gamma, scale, hin, hout, hmix, eps):
    """xs: list of streams [T, W].  One sublayer between the mixing of the streams."""
    n = len(xs)
    u = sum(hin[s] * xs[s] for s in range(n))
    y = fn(rms(u, eps) * gamma) * scale
    return [sum(hmix[s, t] * xs[s] for s in range(n)) + hout[t] * y for t in range(n)]


def layer_order(cfg):
    n = len(cfg["layers"])
    lp = cfg.get("loop")
    if not lp:
        return list(range(n))
    return list(range(lp["start"])) + list(range(lp["start"], lp["stop"])) * lp["times"] + list(range(lp["stop"], n))


def forward(cfg, w, tokens, dtype=torch.float32, collect=None, r=exact):
    """Logits [T, vocab] of one sequence; ``collect`` (a list) receives the summed streams after every layer run."""
    w = {k: v.to(dtype) for k, v in w.items()}
    eps = cfg["norm"]["eps"]
    x = w["embed"][torch.as_tensor(tokens)] * cfg["embedding"]["scale"]
    xs = [x.clone() for _ in range(cfg["streams"])]
    for i in layer_order(cfg):
        lay, p = cfg["layers"][i], f"l{i}."
        m = lay["mixer"]
        if lay["type"] == "mamba1":
            fn = lambda h: mamba_mixer(h, w, p + "mix.", m, r)
        elif lay["type"] == "latent_attention":
            fn = lambda h: latent_attention_mixer(h, w, p + "mix.", m, eps, r)
        else:
            raise ValueError(lay["type"])
        xs = hyper_sublayer(xs, fn, w[p + "norm1"], w[p + "ls1"], w[p + "hc1.in"], w[p + "hc1.out"], w[p + "hc1.mix"], eps)
        if lay["mlp"] is not None:
            fn = lambda h: clamped_glu_mlp(h, w, p + "mlp.", lay["mlp"], r)
            xs = hyper_sublayer(xs, fn, w[p + "norm2"], w[p + "ls2"], w[p + "hc2.in"], w[p + "hc2.out"], w[p + "hc2.mix"], eps)
        if collect is not None:
            collect.append(sum(xs))
    logits = r(rms(sum(xs), eps) * w["final.norm"]) @ w["head"].T
    cap = cfg["logit_softcap"]
    return cap * torch.tanh(logits / cap)
