"""Plain statement of the Lugizen decoder, used only as the oracle of its tests.

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


def scalar_norm(x, g, eps):
    return rms(x, eps) * g


def sigmoid(z):
    return 1.0 / (1.0 + torch.exp(-z))


def silu(z):
    return z * sigmoid(z)


def gelu_tanh(z):
    return 0.5 * z * (1.0 + torch.tanh(math.sqrt(2.0 / math.pi) * (z + 0.044715 * z ** 3)))


def softplus(z):
    return torch.where(z > 0, z, torch.zeros_like(z)) + torch.log1p(torch.exp(-z.abs()))


def causal_conv(x, taps):
    """x [T, C], taps [C, K]: y_t = sum_j taps[:, j] x_{t - K + 1 + j}, zeros before the first token."""
    T, K = x.shape[0], taps.shape[1]
    y = torch.zeros_like(x)
    for t in range(T):
        for j in range(K):
            s = t - K + 1 + j
            if s >= 0:
                y[t] = y[t] + taps[:, j] * x[s]
    return y


# ---- gated delta rule with a decay per key channel --------------------------------------------------------------------------------
def unit(x):
    return x / torch.sqrt((x * x).sum(-1, keepdim=True) + 1e-6)


def delta_rule(q, k, v, beta, g):
    """q, k, g [T, H, D], v [T, H, V], beta [T, H] -> [T, H, V].  S decays, what it holds for k moves towards v by beta, then q reads it."""
    T, H, D = q.shape
    S = torch.zeros(H, D, v.shape[2], dtype=q.dtype)
    out = torch.zeros_like(v)
    for t in range(T):
        S = g[t][:, :, None] * S
        u = beta[t][:, None] * (v[t] - (S * k[t][:, :, None]).sum(1))
        S = S + k[t][:, :, None] * u[:, None, :]
        out[t] = (S * q[t][:, :, None]).sum(1)
    return out


def channel_delta_mixer(h, w, i, m, eps, first, r=exact):
    p, T, H, G, D, V = f"l{i}.mix.", h.shape[0], m["heads"], m["kv_heads"], m["dim"], m["vdim"]
    h, rep = r(h), m["heads"] // m["kv_heads"]
    q, k, v = (r(silu(causal_conv(r(h @ w[p + s].T), w[p + s + ".conv"]))).view(T, n, c) for s, n, c in (("q", G, D), ("k", G, D), ("v", H, V)))
    q, k = (unit(x).repeat_interleave(rep, 1) for x in (q, k))
    beta = sigmoid(r(h @ w[p + "b"].T))
    z = (r(h @ w[p + "a1"].T) @ w[p + "a2"].T + w[p + "dt_bias"]).view(T, H, D)
    g = torch.exp(-torch.exp(w[p + "A_log"])[None, :, None] * softplus(z))
    o = delta_rule(q * D ** -0.5, k, v, beta, g)
    gate = sigmoid(r(r(h @ w[p + "g1"].T) @ w[p + "g2"].T)).view(T, H, V)
    return r((rms(o, eps) * w[p + "norm"] * gate).reshape(T, H * V)) @ w[p + "o"].T


# ---- attention -------------------------------------------------------------------------------------------------------------------
def rotate_half(x, dims, base):
    """x [T, H, D]: dimensions i and i + dims / 2 of the first ``dims`` turned by position * base^(-2i / dims)."""
    out, half = x.clone(), dims // 2
    t = torch.arange(x.shape[0], dtype=torch.float64)
    for i in range(half):
        a = t * float(base) ** (-2.0 * i / dims)
        c, s = torch.cos(a).to(x.dtype)[:, None], torch.sin(a).to(x.dtype)[:, None]
        u, v = x[:, :, i], x[:, :, i + half]
        out[:, :, i], out[:, :, i + half] = u * c - v * s, v * c + u * s
    return out


def causal_mask(T):
    i, j = torch.arange(T)[:, None], torch.arange(T)[None]
    return j <= i


def window_mask(T, size):
    i, j = torch.arange(T)[:, None], torch.arange(T)[None]
    return (j <= i) & (i - j < size)


def softmax_attention(q, k, v, scale, visible, r=exact):
    """q [T, H, D], k [T, G, D], v [T, G, V], scale a number or one per head, visible [T, T] -> [T, H, V]."""
    rep = q.shape[1] // k.shape[1]
    k, v = k.repeat_interleave(rep, 1), v.repeat_interleave(rep, 1)
    s = torch.einsum("ihd,jhd->hij", q, k) * torch.as_tensor(scale, dtype=q.dtype).reshape(-1, 1, 1)
    s = s.masked_fill(~visible[None], float("-inf"))
    return torch.einsum("hij,jhd->ihd", r(torch.softmax(s, -1)), v)


def value_mix(v, v_first, lam):
    return (1.0 - lam) * v + lam * v_first


def attention_mixer(h, w, i, m, eps, first, r=exact):
    p, T, H, G, D, V = f"l{i}.mix.", h.shape[0], m["heads"], m["kv_heads"], m["dim"], m["vdim"]
    h = r(h)
    turn = lambda s, n: r(rms(rotate_half(r(h @ w[p + s].T).view(T, n, D), m["rot"]["dims"], m["rot"]["base"]), eps))
    v = r(h @ w[p + "v"].T).view(T, G, V)
    if m.get("v_mix"):
        if "v" in first:
            v = r(value_mix(v, first["v"], w[p + "vmix"]))
        else:
            first["v"] = v
    o = softmax_attention(turn("q", H), turn("k", G), v, m["scale"] * w[p + "temp"], causal_mask(T), r)
    return r(o.reshape(T, H * V)) @ w[p + "o"].T


def latent_attention_mixer(h, w, i, m, eps, first, r=exact):
    p, T, H, D, V, R, rot = f"l{i}.mix.", h.shape[0], m["heads"], m["dim"], m["vdim"], m["kv_rank"], m["rot_dim"]
    h = r(h)
    turn = lambda x: r(rotate_half(x, m["rot"]["dims"], m["rot"]["base"]))
    q = r(r(rms(r(h @ w[p + "dq"].T), eps) * w[p + "dq.norm"]) @ w[p + "uq"].T).view(T, H, D + rot)
    low = r(h @ w[p + "dkv"].T)
    c, kr = r(rms(low[:, :R], eps) * w[p + "dkv.norm"]), turn(low[:, None, R:])
    k = torch.cat((r(c @ w[p + "uk"].T).view(T, H, D), kr.expand(T, H, rot)), 2)
    q = torch.cat((q[:, :, :D], turn(q[:, :, D:])), 2)
    o = softmax_attention(q, k, r(c @ w[p + "uv"].T).view(T, H, V), m["scale"], window_mask(T, m["mask"]["size"]), r)
    return r(o.reshape(T, H * V)) @ w[p + "o"].T


# ---- feed-forward ------------------------------------------------------------------------------------------------------------------
def gelu_mlp(h, w, p, r=exact):
    return r(gelu_tanh(h @ w[p + "up"].T)) @ w[p + "down"].T


def expert(h, w, p, r=exact):
    return r(silu(h @ w[p + "gate"].T) * (h @ w[p + "up"].T)) @ w[p + "down"].T


def router_weights(logits, top):
    """[T, E] -> [T, E]: softmax over the ``top`` largest logits of a token, zero for the others."""
    out = torch.zeros_like(logits)
    for t in range(logits.shape[0]):
        best = torch.topk(logits[t], top).indices
        e = torch.exp(logits[t][best] - logits[t][best].max())
        out[t, best] = e / e.sum()
    return out


def moe(h, w, p, f, r=exact):
    y, weights = torch.zeros_like(h), router_weights(h @ w[p + "router"].T, f["router"]["top"])
    for e in range(f["router"]["experts"]):
        rows = torch.nonzero(weights[:, e])[:, 0]
        if len(rows):
            y[rows] = y[rows] + weights[rows, e][:, None] * r(expert(h[rows], w, f"{p}e{e}.", r))
    return y


def feed_forward(x, w, i, f, r=exact):
    return gelu_mlp(r(x), w, f"l{i}.mlp.", r) if f["kind"] == "dense" else moe(r(x), w, f"l{i}.mlp.", f, r)


MIXERS = {"channel_delta": channel_delta_mixer, "attention": attention_mixer, "latent_attention": latent_attention_mixer}


def layer(x, cfg, w, i, first, r=exact):
    lay, p, eps = cfg["layers"][i], f"l{i}.", cfg["norm"]["eps"]
    h = x + causal_conv(x, w[p + "canon1"])
    x = x + scalar_norm(MIXERS[lay["type"]](h, w, i, lay["mixer"], eps, first, r), w[p + "norm1"], eps)
    if lay["mlp"] is not None:
        x = x + scalar_norm(feed_forward(x, w, i, lay["mlp"], r), w[p + "norm2"], eps)
    return x


def forward(cfg, w, tokens, dtype=torch.float32, collect=None, r=exact):
    """Logits [T, vocab] of one sequence; ``collect`` (a list) receives the residual stream after every layer."""
    w = {k: v.to(dtype) for k, v in w.items()}
    x, first = w["embed"][torch.as_tensor(tokens)], {}
    for i in range(len(cfg["layers"])):
        x = layer(x, cfg, w, i, first, r)
        if collect is not None:
            collect.append(x)
    return r(scalar_norm(x, w["final.norm"], cfg["norm"]["eps"])) @ w["head"].T
