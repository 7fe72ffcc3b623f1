"""Plain statement of the Bobarax decoder, used only as the oracle of its tests.

One function per mechanism, written for whole sequences with ordinary loops and matrix products, in float32 (or float64 on request), no
cache, no state hand-over, no batching, nothing shared with the product code.  ``w`` maps checkpoint tensor names to tensors and ``cfg``
is the parsed ``config.json`` dictionary.  ``r`` rounds what a 16-bit run may keep in 16 bits (inputs and results of matrix products, cached
rows); it is the identity unless the size of those roundings is wanted."""
from __future__ import annotations

import torch


def exact(x):
    return x


def to_bf16(x):
    return x.to(torch.bfloat16).to(x.dtype)


def rms(x, eps):
    return x / torch.sqrt((x * x).mean(-1, keepdim=True) + eps)


def one_plus_norm(x, w, eps):
    return rms(x, eps) * (1.0 + w)


def sigmoid(z):
    return 1.0 / (1.0 + torch.exp(-z))


def silu(z):
    return z * sigmoid(z)


# ---- lightning attention -------------------------------------------------------------------------------------------------------
def fixed_decay_attention(q, k, v, decay):
    """q, k [T, H, D], v [T, H, V], decay [H] -> [T, H, V]: S_t = decay_h S_{t-1} + k_t v_t^T, read by q_t after the update."""
    T, H, D = q.shape
    S = torch.zeros(H, D, v.shape[2], dtype=q.dtype)
    out = torch.zeros_like(v)
    for t in range(T):
        S = decay[:, None, None] * S + k[t][:, :, None] * v[t][:, None, :]
        out[t] = (S * q[t][:, :, None]).sum(1)
    return out


def joint_norm_gate(o, weight, gate, eps):
    """o [T, H, V]: all heads of a token normed together, then the gate."""
    return rms(o.reshape(o.shape[0], -1), eps) * weight * sigmoid(gate)


def lightning_mixer(h, w, i, m, eps, kv, r=exact):
    p, T, H, D, V = f"l{i}.mix.", h.shape[0], m["heads"], m["dim"], m["vdim"]
    h = r(h)
    q, k, v = (r(silu(h @ w[p + s].T)).view(T, H, n) for s, n in (("q", D), ("k", D), ("v", V)))
    g = r(h @ w[p + "g"].T)
    o = fixed_decay_attention(q, k, v, torch.tensor(m["decay"], dtype=torch.float64).to(q.dtype))
    return r(joint_norm_gate(o, w[p + "norm"], g, eps)) @ w[p + "o"].T


# ---- attention -------------------------------------------------------------------------------------------------------------------
def whole_norm(x, weight, eps):
    """All heads of the projection normed at once."""
    return rms(x, eps) * weight


def rotate(x, dims, base):
    """x [T, H, D]: dimensions 2i and 2i + 1 of the first ``dims`` turned by position * base^(-2i / dims)."""
    out = x.clone()
    t = torch.arange(x.shape[0], dtype=torch.float64)
    for i in range(dims // 2):
        a = t * float(base) ** (-2.0 * i / dims)
        c, s = torch.cos(a).to(x.dtype)[:, None], torch.sin(a).to(x.dtype)[:, None]
        u, v = x[:, :, 2 * i], x[:, :, 2 * i + 1]
        out[:, :, 2 * i], out[:, :, 2 * i + 1] = u * c - v * s, v * c + u * s
    return out


def window_mask(T, size):
    i, j = torch.arange(T)[:, None], torch.arange(T)[None]
    return (j <= i) & (i - j < size)


def chunk_mask(T, size):
    i, j = torch.arange(T)[:, None], torch.arange(T)[None]
    return (j <= i) & (i // size == j // size)


def softcap(s, cap):
    return cap * torch.tanh(s / cap)


def softmax_attention(q, k, v, scale, visible, cap=None, r=exact):
    """q [T, H, D], k [T, G, D], v [T, G, V], visible [T, T] -> [T, H, V]."""
    rep = q.shape[1] // k.shape[1]
    k, v = k.repeat_interleave(rep, 1), v.repeat_interleave(rep, 1)
    s = torch.einsum("ihd,jhd->hij", q, k) * scale
    if cap:
        s = softcap(s, cap)
    s = s.masked_fill(~visible[None], float("-inf"))
    return torch.einsum("hij,jhd->ihd", r(torch.softmax(s, -1)), v)


def queries_keys_values(h, w, i, m, eps, kv, r):
    """Queries of layer i; keys and values of its own, kept in ``kv[i]``, or those of layer ``kv_from``."""
    p, T, H, G, D, V = f"l{i}.mix.", h.shape[0], m["heads"], m["kv_heads"], m["dim"], m["vdim"]
    turn = (lambda x: rotate(x, m["rot"]["dims"], m["rot"]["base"])) if m.get("rot") else (lambda x: x)
    q = r(turn(whole_norm(r(h @ w[p + "q"].T), w[p + "q.norm"], eps).view(T, H, D)))
    if m.get("kv_from") is None:
        kv[i] = (r(turn(whole_norm(r(h @ w[p + "k"].T), w[p + "k.norm"], eps).view(T, G, D))), r(h @ w[p + "v"].T).view(T, G, V))
    else:
        kv[i] = kv[m["kv_from"]]
    return (q, *kv[i])


def chunked_attention_mixer(h, w, i, m, eps, kv, r=exact):
    h = r(h)
    q, k, v = queries_keys_values(h, w, i, m, eps, kv, r)
    o = softmax_attention(q, k, v, m["scale"], chunk_mask(h.shape[0], m["mask"]["size"]), m.get("softcap"), r)
    return r(o.reshape(h.shape[0], -1)) @ w[f"l{i}.mix.o"].T


def window_attention_mixer(h, w, i, m, eps, kv, r=exact):
    h = r(h)
    q, k, v = queries_keys_values(h, w, i, m, eps, kv, r)
    o = softmax_attention(q, k, v, m["scale"], window_mask(h.shape[0], m["mask"]["size"]), m.get("softcap"), r)
    g = r(h @ w[f"l{i}.mix.g"].T)
    return r(o.reshape(h.shape[0], -1) * sigmoid(g)) @ w[f"l{i}.mix.o"].T


# ---- feed-forward ------------------------------------------------------------------------------------------------------------------
def relu_mlp(h, w, p, r=exact):
    return r(torch.relu(h @ w[p + "gate"].T) * (h @ w[p + "up"].T)) @ w[p + "down"].T


def clamped_unit(g, u, limit):
    g, u = torch.clamp(g, max=limit), torch.clamp(u, -limit, limit)
    return g * sigmoid(1.702 * g) * (u + 1.0)


def clamped_mlp(h, w, p, limit, r=exact):
    return r(clamped_unit(h @ w[p + "gate"].T, h @ w[p + "up"].T, limit)) @ w[p + "down"].T


def table_weights(tokens, table, experts):
    """[T, experts]: 1 / top for the experts that the table gives a token, zero for the others."""
    out = torch.zeros(len(tokens), experts)
    for t, tok in enumerate(tokens):
        for e in table[tok].tolist():
            out[t, e] += 1.0 / table.shape[1]
    return out


def moe(h, w, p, m, tokens, r=exact):
    h, y = r(h), torch.zeros_like(h)
    weights = table_weights(tokens, w[p + "table"], m["router"]["experts"]).to(h.dtype)
    for e in range(m["router"]["experts"]):
        rows = torch.nonzero(weights[:, e])[:, 0]
        if len(rows):
            y[rows] = y[rows] + weights[rows, e][:, None] * r(clamped_mlp(h[rows], w, f"{p}e{e}.", m["expert"]["limit"], r))
    return y


def feed_forward(h, w, i, f, tokens, r=exact):
    return relu_mlp(r(h), w, f"l{i}.mlp.", r) if f["kind"] == "dense" else moe(h, w, f"l{i}.mlp.", f, tokens, r)


MIXERS = {"lightning": lightning_mixer, "attention": chunked_attention_mixer, "attention_2": window_attention_mixer}


def layer(x, cfg, w, i, tokens, kv, r=exact):
    lay, p, eps, mult = cfg["layers"][i], f"l{i}.", cfg["norm"]["eps"], cfg["residual_mult"]
    y = MIXERS[lay["type"]](one_plus_norm(x, w[p + "norm1"], eps), w, i, lay["mixer"], eps, kv, r)
    x = x + mult * one_plus_norm(y, w[p + "norm1b"], eps)
    if lay["mlp"] is not None:
        y = feed_forward(one_plus_norm(x, w[p + "norm2"], eps), w, i, lay["mlp"], tokens, r)
        x = x + mult * one_plus_norm(y, w[p + "norm2b"], eps)
    return x


def forward(cfg, w, tokens, dtype=torch.float32, collect=None, r=exact):
    """Logits [T, vocab] of one sequence; ``collect`` (a list) receives the residual stream after every layer."""
    w = {k: v if k.endswith(".table") else v.to(dtype) for k, v in w.items()}
    x, kv = w["embed"][torch.as_tensor(tokens)], {}
    for i in range(len(cfg["layers"])):
        x = layer(x, cfg, w, i, tokens, kv, r)
        if collect is not None:
            collect.append(x)
    return r(one_plus_norm(x, w["final.norm"], cfg["norm"]["eps"])) @ w["embed"].T * cfg["logit_scale"]
