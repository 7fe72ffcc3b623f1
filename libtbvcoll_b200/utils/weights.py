"""Weights in the HF safetensors layout, sharded for tensor parallelism.

The reference's engine did "TP-sharded weight loading" from an HF model directory
(reports/11_custom_engine.md:12; models are mounted read-only, step3b/node_launch.sh:31).
Here: a reader for ``*.safetensors`` (+ ``model.safetensors.index.json``) that slices each
tensor for one rank, and a seeded random initialiser that yields tensors under the SAME HF
names and shapes, so benchmarks and tests go through the same sharding code as a real
checkpoint.  Sharding: q/k/v/gate/up by output rows (column-parallel), o_proj/down_proj by
input columns (row-parallel), embed_tokens/lm_head by vocabulary rows.
"""
from __future__ import annotations

import json
import os
import zlib
from typing import Callable, Dict, Iterable, Optional

import torch

from ..models.config import (BobaraxConfig, ChannelDeltaSpec, GatedMlpSpec, GlaSpec, LatentSpec, LightningSpec, LugizenConfig, MambaSpec, ModelConfig, MoeSpec,
                             NubosunConfig, TableMoeSpec, TinapelConfig, WkvSpec)


def hf_tensor_shapes(cfg: ModelConfig) -> Dict[str, tuple]:
    h, d = cfg.hidden_size, cfg.head_dim
    shapes = {"model.embed_tokens.weight": (cfg.vocab_size, h), "model.norm.weight": (h,)}
    if not cfg.tie_embeddings:
        shapes["lm_head.weight"] = (cfg.vocab_size, h)
    for l in range(cfg.num_layers):
        p = f"model.layers.{l}."
        shapes[p + "input_layernorm.weight"] = (h,)
        shapes[p + "post_attention_layernorm.weight"] = (h,)
        shapes[p + "self_attn.q_proj.weight"] = (cfg.num_heads * d, h)
        shapes[p + "self_attn.k_proj.weight"] = (cfg.num_kv_heads * d, h)
        shapes[p + "self_attn.v_proj.weight"] = (cfg.num_kv_heads * d, h)
        shapes[p + "self_attn.o_proj.weight"] = (h, cfg.num_heads * d)
        if cfg.qkv_bias:
            shapes[p + "self_attn.q_proj.bias"] = (cfg.num_heads * d,)
            shapes[p + "self_attn.k_proj.bias"] = (cfg.num_kv_heads * d,)
            shapes[p + "self_attn.v_proj.bias"] = (cfg.num_kv_heads * d,)
        shapes[p + "mlp.gate_proj.weight"] = (cfg.intermediate_size, h)
        shapes[p + "mlp.up_proj.weight"] = (cfg.intermediate_size, h)
        shapes[p + "mlp.down_proj.weight"] = (h, cfg.intermediate_size)
    return shapes


def nubosun_tensor_shapes(cfg: NubosunConfig) -> Dict[str, tuple]:
    W, S = cfg.hidden_size, cfg.streams
    shapes = {"embed": (cfg.vocab_size, W), "final.norm": (W,), "head": (cfg.vocab_size, W)}
    for i, lay in enumerate(cfg.layers):
        p, m = f"l{i}.", lay.mixer
        for q in (1, 2) if lay.mlp is not None else (1,):
            shapes[f"{p}norm{q}"] = shapes[f"{p}ls{q}"] = (W,)
            shapes[f"{p}hc{q}.in"] = shapes[f"{p}hc{q}.out"] = (S,)
            shapes[f"{p}hc{q}.mix"] = (S, S)
        if isinstance(m, MambaSpec):
            shapes.update({p + "mix.in": (2 * m.inner, W), p + "mix.conv": (m.inner, m.conv), p + "mix.conv.b": (m.inner,),
                           p + "mix.x": (m.dt_rank + 2 * m.state, m.inner), p + "mix.dt": (m.inner, m.dt_rank), p + "mix.dt.b": (m.inner,),
                           p + "mix.A_log": (m.inner, m.state), p + "mix.D": (m.inner,), p + "mix.o": (W, m.inner)})
        else:
            shapes.update({p + "mix.q": (m.heads * (m.dim + m.rot_dim), W), p + "mix.dkv": (m.kv_rank + m.rot_dim, W), p + "mix.dkv.norm": (m.kv_rank,),
                           p + "mix.uk": (m.heads * m.dim, m.kv_rank), p + "mix.uv": (m.heads * m.vdim, m.kv_rank), p + "mix.sink": (m.heads,),
                           p + "mix.o": (W, m.heads * m.vdim)})
        if lay.mlp is not None:
            shapes.update({p + "mlp.gate": (lay.mlp.ff, W), p + "mlp.up": (lay.mlp.ff, W), p + "mlp.down": (W, lay.mlp.ff)})
    return shapes


def tinapel_tensor_shapes(cfg: TinapelConfig) -> Dict[str, tuple]:
    """A decay rank that the configuration leaves open is 16 here; in a checkpoint its tensors tell."""
    W = cfg.hidden_size
    shapes = {"embed": (cfg.vocab_size, W), "final.norm": (W,)}
    if cfg.loop is not None:
        shapes["loop.step"] = (cfg.loop.times, W)
    for i, lay in enumerate(cfg.layers):
        p, m, f = f"l{i}.", lay.mixer, lay.mlp
        shapes[p + "norm1"] = (W,)
        x = p + "mix."
        if isinstance(m, GlaSpec):
            K, V, R = m.heads * m.dim, m.heads * m.vdim, m.decay_rank or 16
            shapes.update({x + "q": (K, W), x + "k": (K, W), x + "v": (V, W), x + "g": (V, W), x + "o": (W, V), x + "norm": (m.vdim,), x + "a1": (R, W),
                           x + "a2": (K, R), x + "a2.b": (K,)})
        elif isinstance(m, WkvSpec):
            K, R = m.heads * m.dim, m.decay_rank or 16
            shapes.update({x + "mu." + s: (W,) for s in "rkvgw"})
            shapes.update({x + s: (K, W) for s in "rkvg"})
            shapes.update({x + "w1": (R, W), x + "w2": (K, R), x + "w0": (K,), x + "u": (m.heads, m.dim), x + "norm": (K,), x + "o": (W, K)})
        else:
            shapes.update({x + "q": (m.heads * m.dim, W), x + "k": (m.kv_heads * m.dim, W), x + "q.norm": (m.dim,), x + "k.norm": (m.dim,),
                           x + "o": (W, m.heads * m.dim)})
        if f is not None:
            shapes[p + "norm2"] = (W,)
            shapes[p + "mlp.router"] = (f.experts, W)
            ffs = {f"e{e}.": f.ff for e in range(f.experts)}
            if f.shared_ff:
                ffs["shared."] = f.shared_ff
            for e, n in ffs.items():
                shapes.update({p + "mlp." + e + "gate": (n, W), p + "mlp." + e + "up": (n, W), p + "mlp." + e + "down": (W, n)})
    return shapes


def bobarax_tensor_shapes(cfg: BobaraxConfig) -> Dict[str, tuple]:
    """``*.table`` holds integers."""
    W = cfg.hidden_size
    shapes = {"embed": (cfg.vocab_size, W), "final.norm": (W,)}
    for i, lay in enumerate(cfg.layers):
        p, m, f = f"l{i}.", lay.mixer, lay.mlp
        x, y = p + "mix.", p + "mlp."
        K, V = m.heads * m.dim, m.heads * m.vdim
        shapes.update({p + n: (W,) for n in (("norm1", "norm1b", "norm2", "norm2b") if f is not None else ("norm1", "norm1b"))})
        shapes.update({x + "q": (K, W), x + "o": (W, V)})
        if isinstance(m, LightningSpec):
            shapes.update({x + "k": (K, W), x + "v": (V, W), x + "g": (V, W), x + "norm": (V,)})
        else:
            shapes[x + "q.norm"] = (K,)
            if m.kv_from is None:
                shapes.update({x + "k": (m.kv_heads * m.dim, W), x + "v": (m.kv_heads * m.vdim, W), x + "k.norm": (m.kv_heads * m.dim,)})
            if m.gated:
                shapes[x + "g"] = (V, W)
        if isinstance(f, TableMoeSpec):
            shapes[y + "table"] = (cfg.vocab_size, f.top)
        for e in [f"e{j}." for j in range(f.experts)] if isinstance(f, TableMoeSpec) else [""] if f is not None else []:
            shapes.update({y + e + "gate": (f.ff, W), y + e + "up": (f.ff, W), y + e + "down": (W, f.ff)})
    return shapes


def lugizen_tensor_shapes(cfg: LugizenConfig) -> Dict[str, tuple]:
    """Ranks that the configuration leaves open are 16 here; in a checkpoint its tensors tell.  Norm weights of shape () are one number."""
    W = cfg.hidden_size
    shapes = {"embed": (cfg.vocab_size, W), "head": (cfg.vocab_size, W), "final.norm": ()}
    for i, lay in enumerate(cfg.layers):
        p, m, f = f"l{i}.", lay.mixer, lay.mlp
        x, y, H, D, V = p + "mix.", p + "mlp.", m.heads, m.dim, m.vdim
        shapes.update({p + "norm1": (), p + "canon1": (W, cfg.canon_taps), x + "o": (W, H * V)})
        if isinstance(m, ChannelDeltaSpec):
            K, Ra, Rg = m.kv_heads * D, m.decay_rank or 16, m.gate_rank or 16
            for s, n in (("q", K), ("k", K), ("v", H * V)):
                shapes.update({x + s: (n, W), x + s + ".conv": (n, m.conv)})
            shapes.update({x + "b": (H, W), x + "A_log": (H,), x + "norm": (V,), x + "a1": (Ra, W), x + "a2": (H * D, Ra), x + "dt_bias": (H * D,), x + "g1": (Rg, W),
                           x + "g2": (H * V, Rg)})
        elif isinstance(m, LatentSpec):
            shapes.update({x + "dq": (m.q_rank, W), x + "dq.norm": (m.q_rank,), x + "uq": (H * (D + m.rot_dim), m.q_rank), x + "dkv": (m.kv_rank + m.rot_dim, W),
                           x + "dkv.norm": (m.kv_rank,), x + "uk": (H * D, m.kv_rank), x + "uv": (H * V, m.kv_rank)})
        else:
            shapes.update({x + "q": (H * D, W), x + "k": (m.kv_heads * D, W), x + "v": (m.kv_heads * V, W), x + "temp": (H,)})
            if m.v_mix:
                shapes[x + "vmix"] = ()
        if f is not None:
            shapes[p + "norm2"] = ()
        if isinstance(f, MoeSpec):
            shapes[y + "router"] = (f.experts, W)
            for e in range(f.experts):
                shapes.update({f"{y}e{e}.gate": (f.ff, W), f"{y}e{e}.up": (f.ff, W), f"{y}e{e}.down": (W, f.ff)})
        elif f is not None:
            shapes.update({y + "up": (f.ff, W), y + "down": (W, f.ff)})
    return shapes


def tensor_shapes(cfg) -> Dict[str, tuple]:
    """Checkpoint tensor names and shapes of a configuration of any architecture."""
    for kind, shapes in ((NubosunConfig, nubosun_tensor_shapes), (TinapelConfig, tinapel_tensor_shapes), (BobaraxConfig, bobarax_tensor_shapes),
                         (LugizenConfig, lugizen_tensor_shapes)):
        if isinstance(cfg, kind):
            return shapes(cfg)
    return hf_tensor_shapes(cfg)


def _tinapel_random(name: str, shape: tuple, g: torch.Generator, device) -> torch.Tensor:
    """Random values that keep a Tinapel's activations near unit size: decays over many time scales, norms near one."""
    leaf = name.split(".", 1)[1] if name.startswith("l") and "." in name else name
    n = lambda: torch.randn(shape, generator=g, device=device, dtype=torch.float32)
    if leaf in ("norm1", "norm2", "final.norm"):
        return 0.1 * n()                              # norms are stored around zero
    if leaf in ("mix.norm", "mix.q.norm", "mix.k.norm"):
        return 1.0 + 0.1 * n()
    if leaf.startswith("mix.mu."):
        return torch.rand(shape, generator=g, device=device, dtype=torch.float32)
    if leaf == "mix.w0":
        return -3.0 + 1.5 * n()                       # decays exp(-exp(.)): memories of a few to a few hundred tokens
    if leaf == "mix.a2.b":
        return 1.0 + n()
    if leaf in ("mix.u", "step"):
        return 0.3 * n()
    return n() if leaf == "embed" else n() / shape[1] ** 0.5


def _bobarax_random(cfg: BobaraxConfig, name: str, shape: tuple, g: torch.Generator, device) -> torch.Tensor:
    """Random values that keep a Bobarax's activations near unit size; tables of random experts, all different per token id (int32)."""
    layer, leaf = name.split(".", 1) if name.startswith("l") and "." in name else ("", name)
    if leaf == "mlp.table":
        experts = cfg.layers[int(layer[1:])].mlp.experts
        return torch.rand(shape[0], experts, generator=g, device=device).argsort(1)[:, : shape[1]].to(torch.int32)
    n = torch.randn(shape, generator=g, device=device, dtype=torch.float32)
    if len(shape) == 1:
        return 0.1 * n if leaf in ("norm1", "norm1b", "norm2", "norm2b", "final.norm") else 1.0 + 0.1 * n      # the former are stored around zero
    return n if leaf == "embed" else n / shape[1] ** 0.5


def _lugizen_random(name: str, shape: tuple, g: torch.Generator, device) -> torch.Tensor:
    """Random values that keep a Lugizen's activations near unit size: decays over many time scales."""
    leaf = name.split(".", 1)[1] if name.startswith("l") and "." in name else name
    n = torch.randn(shape, generator=g, device=device, dtype=torch.float32)
    u = lambda: torch.rand(shape, generator=g, device=device, dtype=torch.float32)
    if len(shape) == 0:
        return 0.5 + 0.1 * n if leaf == "mix.vmix" else 1.0 + 0.1 * n
    if leaf == "mix.A_log":
        return torch.log(1.0 + 15.0 * u())
    if leaf == "mix.dt_bias":
        return -7.0 + 5.0 * u()                       # softplus: steps of 0.001 .. 0.1
    if len(shape) == 1:
        return 1.0 + 0.1 * n
    if leaf == "canon1":
        return 0.3 * n
    return n if leaf == "embed" else n / shape[1] ** 0.5


def _nubosun_random(name: str, shape: tuple, g: torch.Generator, device) -> torch.Tensor:
    """Random values that keep a Nubosun's activations near unit size: decays over many time scales, mixing near the identity."""
    leaf = name.split(".", 1)[1] if name.startswith("l") and "." in name else name
    n = lambda *s: torch.randn(s or shape, generator=g, device=device, dtype=torch.float32)
    u = lambda: torch.rand(shape, generator=g, device=device, dtype=torch.float32)
    if leaf.startswith("norm") or leaf in ("final.norm", "mix.dkv.norm") or leaf.startswith("ls"):
        return 1.0 + 0.1 * n()
    if leaf == "mix.A_log":
        return torch.log(0.5 + 8.0 * u())
    if leaf == "mix.dt.b":
        return -4.0 + 3.0 * u()                       # softplus: steps of 0.02 .. 0.3
    if leaf == "mix.D":
        return 1.0 + 0.1 * n()
    if leaf.endswith(".in") and leaf.startswith("hc"):
        return 1.0 / shape[0] + 0.1 * n()
    if leaf.endswith(".out"):
        return 1.0 + 0.2 * n()
    if leaf.endswith(".mix") and leaf.startswith("hc"):
        return torch.eye(shape[0], device=device) * 0.9 + 0.05 * n()
    if leaf in ("mix.sink", "mix.conv.b"):
        return 0.5 * n()
    if leaf == "mix.conv":
        return n() / shape[1] ** 0.5
    if leaf == "embed":
        return n()
    return n() / shape[1] ** 0.5


class RandomSource:
    """Seeded random weights under HF names.  A tensor's values depend only on (seed, name),
    never on the TP degree, so every rank slices the same virtual checkpoint."""

    def __init__(self, cfg: ModelConfig, seed: int = 0, device="cpu", dtype=torch.bfloat16):
        self.cfg, self.seed, self.device, self.dtype = cfg, seed, torch.device(device), dtype
        self.shapes = tensor_shapes(cfg)

    def names(self) -> Iterable[str]:
        return self.shapes.keys()

    def get(self, name: str) -> torch.Tensor:
        shape = self.shapes[name]
        g = torch.Generator(device=self.device).manual_seed((self.seed * 1000003 + zlib.crc32(name.encode())) & 0x7FFFFFFF)
        if isinstance(self.cfg, NubosunConfig):
            t = _nubosun_random(name, shape, g, self.device)
        elif isinstance(self.cfg, TinapelConfig):
            t = _tinapel_random(name, shape, g, self.device)
        elif isinstance(self.cfg, BobaraxConfig):
            t = _bobarax_random(self.cfg, name, shape, g, self.device)
        elif isinstance(self.cfg, LugizenConfig):
            t = _lugizen_random(name, shape, g, self.device)
        elif name.endswith("layernorm.weight") or name.endswith("norm.weight"):
            t = 1.0 + 0.1 * torch.randn(shape, generator=g, device=self.device, dtype=torch.float32)
        elif name.endswith(".bias"):
            t = 0.1 * torch.randn(shape, generator=g, device=self.device, dtype=torch.float32)
        else:
            t = 0.02 * torch.randn(shape, generator=g, device=self.device, dtype=torch.float32)
        return t.to(self.dtype) if t.is_floating_point() else t


class SafetensorsSource:
    """An HF checkpoint directory (single file or sharded with an index)."""

    def __init__(self, path: str, device="cpu", dtype=torch.bfloat16):
        from safetensors import safe_open
        self.device, self.dtype = device, dtype
        self._open = safe_open
        idx = os.path.join(path, "model.safetensors.index.json")
        self.where: Dict[str, str] = {}
        if os.path.exists(idx):
            with open(idx) as f:
                for k, v in json.load(f)["weight_map"].items():
                    self.where[k] = os.path.join(path, v)
        else:
            files = sorted(f for f in os.listdir(path) if f.endswith(".safetensors"))
            if not files:
                raise FileNotFoundError(f"no .safetensors under {path}")
            for fn in files:
                with safe_open(os.path.join(path, fn), framework="pt") as f:
                    for k in f.keys():
                        self.where[k] = os.path.join(path, fn)

    def names(self) -> Iterable[str]:
        return self.where.keys()

    def get(self, name: str) -> torch.Tensor:
        with self._open(self.where[name], framework="pt", device="cpu") as f:
            t = f.get_tensor(name)
        return (t.to(self.dtype) if t.is_floating_point() else t).to(self.device)

    def get_rows(self, name: str, r0: int, r1: int) -> torch.Tensor:
        """Rows [r0, r1) without reading the rest of the tensor."""
        with self._open(self.where[name], framework="pt", device="cpu") as f:
            return f.get_slice(name)[r0:r1].to(self.dtype).to(self.device)


def save_hf_checkpoint(source, path: str, max_shard_bytes: int = 1 << 30) -> None:
    """Write every tensor of ``source`` as an HF-style sharded safetensors checkpoint."""
    from safetensors.torch import save_file
    os.makedirs(path, exist_ok=True)
    shards, cur, cur_bytes = [], {}, 0
    for n in source.names():
        t = source.get(n).cpu().contiguous()
        if cur and cur_bytes + t.numel() * t.element_size() > max_shard_bytes:
            shards.append(cur)
            cur, cur_bytes = {}, 0
        cur[n] = t
        cur_bytes += t.numel() * t.element_size()
    if cur:
        shards.append(cur)
    weight_map = {}
    for i, sh in enumerate(shards):
        fn = f"model-{i + 1:05d}-of-{len(shards):05d}.safetensors"
        save_file(sh, os.path.join(path, fn))
        for n in sh:
            weight_map[n] = fn
    with open(os.path.join(path, "model.safetensors.index.json"), "w") as f:
        json.dump({"metadata": {}, "weight_map": weight_map}, f)


def _rows(source, name: str, r0: int, r1: int) -> torch.Tensor:
    if hasattr(source, "get_rows"):
        return source.get_rows(name, r0, r1)
    return source.get(name)[r0:r1]


def _pad16(n: int) -> int:
    return (n + 15) // 16 * 16


def _padded(t: torch.Tensor, rows: int, cols: Optional[int] = None) -> torch.Tensor:
    """Zero-padded copy: [rows] or [rows, cols]."""
    out = torch.zeros((rows,) if cols is None else (rows, cols), dtype=t.dtype, device=t.device)
    if cols is None:
        out[: t.shape[0]] = t
    else:
        out[: t.shape[0], : t.shape[1]] = t
    return out


def _pad_heads(t: torch.Tensor, heads: int, dim: int, dim_p: int) -> torch.Tensor:
    """[heads * dim, K] -> [heads * dim_p, K], each head's rows followed by zero rows."""
    out = torch.zeros(heads, dim_p, t.shape[1], dtype=t.dtype, device=t.device)
    out[:, :dim] = t.reshape(heads, dim, -1)
    return out.reshape(heads * dim_p, -1)


def _heads_padded(t: torch.Tensor, heads: int, dim: int) -> torch.Tensor:
    """[heads * dim, K] -> [heads * pad16(dim), K]"""
    return _pad_heads(t, heads, dim, _pad16(dim))


def _head_vector(t: torch.Tensor, heads: int, dim: int) -> torch.Tensor:
    """[heads * dim] -> [heads * pad16(dim)]"""
    return _pad_heads(t.reshape(-1, 1), heads, dim, _pad16(dim)).reshape(-1)


def _pairs_together(t: torch.Tensor, heads: int, dims: int) -> torch.Tensor:
    """Rows of every head reordered so that dimensions i and i + dims / 2 of the first ``dims`` become neighbours 2i and 2i + 1 (a rotation of such pairs, norms and
    products between rows in this order do not notice)."""
    t = t.reshape(heads, -1, t.shape[1])
    order = torch.arange(t.shape[1], device=t.device)
    order[:dims] = torch.arange(dims, device=t.device).view(2, -1).t().reshape(-1)
    return t[:, order].reshape(-1, t.shape[2])


def _latent_products(uk: torch.Tensor, uv: torch.Tensor, m: LatentSpec, dtype) -> Dict[str, torch.Tensor]:
    """The forms in which latent attention takes W_uk and W_uv: ``wabs`` [heads * rank, dim] folds W_uk into the query, ``wuv`` [heads * vdim, rank] expands a latent,
    ``wukv`` [heads * (dim + vdim), rank] gives keys then values (bf16 only)."""
    H, D, V, R = m.heads, _pad16(m.dim), _pad16(m.vdim), _pad16(m.kv_rank)
    wabs = torch.zeros(H, R, D, dtype=uk.dtype, device=uk.device)
    wabs[:, : m.kv_rank, : m.dim] = uk.reshape(H, m.dim, m.kv_rank).transpose(1, 2)
    wuv = _padded(_pad_heads(uv, H, m.vdim, V), H * V, R)
    out = {"wabs": wabs.reshape(H * R, D), "wuv": wuv}
    if dtype is torch.bfloat16:
        out["wukv"] = torch.cat((_padded(_pad_heads(uk, H, m.dim, D), H * D, R), wuv))
    return out


class _Layout:
    """Checked reads from a checkpoint and the product layout being filled (``out``)."""

    def __init__(self, cfg, source, device, dtype):
        self.source, self.device, self.dtype, self.want = source, torch.device(device), dtype, tensor_shapes(cfg)
        self.W, self.Wp = cfg.hidden_size, _pad16(cfg.hidden_size)
        self.out: Dict[str, torch.Tensor] = {}

    def get(self, name: str, open_dim: Optional[int] = None) -> torch.Tensor:
        """A tensor of the expected shape; dimension ``open_dim`` may have any size."""
        t, shape = self.source.get(name), list(self.want[name])
        if open_dim is not None:
            shape[open_dim] = t.shape[open_dim]
        if list(t.shape) != shape:
            raise ValueError(f"{name}: shape {tuple(t.shape)}, expected {tuple(shape)}")
        return t

    def put(self, name: str, t: torch.Tensor, as_dtype: Optional[torch.dtype] = None) -> None:
        self.out[name] = t.to(as_dtype or self.dtype).to(self.device).contiguous()

    def out_proj(self, t: torch.Tensor, heads: int, dim: int) -> torch.Tensor:
        """[W, heads * dim] -> [Wp, heads * pad16(dim)]"""
        return _padded(_heads_padded(t.t(), heads, dim).t(), self.Wp, heads * _pad16(dim))

    def gate_up(self, gate: torch.Tensor, up: torch.Tensor, ff: int) -> torch.Tensor:
        """Rows gate_0, up_0, gate_1, .. [2 * pad16(ff), Wp]"""
        fp = _pad16(ff)
        return torch.stack((_padded(gate, fp, self.Wp), _padded(up, fp, self.Wp)), 1).reshape(2 * fp, self.Wp)

    def put_experts(self, x: str, experts: int, ff: int) -> None:
        fp, Wp = _pad16(ff), self.Wp
        gu = torch.empty(experts * 2 * fp, Wp, dtype=self.dtype, device=self.device)
        down = torch.empty(experts * Wp, fp, dtype=self.dtype, device=self.device)
        for e in range(experts):
            q = f"{x}e{e}."
            gu[e * 2 * fp: (e + 1) * 2 * fp] = self.gate_up(self.get(q + "gate"), self.get(q + "up"), ff)
            down[e * Wp: (e + 1) * Wp] = _padded(self.get(q + "down"), Wp, fp)
        self.out[x + "gate_up"], self.out[x + "down"] = gu, down


def load_nubosun(cfg: NubosunConfig, source, device, dtype=torch.bfloat16) -> Dict[str, torch.Tensor]:
    """Tensors the way the kernels consume them.  Every dimension that a matrix product runs over is padded with zeros to a multiple
    of 16 (so that any configuration meets the TMA alignment rules); small parameters that act in 32-bit are fp32.

    Latent attention: ``qkv`` stacks the heads' unrotated query rows, their rotated rows, the latent rows and the rotated key rows;
    ``wabs`` [heads * rank, dim] folds W_uk into the query, ``wuv`` [heads * vdim, rank] expands a latent, ``wukv`` [heads * (dim + vdim), rank]
    gives keys then values.  Mamba: ``in`` stacks x rows and z rows, ``conv`` is transposed to [taps, inner], ``a2`` = -exp(A_log) * log2 e."""
    dev, out = torch.device(device), {}
    Wp = _pad16(cfg.hidden_size)
    want = nubosun_tensor_shapes(cfg)

    def get(name):
        t = source.get(name)
        if tuple(t.shape) != tuple(want[name]):
            raise ValueError(f"{name}: shape {tuple(t.shape)}, expected {tuple(want[name])}")
        return t

    def put(name, t, as_dtype=dtype):
        out[name] = t.to(as_dtype).to(dev).contiguous()

    f32 = torch.float32
    put("embed", _padded(get("embed"), cfg.vocab_size, Wp))
    put("head", _padded(get("head"), _pad16(cfg.vocab_size), Wp))
    put("final.norm", _padded(get("final.norm"), Wp), f32)
    for i, lay in enumerate(cfg.layers):
        p, m = f"l{i}.", lay.mixer
        for q in (1, 2) if lay.mlp is not None else (1,):
            put(f"{p}norm{q}", _padded(get(f"{p}norm{q}"), Wp), f32)
            put(f"{p}ls{q}", _padded(get(f"{p}ls{q}"), Wp), f32)
            for k in ("in", "out", "mix"):
                put(f"{p}hc{q}.{k}", get(f"{p}hc{q}.{k}"), f32)
        x = p + "mix."
        if isinstance(m, MambaSpec):
            ip, kd = _pad16(m.inner), _pad16(m.dt_rank)
            w = get(x + "in")
            put(x + "in", torch.cat((_padded(w[: m.inner], ip, Wp), _padded(w[m.inner:], ip, Wp))))
            put(x + "conv", _padded(get(x + "conv").t(), m.conv, ip), f32)
            put(x + "conv.b", _padded(get(x + "conv.b"), ip), f32)
            put(x + "x", _padded(get(x + "x"), _pad16(m.dt_rank + 2 * m.state), ip))
            put(x + "dt", _padded(get(x + "dt"), ip, kd))
            put(x + "dt.b", _padded(get(x + "dt.b"), ip))
            put(x + "a2", -torch.exp(get(x + "A_log").float()) * 1.4426950408889634, f32)
            put(x + "D", get(x + "D"), f32)
            put(x + "o", _padded(get(x + "o"), Wp, ip))
        else:
            H, D, V, R, rot = m.heads, _pad16(m.dim), _pad16(m.vdim), _pad16(m.kv_rank), _pad16(m.rot_dim)
            q = get(x + "q").reshape(H, m.dim + m.rot_dim, -1)
            kv = get(x + "dkv")
            rows = torch.cat((_pad_heads(q[:, : m.dim].reshape(H * m.dim, -1), H, m.dim, D),
                              _pad_heads(q[:, m.dim:].reshape(H * m.rot_dim, -1), H, m.rot_dim, rot),
                              _padded(kv[: m.kv_rank], R, kv.shape[1]), _padded(kv[m.kv_rank:], rot, kv.shape[1])))
            put(x + "qkv", _padded(rows, rows.shape[0], Wp))
            put(x + "dkv.norm", get(x + "dkv.norm"), f32)
            put(x + "sink", get(x + "sink"), f32)
            for k, t in _latent_products(get(x + "uk"), get(x + "uv"), m, dtype).items():
                put(x + k, t)
            put(x + "o", _padded(_heads_padded(get(x + "o").t(), H, m.vdim).t(), Wp, H * V))
        if lay.mlp is not None:
            x, fp = p + "mlp.", _pad16(lay.mlp.ff)
            g, u = _padded(get(x + "gate"), fp, Wp), _padded(get(x + "up"), fp, Wp)
            put(x + "gate_up", torch.stack((g, u), 1).reshape(2 * fp, Wp))
            put(x + "down", _padded(get(x + "down"), Wp, fp))
    return out


def load_tinapel(cfg: TinapelConfig, source, device, dtype=torch.bfloat16) -> Dict[str, torch.Tensor]:
    """Tensors the way the kernels consume them; dimensions of matrix products and heads are zero-padded to multiples of 16, parameters that
    act in 32-bit are fp32.

    ``embed`` serves as the head too (rows padded).  GLA: ``in`` stacks q, k, v, g and the first decay projection.  WKV: ``in`` stacks r, k, v,
    g and the first decay projection, each for a mix of its own; ``mu`` [5, width] in the same order.  Attention: ``in`` stacks q and k; ``fold`` =
    query norm * key norm * scale (what is left of a key is one factor per token).  Experts: ``gate_up`` [experts * 2 ff, width], rows
    interleaved, and ``down`` [experts * width, ff].  Norm weights hold 1 + w."""
    L, f32 = _Layout(cfg, source, device, dtype), torch.float32
    W, Wp, get, put, out_proj, gate_up, heads_padded, vector = L.W, L.Wp, L.get, L.put, L.out_proj, L.gate_up, _heads_padded, _head_vector
    put("embed", _padded(get("embed"), _pad16(cfg.vocab_size), Wp))
    put("final.norm", _padded(1.0 + get("final.norm").float(), Wp), f32)
    if cfg.loop is not None:
        put("loop.step", _padded(get("loop.step"), cfg.loop.times, Wp), f32)
    for i, lay in enumerate(cfg.layers):
        p, m, f = f"l{i}.", lay.mixer, lay.mlp
        x = p + "mix."
        put(p + "norm1", _padded(1.0 + get(p + "norm1").float(), Wp), f32)
        if isinstance(m, GlaSpec):
            H, D, V = m.heads, m.dim, m.vdim
            a1 = get(x + "a1", 0)
            R = _pad16(a1.shape[0])
            rows = torch.cat((heads_padded(get(x + "q"), H, D), heads_padded(get(x + "k"), H, D), heads_padded(get(x + "v"), H, V),
                              heads_padded(get(x + "g"), H, V), _padded(a1, R, W)))
            put(x + "in", _padded(rows, rows.shape[0], Wp))
            put(x + "decay", _padded(heads_padded(get(x + "a2", 1), H, D), H * _pad16(D), R))
            put(x + "decay.b", vector(get(x + "a2.b"), H, D))
            put(x + "norm", vector(get(x + "norm").repeat(H), H, V), f32)
            put(x + "o", out_proj(get(x + "o"), H, V))
        elif isinstance(m, WkvSpec):
            H, D = m.heads, m.dim
            w1 = get(x + "w1", 0)
            R = _pad16(w1.shape[0])
            rows = torch.cat([heads_padded(get(x + s), H, D) for s in "rkvg"] + [_padded(w1, R, W)])
            put(x + "in", _padded(rows, rows.shape[0], Wp))
            put(x + "mu", torch.stack([_padded(get(x + "mu." + s), Wp) for s in "rkvgw"]), f32)
            put(x + "decay", _padded(heads_padded(get(x + "w2", 1), H, D), H * _pad16(D), R))
            put(x + "decay.b", vector(get(x + "w0"), H, D))
            put(x + "u", vector(get(x + "u").reshape(-1), H, D), f32)
            put(x + "norm", vector(get(x + "norm"), H, D), f32)
            put(x + "o", out_proj(get(x + "o"), H, D))
        else:
            H, G, D = m.heads, m.kv_heads, m.dim
            rows = torch.cat((heads_padded(get(x + "q"), H, D), heads_padded(get(x + "k"), G, D)))
            put(x + "in", _padded(rows, rows.shape[0], Wp))
            put(x + "fold", _padded(get(x + "q.norm").float() * get(x + "k.norm").float() * m.scale, _pad16(D)), f32)
            put(x + "o", out_proj(get(x + "o"), H, D))
        if f is not None:
            x = p + "mlp."
            put(p + "norm2", _padded(1.0 + get(p + "norm2").float(), Wp), f32)
            put(x + "router", _padded(get(x + "router"), _pad16(f.experts), Wp))
            L.put_experts(x, f.experts, f.ff)
            if f.shared_ff:
                put(x + "shared.gate_up", gate_up(get(x + "shared.gate"), get(x + "shared.up"), f.shared_ff))
                put(x + "shared.down", _padded(get(x + "shared.down"), Wp, _pad16(f.shared_ff)))
    return L.out


def load_bobarax(cfg: BobaraxConfig, source, device, dtype=torch.bfloat16) -> Dict[str, torch.Tensor]:
    """Tensors the way the kernels consume them; dimensions of matrix products and heads are zero-padded to multiples of 16, parameters that act in 32-bit are
    fp32.

    ``embed`` serves as the head too (rows padded); the logits' scale is part of the final norm's weight and the residual multiplier of the norms behind the
    sublayers (norm weights hold 1 + w).  Lightning: ``in`` stacks q, k, v, g.  Attention: ``in`` stacks q, k, v (unless they come from another layer) and g (if
    gated); the score scale is part of the query norm's weight.  Feed-forwards: ``gate_up`` with rows interleaved, ``down``; experts one after the other."""
    L, f32 = _Layout(cfg, source, device, dtype), torch.float32
    W, Wp, get, put = L.W, L.Wp, L.get, L.put
    put("embed", _padded(get("embed"), _pad16(cfg.vocab_size), Wp))
    put("final.norm", _padded((1.0 + get("final.norm").float()) * cfg.logit_scale, Wp), f32)
    for i, lay in enumerate(cfg.layers):
        p, m, f = f"l{i}.", lay.mixer, lay.mlp
        x, y, H, D, V = p + "mix.", p + "mlp.", m.heads, m.dim, m.vdim
        for n in ("1", "2") if f is not None else ("1",):
            put(f"{p}norm{n}", _padded(1.0 + get(f"{p}norm{n}").float(), Wp), f32)
            put(f"{p}norm{n}b", _padded((1.0 + get(f"{p}norm{n}b").float()) * cfg.residual_mult, Wp), f32)
        rows = [_heads_padded(get(x + "q"), H, D)]
        if isinstance(m, LightningSpec):
            rows += [_heads_padded(get(x + "k"), H, D), _heads_padded(get(x + "v"), H, V), _heads_padded(get(x + "g"), H, V)]
            put(x + "norm", _head_vector(get(x + "norm"), H, V), f32)
        else:
            put(x + "q.norm", _head_vector(get(x + "q.norm").float() * m.scale, H, D), f32)
            if m.kv_from is None:
                rows += [_heads_padded(get(x + "k"), m.kv_heads, D), _heads_padded(get(x + "v"), m.kv_heads, V)]
                put(x + "k.norm", _head_vector(get(x + "k.norm"), m.kv_heads, D), f32)
            if m.gated:
                rows.append(_heads_padded(get(x + "g"), H, V))
        rows = torch.cat(rows)
        put(x + "in", _padded(rows, rows.shape[0], Wp))
        put(x + "o", L.out_proj(get(x + "o"), H, V))
        if isinstance(f, GatedMlpSpec):
            put(y + "gate_up", L.gate_up(get(y + "gate"), get(y + "up"), f.ff))
            put(y + "down", _padded(get(y + "down"), Wp, _pad16(f.ff)))
        elif f is not None:
            table = get(y + "table")
            if table.is_floating_point() or int(table.min()) < 0 or int(table.max()) >= f.experts:
                raise ValueError(f"{y}table: not a table of {f.experts} experts")
            put(y + "table", table, torch.int32)
            L.put_experts(y, f.experts, f.ff)
    return L.out


def load_lugizen(cfg: LugizenConfig, source, device, dtype=torch.bfloat16) -> Dict[str, torch.Tensor]:
    """Tensors the way the kernels consume them; dimensions of matrix products and heads are zero-padded to multiples of 16, parameters that act in 32-bit are
    fp32; norms of one number are spread over the width; convolutions are transposed to [taps, channels].

    Delta rule: ``in`` stacks q, k, v, both first low-rank projections (padded to one rank) and the step sizes; ``conv`` covers q, k, v; ``rate`` = exp(A_log).
    Attention: ``in`` stacks q, k, v; rotated pairs lie next to each other; ``qscale`` = score scale times the head's number.  Latent attention: ``down`` stacks the
    queries' latent, the latent and the rotated key part, ``uq`` the heads' unrotated rows, then their rotated ones (pairs next to each other)."""
    L, f32 = _Layout(cfg, source, device, dtype), torch.float32
    W, Wp, get, put = L.W, L.Wp, L.get, L.put
    spread = lambda name: put(name, _padded(get(name).float().reshape(1).expand(W), Wp), f32)
    put("embed", _padded(get("embed"), cfg.vocab_size, Wp))
    put("head", _padded(get("head"), _pad16(cfg.vocab_size), Wp))
    spread("final.norm")
    for i, lay in enumerate(cfg.layers):
        p, m, f = f"l{i}.", lay.mixer, lay.mlp
        x, y, H, D, V = p + "mix.", p + "mlp.", m.heads, m.dim, m.vdim
        spread(p + "norm1")
        put(p + "canon1", _padded(get(p + "canon1").t(), cfg.canon_taps, Wp), f32)
        put(x + "o", L.out_proj(get(x + "o"), H, V))
        if isinstance(m, ChannelDeltaSpec):
            G, a1, g1 = m.kv_heads, get(x + "a1", 0), get(x + "g1", 0)
            R = _pad16(max(a1.shape[0], g1.shape[0]))
            parts = (("q", G, D), ("k", G, D), ("v", H, V))
            rows = torch.cat([_heads_padded(get(x + s), n, d) for s, n, d in parts] + [_padded(a1, R, W), _padded(g1, R, W), _padded(get(x + "b"), _pad16(H), W)])
            put(x + "in", _padded(rows, rows.shape[0], Wp))
            put(x + "conv", torch.cat([_heads_padded(get(x + s + ".conv"), n, d) for s, n, d in parts]).t(), f32)
            put(x + "a2", _padded(_heads_padded(get(x + "a2", 1), H, D), H * _pad16(D), R))
            put(x + "dt_bias", _head_vector(get(x + "dt_bias"), H, D))
            put(x + "g2", _padded(_heads_padded(get(x + "g2", 1), H, V), H * _pad16(V), R))
            put(x + "rate", torch.exp(get(x + "A_log").float()), f32)
            put(x + "norm", _padded(get(x + "norm"), _pad16(V)), f32)
        elif isinstance(m, LatentSpec):
            R, Rq, rot = _pad16(m.kv_rank), _pad16(m.q_rank), _pad16(m.rot_dim)
            q, kv = get(x + "uq").reshape(H, D + m.rot_dim, -1), get(x + "dkv")
            rows = torch.cat((_padded(get(x + "dq"), Rq, W), _padded(kv[: m.kv_rank], R, W), _padded(_pairs_together(kv[m.kv_rank:], 1, m.rot.dims), rot, W)))
            put(x + "down", _padded(rows, rows.shape[0], Wp))
            rows = torch.cat((_heads_padded(q[:, :D].reshape(H * D, -1), H, D), _heads_padded(_pairs_together(q[:, D:].reshape(H * m.rot_dim, -1), H, m.rot.dims), H, m.rot_dim)))
            put(x + "uq", _padded(rows, rows.shape[0], Rq))
            put(x + "dq.norm", get(x + "dq.norm"), f32)
            put(x + "dkv.norm", get(x + "dkv.norm"), f32)
            for k, t in _latent_products(get(x + "uk"), get(x + "uv"), m, dtype).items():
                put(x + k, t)
        else:
            G, dims = m.kv_heads, m.rot.dims if m.rot is not None else 0
            rows = torch.cat((_heads_padded(_pairs_together(get(x + "q"), H, dims), H, D), _heads_padded(_pairs_together(get(x + "k"), G, dims), G, D),
                              _heads_padded(get(x + "v"), G, V)))
            put(x + "in", _padded(rows, rows.shape[0], Wp))
            put(x + "qscale", get(x + "temp").float() * m.scale, f32)
            if m.v_mix:
                put(x + "vmix", get(x + "vmix").reshape(1), f32)
        if f is not None:
            spread(p + "norm2")
        if isinstance(f, MoeSpec):
            put(y + "router", _padded(get(y + "router"), _pad16(f.experts), Wp))
            L.put_experts(y, f.experts, f.ff)
        elif f is not None:
            put(y + "up", _padded(get(y + "up"), _pad16(f.ff), Wp))
            put(y + "down", _padded(get(y + "down"), Wp, _pad16(f.ff)))
    return L.out


def shard_for_rank(cfg: ModelConfig, source, rank: int, tp: int, device, interleave_gate_up: bool = True) -> Dict[str, torch.Tensor]:
    """Per-rank tensors, fused the way the kernels consume them:
    ``layers.{l}.qkv.weight`` [(nq+2nkv)*D / tp', hidden], ``layers.{l}.qkv.bias``,
    ``layers.{l}.o.weight`` [hidden, nq*D/tp], ``layers.{l}.gate_up.weight`` [2*I/tp, hidden]
    (rows interleaved gate_i, up_i when ``interleave_gate_up``; otherwise [gate | up]),
    ``layers.{l}.down.weight`` [hidden, I/tp], the two norm weights per layer, ``embed``
    [V/tp, hidden], ``lm_head`` [V/tp, hidden], ``norm``."""
    cfg.check_tp(tp)
    d = cfg.head_dim
    nq = cfg.num_heads // tp
    nkv = cfg.kv_heads_per_rank(tp)
    # kv heads are split while there are at least `tp` of them, replicated beyond that
    kv0 = rank * nkv if cfg.num_kv_heads >= tp else rank // (tp // cfg.num_kv_heads)
    ipr = cfg.intermediate_size // tp
    vpr = cfg.vocab_size // tp
    out: Dict[str, torch.Tensor] = {}
    dev = torch.device(device)

    def put(k, t):
        out[k] = t.to(dev).contiguous()

    put("embed", _rows(source, "model.embed_tokens.weight", rank * vpr, (rank + 1) * vpr))
    head = "model.embed_tokens.weight" if cfg.tie_embeddings else "lm_head.weight"
    put("lm_head", _rows(source, head, rank * vpr, (rank + 1) * vpr))
    put("norm", source.get("model.norm.weight"))
    for l in range(cfg.num_layers):
        p = f"model.layers.{l}."
        q = _rows(source, p + "self_attn.q_proj.weight", rank * nq * d, (rank + 1) * nq * d)
        k = _rows(source, p + "self_attn.k_proj.weight", kv0 * d, (kv0 + nkv) * d)
        v = _rows(source, p + "self_attn.v_proj.weight", kv0 * d, (kv0 + nkv) * d)
        put(f"layers.{l}.qkv.weight", torch.cat((q, k, v), 0))
        if cfg.qkv_bias:
            qb = _rows(source, p + "self_attn.q_proj.bias", rank * nq * d, (rank + 1) * nq * d)
            kb = _rows(source, p + "self_attn.k_proj.bias", kv0 * d, (kv0 + nkv) * d)
            vb = _rows(source, p + "self_attn.v_proj.bias", kv0 * d, (kv0 + nkv) * d)
            put(f"layers.{l}.qkv.bias", torch.cat((qb, kb, vb), 0))
        put(f"layers.{l}.o.weight", source.get(p + "self_attn.o_proj.weight")[:, rank * nq * d:(rank + 1) * nq * d])
        g = _rows(source, p + "mlp.gate_proj.weight", rank * ipr, (rank + 1) * ipr)
        u = _rows(source, p + "mlp.up_proj.weight", rank * ipr, (rank + 1) * ipr)
        if interleave_gate_up:
            put(f"layers.{l}.gate_up.weight", torch.stack((g, u), 1).reshape(2 * ipr, cfg.hidden_size))
        else:
            put(f"layers.{l}.gate_up.weight", torch.cat((g, u), 0))
        put(f"layers.{l}.down.weight", source.get(p + "mlp.down_proj.weight")[:, rank * ipr:(rank + 1) * ipr])
        put(f"layers.{l}.input_norm", source.get(p + "input_layernorm.weight"))
        put(f"layers.{l}.post_norm", source.get(p + "post_attention_layernorm.weight"))
    return out
