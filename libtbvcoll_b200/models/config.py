"""Model shapes.  The reference serves Qwen2.5-7B-Instruct through vLLM
(step3b/run_vllm_tp.sh:9-10); the benchmark configurations of this repository are
Llama-3-8B- and Llama-3-70B-shaped.  All are the same decoder family (RMSNorm, RoPE,
GQA, SiLU-gated MLP); Qwen2 adds a bias on the q/k/v projections."""
from __future__ import annotations

import json
import math
from dataclasses import dataclass, field
from typing import List, Optional, Union


@dataclass
class ModelConfig:
    name: str = "llama3-8b"
    hidden_size: int = 4096
    num_layers: int = 32
    num_heads: int = 32
    num_kv_heads: int = 8
    head_dim: int = 128
    intermediate_size: int = 14336
    vocab_size: int = 128256
    rope_theta: float = 5e5
    rms_eps: float = 1e-5
    max_position: int = 8192
    qkv_bias: bool = False
    tie_embeddings: bool = False
    rope_scaling: Optional[dict] = field(default=None)

    def check_tp(self, tp: int) -> None:
        if self.num_heads % tp or self.intermediate_size % tp or self.vocab_size % tp:
            raise ValueError(f"{self.name}: heads/intermediate/vocab not divisible by tp={tp}")
        if self.num_kv_heads % tp and tp % self.num_kv_heads:
            raise ValueError(f"{self.name}: kv heads {self.num_kv_heads} incompatible with tp={tp}")
        if self.head_dim != 128:
            raise ValueError("the attention kernels are written for head_dim 128")

    def kv_heads_per_rank(self, tp: int) -> int:
        return max(1, self.num_kv_heads // tp)  # replicated when tp > kv heads

    def param_count(self) -> int:
        h, i, v = self.hidden_size, self.intermediate_size, self.vocab_size
        qkv = h * (self.num_heads + 2 * self.num_kv_heads) * self.head_dim
        per_layer = qkv + self.num_heads * self.head_dim * h + 3 * h * i + 2 * h
        return self.num_layers * per_layer + v * h * (1 if self.tie_embeddings else 2) + h


PRESETS = {
    "llama3-8b": ModelConfig(),
    "llama3-70b": ModelConfig(name="llama3-70b", hidden_size=8192, num_layers=80, num_heads=64, num_kv_heads=8,
                              intermediate_size=28672),
    "qwen2.5-7b": ModelConfig(name="qwen2.5-7b", hidden_size=3584, num_layers=28, num_heads=28, num_kv_heads=4,
                              intermediate_size=18944, vocab_size=152064, rope_theta=1e6, rms_eps=1e-6, max_position=32768,
                              qkv_bias=True),
    # small shapes for tests: every dimension still meets the kernels' divisibility rules
    "tiny": ModelConfig(name="tiny", hidden_size=512, num_layers=2, num_heads=8, num_kv_heads=2, intermediate_size=1024,
                        vocab_size=2048, max_position=512),
    "tiny-bias": ModelConfig(name="tiny-bias", hidden_size=512, num_layers=2, num_heads=8, num_kv_heads=4, intermediate_size=1024,
                             vocab_size=2048, max_position=512, qkv_bias=True, rope_theta=1e4),
}


def get_config(name: str) -> ModelConfig:
    import copy
    return copy.deepcopy(PRESETS[name])


def from_hf_config(path: str) -> ModelConfig:
    """Read an HF ``config.json`` (Llama / Qwen2 families)."""
    with open(path) as f:
        c = json.load(f)
    heads = c["num_attention_heads"]
    return ModelConfig(
        name=c.get("_name_or_path", c.get("model_type", "hf")),
        hidden_size=c["hidden_size"], num_layers=c["num_hidden_layers"], num_heads=heads,
        num_kv_heads=c.get("num_key_value_heads", heads), head_dim=c.get("head_dim", c["hidden_size"] // heads),
        intermediate_size=c["intermediate_size"], vocab_size=c["vocab_size"], rope_theta=c.get("rope_theta", 1e4),
        rms_eps=c.get("rms_norm_eps", 1e-5), max_position=c.get("max_position_embeddings", 8192),
        qkv_bias=c.get("attention_bias", c.get("model_type") == "qwen2"), tie_embeddings=c.get("tie_word_embeddings", False),
        rope_scaling=c.get("rope_scaling"))


# ---- Nubosun: selective-scan and latent-attention layers over several residual streams ------------------------------------
@dataclass
class MambaSpec:
    inner: int
    state: int
    dt_rank: int
    conv: int                              # taps of the causal convolution, the current token's included


@dataclass
class RotationSpec:
    dims: int
    base: float
    scaling: Optional[dict] = None         # YaRN: factor, original, fast, slow


@dataclass
class LatentSpec:
    heads: int
    dim: int                               # unrotated query / key dimensions per head
    rot_dim: int                           # rotated ones; the key's rotated part is shared by all heads
    vdim: int
    kv_rank: int                           # size of the cached latent
    scale: float
    rot: RotationSpec = None
    q_rank: Optional[int] = None           # size of the queries' latent (None: queries come from the input itself)
    window: int = 0                        # a query sees the last `window` keys, its own included (0: no such limit)


@dataclass
class ClampedGluSpec:
    ff: int
    limit: float
    slope: float = 1.702                   # of the sigmoid gate


@dataclass
class LayerSpec:
    mixer: Union[MambaSpec, LatentSpec]
    mlp: Optional[ClampedGluSpec] = None


@dataclass
class NubosunConfig:
    name: str
    vocab_size: int
    hidden_size: int
    layers: List[LayerSpec]
    streams: int = 1
    embedding_scale: float = 1.0
    rms_eps: float = 1e-5
    logit_softcap: Optional[float] = None
    loop: Optional[tuple] = None           # (start, stop, times): layers start .. stop-1 run `times` times in a row

    def __post_init__(self):
        if self.loop is not None:
            a, b, n = self.loop
            if not (0 <= a <= b <= len(self.layers) and n >= 0):
                raise ValueError(f"loop {self.loop} does not fit {len(self.layers)} layers")
        if not 1 <= self.streams <= 8:
            raise ValueError(f"{self.streams} residual streams: 1 to 8 are supported")

    def check_tp(self, tp: int) -> None:
        if tp != 1:
            raise ValueError("Nubosun models run on one GPU (no tensor-parallel sharding of the scan and the latent cache)")

    @property
    def runs(self) -> List[int]:
        """Layer index of every layer run, in order; each run has a cache or state of its own."""
        n = list(range(len(self.layers)))
        if self.loop is None:
            return n
        a, b, times = self.loop
        return n[:a] + n[a:b] * times + n[b:]

    @property
    def num_layers(self) -> int:
        return len(self.runs)

    def param_count(self) -> int:
        from ..utils.weights import tensor_shapes
        total = 0
        for shape in tensor_shapes(self).values():
            k = 1
            for d in shape:
                k *= d
            total += k
        return total


def parse_nubosun_config(c: dict) -> NubosunConfig:
    """``config.json`` of a Nubosun checkpoint."""
    layers = []
    for i, e in enumerate(c["layers"]):
        m = e["mixer"]
        if e["type"] == "mamba1":
            mixer = MambaSpec(inner=m["inner"], state=m["state"], dt_rank=m["dt_rank"], conv=m["conv"])
        elif e["type"] == "latent_attention":
            r = m["rot"]
            if r["dims"] % 2 or not 0 <= r["dims"] <= m["rot_dim"]:
                raise ValueError(f"layer {i}: {r['dims']} rotated dimensions of {m['rot_dim']}")
            mixer = LatentSpec(heads=m["heads"], dim=m["dim"], rot_dim=m["rot_dim"], vdim=m["vdim"], kv_rank=m["kv_rank"], scale=float(m["scale"]),
                               rot=RotationSpec(dims=r["dims"], base=float(r["base"]), scaling=r.get("scaling")))
        else:
            raise ValueError(f"layer {i}: unknown type {e['type']!r}")
        mlp = e.get("mlp")
        if mlp is not None and mlp["kind"] != "dense":
            raise ValueError(f"layer {i}: unknown feed-forward {mlp['kind']!r}")
        layers.append(LayerSpec(mixer, None if mlp is None else ClampedGluSpec(ff=mlp["ff"], limit=float(mlp["limit"]))))
    loop = c.get("loop")
    cap = c.get("logit_softcap")
    return NubosunConfig(name=c.get("name", "nubosun"), vocab_size=c["vocab"], hidden_size=c["width"], layers=layers, streams=c.get("streams", 1),
                         embedding_scale=float(c.get("embedding", {}).get("scale", 1.0)), rms_eps=float(c["norm"]["eps"]),
                         logit_softcap=float(cap) if cap else None,
                         loop=(loop["start"], loop["stop"], loop["times"]) if loop else None)


def nubosun_like(hidden: int, layers: int, ff: int, heads: int, vocab: int, head_dim: int = 128, kv_rank: int = 512, state: int = 16,
                 attention_every: int = 2, streams: int = 2, name: str = "nubosun") -> NubosunConfig:
    """A Nubosun of ordinary proportions (inner = 2 x width, dt_rank = width / 16, four taps, half of head_dim rotated): a latent-
    attention layer with a feed-forward after every ``attention_every`` - 1 selective-scan layers with one."""
    lay = []
    for i in range(layers):
        if (i + 1) % attention_every:
            mixer = MambaSpec(inner=2 * hidden, state=state, dt_rank=hidden // 16, conv=4)
        else:
            mixer = LatentSpec(heads=heads, dim=head_dim, rot_dim=head_dim // 2, vdim=head_dim, kv_rank=kv_rank, scale=(1.5 * head_dim) ** -0.5,
                               rot=RotationSpec(head_dim // 2, 5e5, {"factor": 4.0, "original": 2048, "fast": 32.0, "slow": 1.0}))
        lay.append(LayerSpec(mixer, ClampedGluSpec(ff=ff, limit=7.0)))
    return NubosunConfig(name=name, vocab_size=vocab, hidden_size=hidden, layers=lay, streams=streams, logit_softcap=30.0)


# ---- Tinapel: gated linear attention, WKV and key-as-value attention beside mixtures of experts ------------------------------
@dataclass
class GlaSpec:
    heads: int
    dim: int                               # key channels per head
    vdim: int
    tau: float                             # decay = sigmoid(z)^(1 / tau)
    decay_rank: Optional[int] = None       # of the low-rank decay projection; None: the checkpoint's tensors tell


@dataclass
class WkvSpec:
    heads: int
    dim: int                               # key and value channels per head
    decay_rank: Optional[int] = None


@dataclass
class SharedKvSpec:
    """Attention whose values are the keys before their norm: one cached row per token and key head serves as both."""
    heads: int
    kv_heads: int
    dim: int
    scale: float
    softcap: Optional[float] = None
    temp_coef: float = 0.0                 # query factor at position p: 1 + coef * ln(floor((p + 1) / every) + 1)
    temp_every: float = 1.0


@dataclass
class MoeSpec:
    experts: int
    top: int
    ff: int                                # of an expert
    scale: float = 1.0                     # on the normalised weights of the chosen experts
    shared_ff: Optional[int] = None        # of the expert that every token uses


@dataclass
class ParallelLayerSpec:
    mixer: Union[GlaSpec, WkvSpec, SharedKvSpec]
    mlp: Optional[MoeSpec] = None


@dataclass
class LoopSpec:
    start: int
    stop: int
    times: int


@dataclass
class TinapelConfig:
    name: str
    vocab_size: int
    hidden_size: int
    layers: List[ParallelLayerSpec]
    embedding_scale: float = 1.0
    rms_eps: float = 1e-6
    loop: Optional[LoopSpec] = None

    def __post_init__(self):
        lp = self.loop
        if lp is not None and not (0 <= lp.start < lp.stop <= len(self.layers) and lp.times >= 0):
            raise ValueError(f"loop {lp} does not fit {len(self.layers)} layers")
        for i, lay in enumerate(self.layers):
            m = lay.mixer
            if isinstance(m, SharedKvSpec) and m.heads % m.kv_heads:
                raise ValueError(f"layer {i}: {m.heads} query heads on {m.kv_heads} key heads")
            if lay.mlp is not None and not 1 <= lay.mlp.top <= lay.mlp.experts:
                raise ValueError(f"layer {i}: {lay.mlp.top} of {lay.mlp.experts} experts")

    def check_tp(self, tp: int) -> None:
        if tp != 1:
            raise ValueError("Tinapel models run on one GPU (no tensor-parallel sharding of the recurrent states and the shared cache rows)")

    @property
    def schedule(self) -> List[tuple]:
        """(layer, pass) of every layer run in order; pass = number of the loop's pass that begins right before this run, else None."""
        n, lp = len(self.layers), self.loop
        if lp is None:
            return [(i, None) for i in range(n)]
        out = [(i, None) for i in range(lp.start)]
        for t in range(lp.times):
            out += [(i, t if i == lp.start else None) for i in range(lp.start, lp.stop)]
        return out + [(i, None) for i in range(lp.stop, n)]

    @property
    def runs(self) -> List[int]:
        return [i for i, _ in self.schedule]

    @property
    def num_layers(self) -> int:
        return len(self.schedule)

    def param_count(self) -> int:
        from ..utils.weights import tensor_shapes
        return sum(math.prod(s) for s in tensor_shapes(self).values())


def _parse_moe(i: int, c: Optional[dict]) -> Optional[MoeSpec]:
    if c is None:
        return None
    if c.get("kind") != "moe":
        raise ValueError(f"layer {i}: unknown feed-forward {c.get('kind')!r}")
    r, shared = c["router"], c.get("shared")
    return MoeSpec(experts=r["experts"], top=r["top"], ff=c["expert"]["ff"], scale=float(r.get("scale", 1.0)), shared_ff=shared["ff"] if shared else None)


def parse_tinapel_config(c: dict) -> TinapelConfig:
    """``config.json`` of a Tinapel checkpoint."""
    layers = []
    for i, e in enumerate(c["layers"]):
        m = e["mixer"]
        if e["type"] == "gla":
            mixer = GlaSpec(heads=m["heads"], dim=m["dim"], vdim=m["vdim"], tau=float(m["tau"]))
        elif e["type"] == "wkv":
            mixer = WkvSpec(heads=m["heads"], dim=m["dim"])
        elif e["type"] == "attention":
            if m.get("vdim", m["dim"]) != m["dim"]:
                raise ValueError(f"layer {i}: values are keys, but have {m['vdim']} channels of {m['dim']}")
            temp, cap = m.get("q_temp"), m.get("softcap")
            mixer = SharedKvSpec(heads=m["heads"], kv_heads=m.get("kv_heads", m["heads"]), dim=m["dim"], scale=float(m["scale"]),
                                 softcap=float(cap) if cap else None, temp_coef=float(temp["coef"]) if temp else 0.0,
                                 temp_every=float(temp["every"]) if temp else 1.0)
        else:
            raise ValueError(f"layer {i}: unknown type {e['type']!r}")
        layers.append(ParallelLayerSpec(mixer, _parse_moe(i, e.get("mlp"))))
    lp = c.get("loop")
    return TinapelConfig(name=c.get("name", "tinapel"), vocab_size=c["vocab"], hidden_size=c["width"], layers=layers,
                         embedding_scale=float(c.get("embedding", {}).get("scale", 1.0)), rms_eps=float(c["norm"]["eps"]),
                         loop=LoopSpec(lp["start"], lp["stop"], lp["times"]) if lp and lp["stop"] > lp["start"] else None)


def tinapel_like(hidden: int, layers: int, ff: int, heads: int, kv_heads: int, vocab: int, head_dim: int = 128, experts: int = 8, top: int = 2,
                 name: str = "tinapel") -> TinapelConfig:
    """A Tinapel of ordinary proportions: layers in turn gated linear attention, WKV and attention; a token uses a shared expert of half of
    ``ff`` and ``top`` experts that make up the other half, so that it meets as many feed-forward weights as in a dense model of ``ff``."""
    kinds = (lambda: GlaSpec(heads=heads, dim=head_dim, vdim=head_dim, tau=16.0, decay_rank=64), lambda: WkvSpec(heads=heads, dim=head_dim, decay_rank=64),
             lambda: SharedKvSpec(heads=heads, kv_heads=kv_heads, dim=head_dim, scale=head_dim ** -0.5, softcap=50.0, temp_coef=0.1, temp_every=4096))
    lay = [ParallelLayerSpec(kinds[i % 3](), MoeSpec(experts=experts, top=top, ff=ff // (2 * top), scale=1.0, shared_ff=ff // 2)) for i in range(layers)]
    return TinapelConfig(name=name, vocab_size=vocab, hidden_size=hidden, layers=lay)


# ---- Bobarax: fixed-decay recurrences, windowed and chunked attention, a norm before and behind every sublayer -----------------------
@dataclass
class LightningSpec:
    heads: int
    dim: int                               # key channels per head
    vdim: int
    decay: List[float] = field(default_factory=list)   # one constant per head


@dataclass
class PairedAttentionSpec:
    """Grouped-query attention with one cached row (key, value) per token and key head; queries and keys are normed over the whole projection."""
    heads: int
    kv_heads: int
    dim: int
    vdim: int
    scale: float
    softcap: Optional[float] = None
    window: int = 0                        # a query sees the last `window` keys, its own included (0: no such limit)
    chunk: int = 0                         # a query sees the keys of its own block of `chunk` positions (0: no such limit)
    rot: Optional[RotationSpec] = None     # None: positions do not enter the scores
    gated: bool = False                    # sigmoid gate on the result
    kv_from: Optional[int] = None          # keys and values of that layer instead of its own


@dataclass
class GatedMlpSpec:
    ff: int                                # relu(gate) * up


@dataclass
class TableMoeSpec:
    """Mixture of experts whose choice is looked up by token id; the chosen ones weigh the same."""
    experts: int
    top: int
    ff: int
    limit: float                           # of the experts' clamped gated unit
    slope: float = 1.702


@dataclass
class SandwichLayerSpec:
    mixer: Union[LightningSpec, PairedAttentionSpec]
    mlp: Optional[Union[GatedMlpSpec, TableMoeSpec]] = None


@dataclass
class BobaraxConfig:
    name: str
    vocab_size: int
    hidden_size: int
    layers: List[SandwichLayerSpec]
    residual_mult: float = 1.0
    logit_scale: float = 1.0
    rms_eps: float = 1e-5

    def __post_init__(self):
        for i, lay in enumerate(self.layers):
            m, f = lay.mixer, lay.mlp
            if isinstance(m, LightningSpec):
                if len(m.decay) != m.heads or not all(0.0 <= a <= 1.0 for a in m.decay):
                    raise ValueError(f"layer {i}: {len(m.decay)} decays (each 0 to 1) for {m.heads} heads")
            else:
                if m.kv_heads < 1 or m.heads % m.kv_heads:
                    raise ValueError(f"layer {i}: {m.heads} query heads on {m.kv_heads} key heads")
                if m.window < 0 or m.chunk < 0 or (m.window and m.chunk):
                    raise ValueError(f"layer {i}: a window of {m.window} and chunks of {m.chunk} positions")
                if m.rot is not None and (m.rot.dims % 2 or not 0 <= m.rot.dims <= m.dim):
                    raise ValueError(f"layer {i}: {m.rot.dims} rotated dimensions of {m.dim}")
                if m.kv_from is not None:
                    j = m.kv_from
                    s = self.layers[j].mixer if 0 <= j < i else None
                    if not isinstance(s, PairedAttentionSpec) or s.kv_from is not None or (s.kv_heads, s.dim, s.vdim, s.rot) != (m.kv_heads, m.dim, m.vdim, m.rot):
                        raise ValueError(f"layer {i}: layer {j} has no keys and values that fit")
            if isinstance(f, TableMoeSpec) and not 1 <= f.top <= f.experts:
                raise ValueError(f"layer {i}: {f.top} of {f.experts} experts")

    def check_tp(self, tp: int) -> None:
        if tp != 1:
            raise ValueError("Bobarax models run on one GPU (no tensor-parallel sharding of the recurrent states and the paired cache rows)")

    @property
    def num_layers(self) -> int:
        return len(self.layers)

    def param_count(self) -> int:
        from ..utils.weights import tensor_shapes
        return sum(math.prod(s) for s in tensor_shapes(self).values())


def parse_bobarax_config(c: dict) -> BobaraxConfig:
    """``config.json`` of a Bobarax checkpoint."""
    layers = []
    for i, e in enumerate(c["layers"]):
        m, f, kind = e["mixer"], e.get("mlp"), e["type"]
        if kind == "lightning":
            mixer = LightningSpec(heads=m["heads"], dim=m["dim"], vdim=m["vdim"], decay=[float(a) for a in m["decay"]])
        elif kind in ("attention", "attention_2"):
            rot, cap, mask = m.get("rot") if kind == "attention_2" else None, m.get("softcap"), m.get("mask") or {"size": 0}
            mixer = PairedAttentionSpec(heads=m["heads"], kv_heads=m.get("kv_heads", m["heads"]), dim=m["dim"], vdim=m.get("vdim", m["dim"]), scale=float(m["scale"]),
                                        softcap=float(cap) if cap else None, window=mask["size"] if kind == "attention_2" else 0,
                                        chunk=mask["size"] if kind == "attention" else 0, rot=RotationSpec(rot["dims"], float(rot["base"])) if rot else None,
                                        gated=kind == "attention_2", kv_from=m.get("kv_from"))
        else:
            raise ValueError(f"layer {i}: unknown type {kind!r}")
        if f is None:
            mlp = None
        elif f.get("kind") == "dense":
            mlp = GatedMlpSpec(ff=f["ff"])
        elif f.get("kind") == "moe":
            mlp = TableMoeSpec(experts=f["router"]["experts"], top=f["router"]["top"], ff=f["expert"]["ff"], limit=float(f["expert"]["limit"]))
        else:
            raise ValueError(f"layer {i}: unknown feed-forward {f.get('kind')!r}")
        layers.append(SandwichLayerSpec(mixer, mlp))
    return BobaraxConfig(name=c.get("name", "bobarax"), vocab_size=c["vocab"], hidden_size=c["width"], layers=layers, residual_mult=float(c.get("residual_mult", 1.0)),
                         logit_scale=float(c.get("logit_scale", 1.0)), rms_eps=float(c["norm"]["eps"]))


def bobarax_like(hidden: int, layers: int, ff: int, heads: int, kv_heads: int, vocab: int, head_dim: int = 128, experts: int = 8, top: int = 2,
                 window: int = 4096, chunk: int = 8192, name: str = "bobarax") -> BobaraxConfig:
    """A Bobarax of ordinary proportions: layers in turn lightning, windowed attention, lightning, chunked attention, every fourth windowed layer with the keys
    and values of the one before; every other feed-forward a mixture of experts of which a token meets ``ff`` in all, the others dense."""
    lay = []
    for i in range(layers):
        if i % 2 == 0:
            mixer = LightningSpec(heads, head_dim, head_dim, [math.exp(-2.0 ** (-0.5 - 8.0 * h / heads)) for h in range(heads)])
        elif i % 4 == 1:
            mixer = PairedAttentionSpec(heads, kv_heads, head_dim, head_dim, head_dim ** -0.5, window=window, rot=RotationSpec(head_dim // 2, 5e5), gated=True,
                                        kv_from=i - 4 if i % 16 == 13 else None)
        else:
            mixer = PairedAttentionSpec(heads, kv_heads, head_dim, head_dim, head_dim ** -0.5, softcap=50.0, chunk=chunk)
        lay.append(SandwichLayerSpec(mixer, TableMoeSpec(experts, top, ff // top, 7.0) if i // 2 % 2 else GatedMlpSpec(ff)))
    return BobaraxConfig(name=name, vocab_size=vocab, hidden_size=hidden, layers=lay, residual_mult=0.8, logit_scale=hidden ** -0.5)


# ---- Lugizen: delta-rule recurrences, attention with norms per head, windowed latent attention; norms behind the sublayers -------------------
@dataclass
class ChannelDeltaSpec:
    """Gated delta rule with a decay per head and key channel."""
    heads: int
    kv_heads: int                          # heads of queries and keys
    dim: int
    vdim: int
    conv: int                              # taps of the convolutions of q, k and v, the current token's included
    decay_rank: Optional[int] = None       # of the low-rank decay and gate projections; None: the checkpoint's tensors tell
    gate_rank: Optional[int] = None


@dataclass
class HeadAttentionSpec:
    """Grouped-query attention over paired cache rows; queries and keys are normed per head without weights, scores scaled by a number per head."""
    heads: int
    kv_heads: int
    dim: int
    vdim: int
    scale: float
    rot: Optional[RotationSpec] = None
    v_mix: bool = False                    # values are mixed with those of the first such layer


@dataclass
class GeluMlpSpec:
    ff: int                                # down(gelu(up)), tanh form


@dataclass
class PostNormLayerSpec:
    mixer: Union[ChannelDeltaSpec, HeadAttentionSpec, LatentSpec]
    mlp: Optional[Union[GeluMlpSpec, MoeSpec]] = None


@dataclass
class LugizenConfig:
    name: str
    vocab_size: int
    hidden_size: int
    layers: List[PostNormLayerSpec]
    canon_taps: int = 4                    # of the convolution over what a mixer reads
    rms_eps: float = 1e-5

    def __post_init__(self):
        if self.canon_taps < 1:
            raise ValueError(f"a convolution of {self.canon_taps} taps")
        first = None
        for i, lay in enumerate(self.layers):
            m, f = lay.mixer, lay.mlp
            if isinstance(m, LatentSpec):
                if m.window < 0 or not m.q_rank or m.rot is None:
                    raise ValueError(f"layer {i}: a window of {m.window}, a query latent of {m.q_rank}, rotation {m.rot}")
            else:
                if m.kv_heads < 1 or m.heads % m.kv_heads:
                    raise ValueError(f"layer {i}: {m.heads} heads on {m.kv_heads} key heads")
                if isinstance(m, ChannelDeltaSpec) and m.conv < 1:
                    raise ValueError(f"layer {i}: a convolution of {m.conv} taps")
                if isinstance(m, HeadAttentionSpec):
                    if m.rot is not None and (m.rot.dims % 2 or not 0 <= m.rot.dims <= m.dim):
                        raise ValueError(f"layer {i}: {m.rot.dims} rotated dimensions of {m.dim}")
                    if m.v_mix:
                        first = first or m
                        if (m.kv_heads, m.vdim) != (first.kv_heads, first.vdim):
                            raise ValueError(f"layer {i}: values of {m.kv_heads} x {m.vdim} do not mix with {first.kv_heads} x {first.vdim}")
            if isinstance(f, MoeSpec) and not 1 <= f.top <= f.experts:
                raise ValueError(f"layer {i}: {f.top} of {f.experts} experts")

    def check_tp(self, tp: int) -> None:
        if tp != 1:
            raise ValueError("Lugizen models run on one GPU (no tensor-parallel sharding of the recurrent states and the latent cache)")

    @property
    def num_layers(self) -> int:
        return len(self.layers)

    def param_count(self) -> int:
        from ..utils.weights import tensor_shapes
        return sum(math.prod(s) for s in tensor_shapes(self).values())


def parse_lugizen_config(c: dict) -> LugizenConfig:
    """``config.json`` of a Lugizen checkpoint."""
    layers = []
    for i, e in enumerate(c["layers"]):
        m, f, kind = e["mixer"], e.get("mlp"), e["type"]
        rot = m.get("rot")
        rot = RotationSpec(rot["dims"], float(rot["base"])) if rot else None
        if kind == "channel_delta":
            mixer = ChannelDeltaSpec(heads=m["heads"], kv_heads=m.get("kv_heads", m["heads"]), dim=m["dim"], vdim=m["vdim"], conv=m["conv"])
        elif kind == "attention":
            mixer = HeadAttentionSpec(heads=m["heads"], kv_heads=m.get("kv_heads", m["heads"]), dim=m["dim"], vdim=m.get("vdim", m["dim"]), scale=float(m["scale"]), rot=rot,
                                      v_mix=bool(m.get("v_mix", False)))
        elif kind == "latent_attention":
            if rot is None or rot.dims != m["rot_dim"]:
                raise ValueError(f"layer {i}: {rot and rot.dims} rotated dimensions of {m['rot_dim']}")
            mixer = LatentSpec(heads=m["heads"], dim=m["dim"], rot_dim=m["rot_dim"], vdim=m["vdim"], kv_rank=m["kv_rank"], scale=float(m["scale"]), rot=rot,
                               q_rank=m["q_rank"], window=(m.get("mask") or {"size": 0})["size"])
        else:
            raise ValueError(f"layer {i}: unknown type {kind!r}")
        mlp = GeluMlpSpec(ff=f["ff"]) if f is not None and f.get("kind") == "dense" else _parse_moe(i, f)
        layers.append(PostNormLayerSpec(mixer, mlp))
    return LugizenConfig(name=c.get("name", "lugizen"), vocab_size=c["vocab"], hidden_size=c["width"], layers=layers, canon_taps=c["canon"]["taps"],
                         rms_eps=float(c["norm"]["eps"]))


def lugizen_like(hidden: int, layers: int, ff: int, heads: int, kv_heads: int, vocab: int, head_dim: int = 128, experts: int = 8, top: int = 2, window: int = 4096,
                 rank: int = 64, name: str = "lugizen") -> LugizenConfig:
    """A Lugizen of ordinary proportions: every other layer a delta-rule recurrence, between them in turn windowed latent attention and attention; every other pair of
    feed-forwards a mixture of experts of which a token meets ``ff`` in all, the others dense with as many weights (two matrices for three)."""
    kv_rank, rot = 4 * head_dim, head_dim // 2
    kinds = (lambda: ChannelDeltaSpec(heads, heads, head_dim, head_dim, 4, rank, rank),
             lambda: LatentSpec(heads=heads, dim=head_dim, rot_dim=rot, vdim=head_dim, kv_rank=kv_rank, scale=(1.5 * head_dim) ** -0.5, rot=RotationSpec(rot, 5e5),
                                q_rank=3 * kv_rank, window=window),
             lambda: ChannelDeltaSpec(heads, heads, head_dim, head_dim, 4, rank, rank),
             lambda: HeadAttentionSpec(heads, kv_heads, head_dim, head_dim, head_dim ** -0.5, RotationSpec(rot, 5e5), True))
    lay = [PostNormLayerSpec(kinds[i % 4](), MoeSpec(experts, top, ff // top) if i // 2 % 2 else GeluMlpSpec(3 * ff // 2)) for i in range(layers)]
    return LugizenConfig(name=name, vocab_size=vocab, hidden_size=hidden, layers=lay)


PRESETS["nubosun-8b"] = nubosun_like(4096, 32, 14336, 32, 128256, name="nubosun-8b")
PRESETS["nubosun-2k"] = nubosun_like(2048, 16, 7168, 16, 32768, name="nubosun-2k")
PRESETS["llama3-2k"] = ModelConfig(name="llama3-2k", hidden_size=2048, num_layers=16, num_heads=16, num_kv_heads=4, intermediate_size=7168,
                                   vocab_size=32768)
PRESETS["tinapel-8b"] = tinapel_like(4096, 32, 14336, 32, 8, 128256, name="tinapel-8b")
PRESETS["tinapel-2k"] = tinapel_like(2048, 16, 7168, 16, 4, 32768, name="tinapel-2k")
PRESETS["bobarax-8b"] = bobarax_like(4096, 32, 14336, 32, 8, 128256, name="bobarax-8b")
PRESETS["bobarax-2k"] = bobarax_like(2048, 16, 7168, 16, 4, 32768, name="bobarax-2k")
PRESETS["lugizen-8b"] = lugizen_like(4096, 32, 14336, 32, 8, 128256, name="lugizen-8b")
PRESETS["lugizen-2k"] = lugizen_like(2048, 16, 7168, 16, 4, 32768, name="lugizen-2k")
