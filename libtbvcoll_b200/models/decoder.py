"""What the decoders with one fp32 residual stream and carried state share: flat activation storage, the cut of long segments, routed experts, the output head."""
from __future__ import annotations

from typing import Dict

import torch

from .. import ops
from ..engine.batch import StepBatch
from .latent import pad16  # noqa: F401  (also for the decoders)


class StreamDecoder:
    # portions of at most this many tokens take the attention's rows form
    ROWS_FORM_MAX = 32
    SCAN_CHUNK = 16                        # tokens per chunk of the recurrences
    uses_state = True
    expands_context = False
    context_window = 0                     # latent attention: no layer looks further back than this many keys (0: no such limit)
    head_weight = "embed"

    cfg: object
    w: Dict[str, torch.Tensor]
    dtype: torch.dtype
    device: torch.device
    max_batch: int
    Wp: int
    scan_heads: int                        # fewest heads of a recurrent layer (0: none)
    _flat: Dict[str, torch.Tensor]

    @staticmethod
    def attn_cta_slots(splits: int, sms: int) -> int:
        """CTAs of the rows kernel that run at once: two per SM, but clusters of eight find only about four fifths of the places."""
        return 2 * sms if splits < 8 else 2 * sms * 4 // 5

    def scan_group_rows(self, rows) -> int:
        """Rows per group of the chunked recurrence for segments of the given lengths; 0: the sequential (32-bit) kernel.  Cutting a segment costs a
        second pass over its keys and values, so it is done only as far as the GPU would otherwise be short of CTAs."""
        if self.dtype is not torch.bfloat16 or not self.scan_heads:
            return 0
        sms, c = torch.cuda.get_device_properties(self.device).multi_processor_count, self.SCAN_CHUNK
        fair = max(256, -(-int(rows.sum()) * self.scan_heads // (2 * sms * c)) * c)
        longest = -(-int(rows.max()) // c) * c
        return longest if 2 * longest <= 3 * fair else fair

    def _buf(self, name: str, rows: int, *shape: int) -> torch.Tensor:
        n = rows
        for s in shape:
            n *= s
        return self._flat[name][:n].view(rows, *shape)

    # -- mixtures of experts whose choice comes from a router ---------------------------------------------------
    def _expert_buffers(self, moes, extra_act: int = 0) -> Dict[str, torch.Tensor]:
        """Flat storage of the specs ``moes`` (``act`` for at least ``extra_act`` columns), and the counters beside it."""
        T, f32, i32 = self.max_tokens, torch.float32, torch.int32
        zeros = lambda n, dt=self.dtype: torch.zeros(n, dtype=dt, device=self.device)
        big = lambda sizes: max(sizes, default=0)
        self.offsets = zeros(big([f.experts for f in moes]) + 1, i32)
        self.counts = zeros(big([f.experts for f in moes]), i32)
        return {
            "router": zeros(T * big([pad16(f.experts) for f in moes]), f32),
            "xp": zeros(T * big([f.top * self.Wp for f in moes])),
            "act": zeros(T * max(extra_act, big([f.top * pad16(f.ff) for f in moes]))),
            "routed": zeros(T * big([f.top * self.Wp for f in moes])),
            "place": zeros(T * big([f.top for f in moes]), i32),
            "choice": zeros(T * big([2 * f.top for f in moes]), i32),
            "weight": zeros(T * big([f.top for f in moes]), f32),
        }

    def _experts(self, b: StepBatch, p: str, f, h: torch.Tensor) -> tuple:
        """The routed experts' results as ``ops.residual`` takes them; ``p``: prefix of their weights, ``f``: experts, top, ff and the weights' scale."""
        w, T = self.w, b.T
        P, fp = T * f.top, pad16(f.ff)
        logits = self._buf("router", T, pad16(f.experts))
        xp, act, routed = self._buf("xp", P, self.Wp), self._buf("act", P, fp), self._buf("routed", P, self.Wp)
        place, weight, off = self._buf("place", T, f.top), self._buf("weight", T, f.top), self.offsets[: f.experts + 1]
        ops.linear(h, w[p + "router"], logits)
        ops.moe_route(logits, h, xp, place, weight, off, self.counts, self._flat["choice"], f.experts, f.scale)
        ops.linear_rows(xp, w[p + "gate_up"], act, off, f.experts, T, glu=ops.SILU_GLU)
        ops.linear_rows(act, w[p + "down"], routed, off, f.experts, T)
        return routed, place, weight

    def _init_head(self) -> None:
        dev, f32, V = self.device, torch.float32, pad16(self.cfg.vocab_size)
        self.Vp = V
        self.hl = torch.zeros(self.max_batch, self.Wp, dtype=self.dtype, device=dev)
        self.logits = torch.zeros(self.max_batch, V, dtype=f32, device=dev)
        self.argmax_ws = ops.argmax_workspace(self.max_batch, dev)
        self.argmax_val = torch.zeros(self.max_batch, dtype=f32, device=dev)

    def _head_rows(self, n: int) -> torch.Tensor:
        """Storage for the normed rows whose logits are wanted (preallocated up to a batch of decoded tokens)."""
        return self.hl[:n] if n <= self.max_batch else torch.empty(n, self.Wp, dtype=self.dtype, device=self.device)

    def _head(self, b: StepBatch, hl: torch.Tensor) -> None:
        """Logits of the rows ``hl`` against the embedding (or the head, where a model has one); greedy tokens and / or the logits themselves to where the batch wants them."""
        n, V = b.n_logits, self.cfg.vocab_size
        logits = self.logits[:n] if n <= self.max_batch else torch.empty(n, self.Vp, dtype=torch.float32, device=self.device)
        ops.linear(hl, self.w[self.head_weight], logits)
        if b.logits_out is not None:
            b.logits_out.copy_(logits[:, :V])
        if b.out_tokens is not None:
            assert n <= self.max_batch
            ops.argmax(logits[:, :V], self.argmax_ws, 0, self.argmax_val[:n], b.out_tokens[:n])
