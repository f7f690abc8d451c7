"""The engine of the hybrid float models: the same contract as the integer engines (token rows over a paged cache,
`forward` / `logits` / `check`), so `decode.Session`, `generate`, the CUDA-graph decoders and the integer sampler serve
it unchanged. Logits leave as fixed-point integers at 24 bits, rounded once from the 32-bit accumulators.

The residual stream is float [rows, D]. Caches per layer: pages of latent rows (attention) or one float state per
sequence (recurrent layers), indexed by the block table and its row number."""

import torch

from .. import _native as nv
from ..engine_base import TokenRowEngine
from . import ops
from .layers import DenseFF, ExpertsFF, LatentAttention, MinGRU, Step
from .spec import DenseSpec, ExpertsSpec, LatentAttentionSpec, MinGRUSpec

MIXERS = {MinGRUSpec: MinGRU, LatentAttentionSpec: LatentAttention}
FEED_FORWARDS = {DenseSpec: DenseFF, ExpertsSpec: ExpertsFF}


class HybridEngine(TokenRowEngine):
    FR = 24
    page = 64               # the attention kernel's key block: one copy per page and column block
    tiles_from = 0

    def __init__(self, spec, weights, dev="cuda", dtype="bfloat16", n_layers=None):
        """spec: ModelSpec; weights: {'embed', 'head', 'final': (w, b), 'layers': [{'norm1', 'norm2': (w, b), 'mixer',
        'ff': dicts of the mechanism}]} as tensors (a design's `read_weights`)."""
        self.dev, self.spec = torch.device(dev), spec
        self.dtype, _ = ops.DTYPES[dtype]
        self.D, self.V = spec.width, spec.vocab
        self.L = len(spec.layers) if n_layers is None else n_layers
        vec = lambda pair: tuple(t.to(self.dev).float().contiguous() for t in pair)
        make = lambda table, s, w: None if s is None else table[type(s)](w, s, self.D, self.dtype, self.dev)
        self.embed = weights["embed"].to(self.dev).to(self.dtype).contiguous()
        self.head = ops.pack(weights["head"], self.dtype, self.dev)
        self.final = vec(weights["final"])
        self.layers = []
        for s, w in zip(spec.layers[: self.L], weights["layers"]):
            self.layers.append((vec(w["norm1"]), make(MIXERS, s.mixer, w["mixer"]),
                                vec(w["norm2"]) if s.ff is not None else None, make(FEED_FORWARDS, s.ff, w["ff"])))
        counters = max([ff.counters for _, _, _, ff in self.layers if ff is not None], default=0)
        self.counts = torch.zeros(max(1, counters), dtype=torch.int32, device=self.dev)
        self._ln = None

    @property
    def ln(self):
        """The sampler's logarithm table (built on first use)."""
        if self._ln is None:
            from ..exact.consts import FL, ln_table
            self._ln = ln_table(FL, self.dev)
        return self._ln

    def check(self):
        """Raises `_native.DeviceWaitError` when a bounded device-side wait gave up since the last clear."""
        nv.check_device_status(nv.float_device_status)

    def new_cache(self, n_seqs, n_blocks, bs):
        return [mixer.new_cache(n_seqs, n_blocks, bs) for _, mixer, _, _ in self.layers]

    def tile_table(self, runs, bs):
        per = [mixer.spec.heads for _, mixer, _, _ in self.layers if isinstance(mixer, LatentAttention)]
        if not per or self.dtype != torch.bfloat16:
            return None
        n = min(nv.float_lib().bxf_latent_attention_tile(h) for h in per)
        return torch.tensor([[r, t0 + s, min(n, ql - s)] for r, t0, ql, _ in runs for s in range(0, ql, n)],
                            dtype=torch.int32).reshape(-1, 3)

    def forward(self, caches, ids, pos, slot, bt, rmap, tiles=None):
        """ids, pos, slot [N]: the step's tokens (slot < 0: padding, written to page 0); caches: `new_cache`; bt
        [*, blocks] block table, rmap [N] the table row of each token, also the slot of its recurrent states. Rows of a
        sequence are consecutive and in position order; a row at position 0 starts from a zero state. Returns the
        residual stream float [N, D]."""
        ids, pos, slot, seq = ids.long().contiguous(), pos.long().contiguous(), slot.long().contiguous(), rmap.long().contiguous()
        M = ids.shape[0]
        step = Step(pos, slot, seq, bt, ops.row_flags(seq, slot, pos), tiles)
        x = torch.empty(M, self.D, dtype=torch.float32, device=self.dev)
        h = torch.empty(M, ops.pad8(self.D), dtype=self.dtype, device=self.dev)
        due, start = None, dict(ids=ids, embed=self.embed)
        for (norm1, mixer, norm2, ff), cache in zip(self.layers, caches):
            ops.norm(x, *norm1, self.spec.eps, h, experts=due, **start)
            due, start = None, {}
            mixer.run(step, h, x, cache)
            if ff is not None:
                counts = self.counts[: ff.counters] if ff.counters else None
                ops.norm(x, *norm2, self.spec.eps, h, zero=counts)
                due = ff.run(h, x, counts)
        if due is not None or start:
            ops.norm(x, None, None, self.spec.eps, experts=due, **start)
        return x

    def _head(self, x, out_type, dtype):
        h = torch.empty(x.shape[0], ops.pad8(self.D), dtype=self.dtype, device=self.dev)
        ops.norm(x, *self.final, self.spec.eps, h)
        out = torch.empty(x.shape[0], self.V, dtype=dtype, device=self.dev)
        ops.linear(self.head, h, x.shape[0], self.V, self.D, ops.store(out, self.V, self.V, out_type=out_type))
        return out

    def logits(self, x):
        """Final residual rows [M, D] -> int64 logits [M, V] at 24 bits."""
        return self._head(x.contiguous(), ops.OUT_I64, torch.int64)

    def logits_float(self, x):
        return self._head(x.contiguous(), ops.OUT_F32, torch.float32)
