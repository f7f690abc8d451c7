"""The engine of the hybrid float models: the same contract as the integer engines (token rows over a paged cache,
`forward` / `logits` / `check`), so `decode.Session`, `generate`, the CUDA-graph decoders and the integer sampler serve
it unchanged. Logits leave as fixed-point integers at 24 bits, rounded once from the 32-bit accumulators.

The residual (`residual.py`) is float: one stream or several. Caches per layer run: pages of rows (attention) or float states
and convolution inputs per sequence (recurrent layers), indexed by the block table and its row number. A layer that runs
several times in a row shares its weights and has a cache per run."""

import torch

from .. import _native as nv
from ..engine_base import TokenRowEngine
from . import ops
from .layers import GLA, Attention, DenseFF, ExpertsFF, GatedFF, LatentAttention, Mamba2, MinGRU, Step, Tiles
from .residual import LayerNormResidual, StreamsResidual
from .spec import (AttentionSpec, DenseSpec, ExpertsSpec, GatedSpec, GLASpec, LatentAttentionSpec, Mamba2Spec, MinGRUSpec)

MIXERS = {MinGRUSpec: MinGRU, LatentAttentionSpec: LatentAttention, AttentionSpec: Attention, Mamba2Spec: Mamba2, GLASpec: GLA}
FEED_FORWARDS = {DenseSpec: DenseFF, GatedSpec: GatedFF, ExpertsSpec: ExpertsFF}


class HybridEngine(TokenRowEngine):
    FR = 24
    page = 64               # the attention kernel's key block: one copy per page and column block
    tiles_from = 0

    def __init__(self, spec, weights, dev="cuda", dtype="bfloat16", n_layers=None):
        """spec: ModelSpec; weights: {'embed', 'head', 'final', 'layers': [{'norm1', 'norm2', 'mixer', 'ff': dicts of the
        mechanism, 'hc1', 'hc2'}]} as tensors (a design's `read_weights`). Norms are (w, b), with streams w around zero;
        'hc<q>' are the dicts 'in', 'out', 'mix' of a sublayer's streams. n_layers: only the first runs."""
        self.dev, self.spec = torch.device(dev), spec
        self.dtype, _ = ops.DTYPES[dtype]
        self.D, self.V = spec.width, spec.vocab
        runs = (tuple(range(len(spec.layers))) if spec.runs is None else spec.runs)[:n_layers]
        self.L = len(runs)
        self.residual = StreamsResidual if spec.streams else LayerNormResidual
        sub = lambda w, q: self.residual.prepare(w[f"norm{q}"], w.get(f"hc{q}"), self.dev)
        make = lambda table, s, w: None if s is None else table[type(s)](w, s, self.D, self.dtype, self.dev)
        self.embed = weights["embed"].to(self.dev).to(self.dtype).contiguous()
        self.head = ops.pack(weights["head"], self.dtype, self.dev)
        self.final = self.residual.prepare(weights["final"], None, self.dev)
        made = {}
        for i in set(runs):
            s, w = spec.layers[i], weights["layers"][i]
            made[i] = (sub(w, 1), make(MIXERS, s.mixer, w["mixer"]), sub(w, 2) if s.ff is not None else None,
                       make(FEED_FORWARDS, s.ff, w["ff"]))
        self.layers = [made[i] for i in runs]
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
        if self.dtype != torch.bfloat16:
            return None
        heads = {mixer.tile_heads for _, mixer, _, _ in self.layers if isinstance(mixer, (LatentAttention, Attention))}
        return Tiles.of(runs, {nv.float_lib().bxf_latent_attention_tile(h) for h in heads})

    def forward(self, caches, ids, pos, slot, bt, rmap, tiles=None):
        """ids, pos, slot [N]: the step's tokens (slot < 0: padding, written to page 0); caches: `new_cache`; bt
        [*, blocks] block table, rmap [N] the table row of each token, also the slot of its recurrent states. Rows of a
        sequence are consecutive and in position order; a row at position 0 starts from a zero state. Returns the
        residual stream float [N, D]."""
        ids, pos, slot, seq = ids.long().contiguous(), pos.long().contiguous(), slot.long().contiguous(), rmap.long().contiguous()
        M = ids.shape[0]
        step = Step(pos, slot, seq, bt, ops.row_flags(seq, slot, pos), tiles)
        res = self.residual(self, M, ids)
        for (sub1, mixer, sub2, ff), cache in zip(self.layers, caches):
            h = res.open(sub1)
            x, add = res.target()
            mixer.run(step, h, x, cache, add)
            if ff is not None:
                counts = self.counts[: ff.counters] if ff.counters else None
                h = res.open(sub2, counts)
                x, add = res.target()
                res.due(ff.run(h, x, counts, add))
        return res.close()

    def _head(self, x, out_type, dtype):
        h = torch.empty(x.shape[0], ops.pad8(self.D), dtype=self.dtype, device=self.dev)
        self.residual.final_norm(x, self.final, self.spec.eps, h)
        out = torch.empty(x.shape[0], self.V, dtype=dtype, device=self.dev)
        scale, cap = self.spec.logit_scale, self.spec.logit_softcap
        act = ("softcap", scale / cap, cap) if cap else ("none", 0.0, 0.0) if scale == 1.0 else ("scale", scale, 0.0)
        ops.linear(self.head, h, x.shape[0], self.V, self.D, ops.store(out, self.V, self.V, *act, out_type=out_type))
        return out

    def logits(self, x):
        """Final residual rows [M, D] -> int64 logits [M, V] at 24 bits."""
        return self._head(x.contiguous(), ops.OUT_I64, torch.int64)

    def logits_float(self, x):
        return self._head(x.contiguous(), ops.OUT_F32, torch.float32)
