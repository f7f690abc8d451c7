"""The layer mechanisms of the hybrid float models: mixers (minGRU, latent attention, grouped-query attention, Mamba-2, gated
linear attention) and feed-forwards (dense, gated, experts).

A mixer owns its packed weights and the shape of its per-layer cache; `run(step, h, x, cache, add)` reads the normed rows h
and adds its output to the rows x, or stores it there. A feed-forward's `run(h, x, counts, add)` does the same and returns
what is still due to x (the experts' outputs, folded into the next norm) or None. Weights arrive as a dict name -> tensor with the
mechanism's own names ('z', 'dq.norm', 'e0.up', ...)."""

import functools
import math
from dataclasses import dataclass, field

import torch

from .. import _native as nv
from . import ops


@dataclass
class Step:
    """The token rows of one forward call (device tensors; rows of a sequence consecutive, in position order)."""
    pos: torch.Tensor           # int64 [M]
    slot: torch.Tensor          # int64 [M] cache slot (negative: padding)
    seq: torch.Tensor           # int64 [M] block-table row = state slot
    bt: torch.Tensor            # [slots, blocks]
    flags: torch.Tensor         # int32 [M] bxf_row_flags
    tiles: object = None        # Tiles of a prompt portion
    turned: dict = field(default_factory=dict)

    def angles(self, freq):
        """(cos, sin) of every row's position times freq, computed once per step and set of frequencies."""
        key = freq.data_ptr()
        if key not in self.turned:
            self.turned[key] = ops.angles(freq, self.pos)
        return self.turned[key]


class Tiles:
    """What the tile kernels of a prompt portion walk: attention tiles int32 [T, 3] (table row, first row, rows) by their
    number of tokens; for the recurrences the runs int32 [R, 3] (first row, rows, first chunk) of its sequences, their chunks
    int32 [C, 2] (first row, rows), the segments [S, 3] (like runs) that long runs are cut into and the spans [R, 3] (first row,
    first segment, segments) of the runs."""

    CHUNK, SEGMENT = 64, 512    # a segment costs two passes over the states: short ones only where rows are few

    def __init__(self, attention, runs, chunks, segments, spans):
        self.attention, self.runs, self.chunks, self.segments, self.spans = attention, runs, chunks, segments, spans

    @classmethod
    def of(cls, runs, sizes):
        """runs = [(table row, first token row, tokens, context length)], sizes: the tile heights in use."""
        table = lambda n: torch.tensor([[r, t0 + s, min(n, ql - s)] for r, t0, ql, _ in runs for s in range(0, ql, n)],
                                       dtype=torch.int32).reshape(-1, 3)
        size = cls.SEGMENT if sum(ql for _, _, ql, _ in runs) >= 4096 else cls.SEGMENT // 2
        per_run, chunks, segments, spans = [], [], [], []
        for _, t0, ql, _ in runs:
            per_run.append([t0, ql, len(chunks)])
            spans.append([t0, len(segments), (ql + size - 1) // size])
            segments += [[t0 + s, min(size, ql - s), len(chunks) + s // cls.CHUNK] for s in range(0, ql, size)]
            chunks += [[t0 + s, min(cls.CHUNK, ql - s)] for s in range(0, ql, cls.CHUNK)]
        tensor = lambda rows, n: torch.tensor(rows, dtype=torch.int32).reshape(-1, n)
        return cls({n: table(n) for n in sizes}, tensor(per_run, 3), tensor(chunks, 2), tensor(segments, 3), tensor(spans, 3))

    def to(self, dev):
        return Tiles({n: t.to(dev) for n, t in self.attention.items()},
                     *(t.to(dev) for t in (self.runs, self.chunks, self.segments, self.spans)))

    def chunked(self, K, V, rows):
        """Whether a recurrence of these sizes runs in chunks: portions of a few rows are shorter row by row."""
        return rows >= 16 * self.runs.shape[0] and nv.float_lib().bxf_recurrence_chunk_rows(0, K, V) == self.CHUNK

    def for_heads(self, heads):
        return self.attention.get(nv.float_lib().bxf_latent_attention_tile(heads))


def _vec(t, dev):
    return t.to(dev).float().contiguous()


@functools.lru_cache(maxsize=None)
def _frequencies(base, dims, dev):
    """base^(-2 i / dims) in double; layers with the same rotation share the tensor."""
    return torch.tensor([base ** (-2.0 * i / dims) for i in range(dims // 2)], dtype=torch.float64, device=dev)


class MinGRU:
    """z, u, g = three products of h; S = (1 - z) S + z candidate(u); x += W_o (S silu(g)). State: float [slots, width]."""

    def __init__(self, w, spec, D, dtype, dev):
        self.spec, self.D = spec, D
        self.w = ops.pack(torch.stack([w["z"], w["x"], w["g"]]), dtype, dev)
        self.bz, self.bx = _vec(w["z.b"], dev), _vec(w["x.b"], dev)
        self.o = ops.pack(w["o"], dtype, dev)
        assert self.w.shape[1] == spec.width

    def new_cache(self, n_seqs, n_blocks, bs):
        return torch.zeros(n_seqs, self.spec.width, dtype=torch.float32, device=self.w.device)

    def run(self, step, h, x, cache, add=True):
        s = ops.min_gru(self.w, self.bz, self.bx, h, self.spec.width, self.D, cache, step.flags, step.seq)
        ops.linear(self.o, s, x.shape[0], self.D, self.spec.width, ops.sublayer_output(x, add))


class LatentAttention:
    """Attention in the latent space: the per-head key matrix is applied to the query instead of to every cached key, the
    value matrix to the attention output, so that a token's cache row [latent | rotated key part] serves all heads."""

    def __init__(self, w, spec, D, dtype, dev):
        self.spec, self.D, self.dtype = spec, D, dtype
        H, dn, dr, R = spec.heads, spec.dim, spec.rot_dim, spec.kv_rank
        if dr < 2 or dr % 2:
            raise ValueError("the rotated part needs an even, positive size")
        self.first = ops.pack(torch.cat([w["dq"], w["dkv"], w["g"]]), dtype, dev)
        self.dq_norm, self.dkv_norm = _vec(w["dq.norm"], dev), _vec(w["dkv.norm"], dev)
        # query rows: every head's unrotated part (padded to 8), then every head's rotated part
        uq = w["uq"].view(H, dn + dr, spec.q_rank)
        self.dnp = ops.pad8(dn)
        nope = torch.zeros(H, self.dnp, spec.q_rank, dtype=uq.dtype, device=uq.device)
        nope[:, :dn] = uq[:, :dn]
        self.uq = ops.pack(torch.cat([nope.view(-1, spec.q_rank), uq[:, dn:].reshape(-1, spec.q_rank)]), dtype, dev)
        self.uk = ops.pack(w["uk"].view(H, dn, R).transpose(1, 2), dtype, dev)          # [H, R, dn]
        self.uv = ops.pack(w["uv"].view(H, spec.vdim, R), dtype, dev)
        self.o = ops.pack(w["o"], dtype, dev)
        self.sink = _vec(w["sink"], dev) if "sink" in w else None
        self.freq = torch.tensor([spec.rot_base ** (-2.0 * i / dr) for i in range(dr // 2)], dtype=torch.float32, device=dev)

    def new_cache(self, n_seqs, n_blocks, bs):
        return torch.zeros(n_blocks, bs, ops.pad8(self.spec.kv_rank + self.spec.rot_dim), dtype=self.dtype,
                           device=self.first.device)

    @property
    def tile_heads(self):
        return self.spec.heads

    def run(self, step, h, x, cache, add=True):
        sp, M, dev = self.spec, x.shape[0], x.device
        H, R, dnp = sp.heads, sp.kv_rank, self.dnp
        n1 = self.first.shape[0]
        y = torch.empty(M, n1, dtype=torch.float32, device=dev)
        ops.linear(self.first, h, M, n1, self.D, ops.store(y, n1, n1, out_type=ops.OUT_F32))
        cq, cs, gate = ops.latent_prepare(y, sp, self.dq_norm, self.dkv_norm, self.freq, step.pos, step.slot, cache)
        qn = torch.empty(M, H * dnp, dtype=self.dtype, device=dev)
        q = torch.empty(M, H, ops.pad8(R + sp.rot_dim), dtype=self.dtype, device=dev)
        ldq = q.shape[2]
        ops.linear(self.uq, cq, M, H * (dnp + sp.rot_dim), sp.q_rank,
                   nv.Epilogue(kind=ops.ROPE, n_main=H * dnp, out=qn.data_ptr(), ldo=H * dnp, cs=cs.data_ptr(),
                               rot_out=q.data_ptr() + R * q.element_size(), ldr=H * ldq, hsr=ldq, rot_dim=sp.rot_dim))
        ops.linear(self.uk, qn, M, R, sp.dim, ops.store(q, H * ldq, R, gso=ldq), groups=H, gsw=R * self.uk.shape[2], gsx=dnp)
        o = ops.latent_attention(q, sp, cache, step.bt, step.seq, step.pos, self.sink,
                                 step.tiles.for_heads(H) if step.tiles is not None else None)
        og = torch.empty(M, ops.pad8(H * sp.vdim), dtype=self.dtype, device=dev)
        ops.linear(self.uv, o, M, sp.vdim, R,
                   nv.Epilogue(kind=ops.GATE, n_main=sp.vdim, out=og.data_ptr(), ldo=og.shape[1], gso=sp.vdim,
                               gate=gate.data_ptr(), ldg=H),
                   groups=H, gsw=sp.vdim * self.uv.shape[2], ldx=H * o.shape[2], gsx=o.shape[2])
        ops.linear(self.o, og, M, self.D, H * sp.vdim, ops.sublayer_output(x, add))


class Attention:
    """Grouped-query attention with rotated halves, a sliding window and a sink per head; queries and keys normed over their
    whole projections. A token's cache row holds [key | value] of every key/value head."""

    def __init__(self, w, spec, D, dtype, dev):
        self.spec, self.D, self.dtype = spec, D, dtype
        if spec.heads % spec.kv_heads or spec.rot_dims % 2 or spec.rot_dims > spec.dim:
            raise ValueError("attention: heads in equal groups, an even number of rotated entries within a head")
        self.qkv = ops.pack(torch.cat([w["q"], w["k"], w["v"]]), dtype, dev)
        biases = [w.get(n + ".b") for n in "qkv"]
        self.bias = None
        if any(b is not None for b in biases):
            self.bias = _vec(torch.cat([torch.zeros(w[n].shape[0]) if b is None else b.float().cpu() for n, b in zip("qkv", biases)]), dev)
        self.q_norm, self.k_norm, self.sink = (_vec(w[n], dev) if n in w else None for n in ("q.norm", "k.norm", "sink"))
        self.o = ops.pack(w["o"], dtype, dev)
        half = spec.rot_dims // 2
        self.freq = _frequencies(spec.rot_base, spec.rot_dims, dev) if half else None

    @property
    def tile_heads(self):
        return self.spec.heads // self.spec.kv_heads

    def new_cache(self, n_seqs, n_blocks, bs):
        sp = self.spec
        return torch.zeros(n_blocks, sp.kv_heads, bs, ops.pad8(sp.dim) + ops.pad8(sp.vdim), dtype=self.dtype, device=self.o.device)

    def run(self, step, h, x, cache, add=True):
        sp, M = self.spec, x.shape[0]
        n = self.qkv.shape[0]
        y = torch.empty(M, ops.pad8(n), dtype=self.dtype, device=x.device)
        ops.linear(self.qkv, h, M, n, self.D, ops.store(y, y.shape[1], n, main_bias=self.bias))
        cs = step.angles(self.freq) if self.freq is not None else None
        q = ops.gqa_prepare(y, sp, self.q_norm, self.k_norm, cs, step.slot, cache)
        o = ops.gqa_attention(q, sp, cache, step.bt, step.seq, step.pos, self.sink,
                              step.tiles.for_heads(self.tile_heads) if step.tiles is not None else None)
        ops.linear(self.o, o, M, self.D, sp.heads * sp.vdim, ops.sublayer_output(x, add))


class GLA:
    """Gated linear attention: state [dim, vdim] per head with a decay per key channel, sigmoid(z)^(1 / tau) through a product
    of low rank; outputs normed per head, gated. State: float [slots, heads, dim, vdim]."""

    def __init__(self, w, spec, D, dtype, dev):
        self.spec, self.D = spec, D
        self.first = ops.pack(torch.cat([w["q"], w["k"], w["v"], w["g"], w["a1"]]), dtype, dev)
        self.rank = w["a1"].shape[0]
        self.a2, self.a2_b, self.norm = _vec(w["a2"].t(), dev), _vec(w["a2.b"], dev), _vec(w["norm"], dev)
        self.o = ops.pack(w["o"], dtype, dev)

    def new_cache(self, n_seqs, n_blocks, bs):
        sp = self.spec
        return torch.zeros(n_seqs, sp.heads, sp.dim, sp.vdim, dtype=torch.float32, device=self.o.device)

    def run(self, step, h, x, cache, add=True):
        sp, M = self.spec, x.shape[0]
        nk, nv_ = sp.heads * sp.dim, sp.heads * sp.vdim
        n = 2 * nk + 2 * nv_
        y = torch.empty(M, ops.pad8(n), dtype=h.dtype, device=x.device)
        a1 = torch.empty(M, self.rank, dtype=torch.float32, device=x.device)
        ops.linear(self.first, h, M, n + self.rank, self.D, ops.store(y, y.shape[1], n, side=a1))
        o = ops.recurrence(ops.DECAY_CHANNEL, y, a1, cache, step, sp.heads, (0, nk, 2 * nk), a2=self.a2, a2_b=self.a2_b,
                           inv_tau=1.0 / sp.tau, q_scale=sp.dim ** -0.5,
                           tiles=step.tiles if step.tiles is not None and step.tiles.chunked(sp.dim, sp.vdim, M) else None)
        o = ops.gated_norm(o, y[:, 2 * nk + nv_:], nv_, sp.heads, self.norm, sp.eps, gate_first=False)
        ops.linear(self.o, o, M, self.D, nv_, ops.sublayer_output(x, add))


class Mamba2:
    """Mamba-2: a causal convolution over x, B, C, a state [N, vdim] per head with a scalar decay, gate before the grouped norm.
    Cache: (state float [slots, heads, N, vdim], the convolution's last inputs T [slots, taps - 1, channels])."""

    def __init__(self, w, spec, D, dtype, dev):
        self.spec, self.D, self.dtype = spec, D, dtype
        self.first = ops.pack(w["in"], dtype, dev)
        self.conv, self.conv_b, self.dt_bias, self.A_log, self.skip, self.norm = (
            _vec(w[n], dev) for n in ("conv", "conv.b", "dt_bias", "A_log", "D", "norm"))
        self.o = ops.pack(w["o"], dtype, dev)
        self.channels, taps = self.conv.shape
        self.conv = self.conv.t().contiguous()
        inner = spec.heads * spec.vdim
        if self.channels != inner + 2 * spec.groups * spec.state or taps != spec.taps or inner % spec.norm_groups:
            raise ValueError("mamba2: sizes of the convolution or the norm groups do not fit")

    def new_cache(self, n_seqs, n_blocks, bs):
        sp, dev = self.spec, self.o.device
        return (torch.zeros(n_seqs, sp.heads, sp.state, sp.vdim, dtype=torch.float32, device=dev),
                torch.zeros(n_seqs, max(1, sp.taps - 1), self.channels, dtype=self.dtype, device=dev))

    def run(self, step, h, x, cache, add=True):
        sp, M = self.spec, x.shape[0]
        inner, gn = sp.heads * sp.vdim, sp.groups * sp.state
        n = inner + self.channels
        y = torch.empty(M, ops.pad8(n), dtype=h.dtype, device=x.device)
        dt = torch.empty(M, sp.heads, dtype=torch.float32, device=x.device)
        ops.linear(self.first, h, M, n + sp.heads, self.D, ops.store(y, y.shape[1], n, side=dt, bias=self.dt_bias))
        conv = ops.conv_of(y[:, inner:], self.conv, self.conv_b, cache[1], step)
        o = ops.recurrence(ops.DECAY_HEAD, ops.causal_conv(conv, M, y), dt, cache[0], step, sp.groups, (inner + gn, inner, 0),
                           A_log=self.A_log, skip=self.skip,
                           tiles=step.tiles if step.tiles is not None and step.tiles.chunked(sp.state, sp.vdim, M) else None)
        o = ops.gated_norm(o, y, inner, sp.norm_groups, self.norm, sp.eps, gate_first=True, conv=conv)
        ops.linear(self.o, o, M, self.D, inner, ops.sublayer_output(x, add))


class GatedFF:
    """W_down(act(W_gate h) * (W_up h)); the two first products are one, their rows in turn."""

    counters = 0

    def __init__(self, w, spec, D, dtype, dev):
        self.spec, self.D = spec, D
        self.first = ops.pack(ops.interleave(w["gate"], w["up"]), dtype, dev)
        self.down = ops.pack(w["down"], dtype, dev)

    def run(self, h, x, counts, add=True):
        M, ff = x.shape[0], self.spec.ff
        a = torch.empty(M, ops.pad8(ff), dtype=h.dtype, device=h.device)
        ops.linear(self.first, h, M, 2 * ff, self.D, ops.glu(a, self.spec.act))
        ops.linear(self.down, a, M, self.D, ff, ops.sublayer_output(x, add))
        return None


class DenseFF:
    def __init__(self, w, spec, D, dtype, dev):
        self.spec, self.D = spec, D
        self.up, self.down = ops.pack(w["up"], dtype, dev), ops.pack(w["down"], dtype, dev)
        self.p = self.q = 0.0
        if spec.act == "xielu":
            a, b = (math.log1p(math.exp(-abs(v))) + max(v, 0.0) for v in w["act"].double().tolist())    # softplus
            self.p, self.q = a, 0.5 + b

    counters = 0

    def run(self, h, x, counts, add=True):
        M, ff = x.shape[0], self.spec.ff
        a = torch.empty(M, ops.pad8(ff), dtype=h.dtype, device=h.device)
        ops.linear(self.up, h, M, ff, self.D, ops.store(a, a.shape[1], ff, self.spec.act, self.p, self.q))
        ops.linear(self.down, a, M, self.D, ff, ops.sublayer_output(x, add))
        return None


class ExpertsFF:
    """The `top` experts of every token (softmax over the chosen logits), and a shared expert whose first product also
    carries the router's rows."""

    def __init__(self, w, spec, D, dtype, dev):
        self.spec, self.D = spec, D
        E = spec.experts
        self.up = ops.pack(torch.stack([w[f"e{i}.up"] for i in range(E)]), dtype, dev)
        self.down = ops.pack(torch.stack([w[f"e{i}.down"] for i in range(E)]), dtype, dev)
        rows = [w["shared.up"], w["router"]] if spec.shared_ff else [w["router"]]
        self.front = ops.pack(torch.cat(rows), dtype, dev)
        self.router_b = _vec(w["router.b"], dev)
        self.shared_down = ops.pack(w["shared.down"], dtype, dev) if spec.shared_ff else None

    @property
    def counters(self):
        return self.spec.experts

    def run(self, h, x, counts, add=True):
        sp, M, D, dev = self.spec, x.shape[0], self.D, x.device
        E, fs = sp.experts, sp.shared_ff
        logits = torch.empty(M, E, dtype=torch.float32, device=dev)
        a = torch.empty(M, ops.pad8(fs), dtype=h.dtype, device=dev) if fs else logits
        ops.linear(self.front, h, M, fs + E, D, ops.store(a, a.shape[1], fs, sp.shared_act, side=logits, bias=self.router_b))
        chosen, weight, rank = ops.route(logits, E, sp.top, counts)
        hp, place = ops.gather(h, D, chosen, rank, counts)
        u = torch.empty(M * sp.top, ops.pad8(sp.ff), dtype=h.dtype, device=dev)
        y = torch.empty(M * sp.top, D, dtype=torch.float32, device=dev)
        ops.linear(self.up, hp, M * sp.top, sp.ff, D, ops.store(u, u.shape[1], sp.ff, sp.act), groups=E,
                   gsw=sp.ff * self.up.shape[2], counts=counts)
        ops.linear(self.down, u, M * sp.top, D, sp.ff, ops.store(y, D, D, out_type=ops.OUT_F32), groups=E,
                   gsw=D * self.down.shape[2], counts=counts)
        if fs:
            ops.linear(self.shared_down, a, M, D, fs, ops.sublayer_output(x, add))
        elif not add:
            x.zero_()
        return y, place, weight
