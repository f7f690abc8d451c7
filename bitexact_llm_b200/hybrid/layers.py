"""The layer mechanisms of the hybrid float models: mixers (minGRU, latent attention) and feed-forwards (dense, experts).

A mixer owns its packed weights and the shape of its per-layer cache; `run(step, h, x, cache)` reads the normed rows h
and adds its output to the residual rows x. A feed-forward's `run(h, x, counts)` does the same and returns what is still
due to x (the experts' outputs, folded into the next norm) or None. Weights arrive as a dict name -> tensor with the
mechanism's own names ('z', 'dq.norm', 'e0.up', ...)."""

import math
from dataclasses import dataclass

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
    tiles: torch.Tensor = None  # int32 [T, 3] attention tiles of a prompt portion


def _vec(t, dev):
    return t.to(dev).float().contiguous()


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

    def run(self, step, h, x, cache):
        s = ops.min_gru(self.w, self.bz, self.bx, h, self.spec.width, self.D, cache, step.flags, step.seq)
        ops.linear(self.o, s, x.shape[0], self.D, self.spec.width, ops.add(x))


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

    def run(self, step, h, x, cache):
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
        o = ops.latent_attention(q, sp, cache, step.bt, step.seq, step.pos, self.sink, step.tiles)
        og = torch.empty(M, ops.pad8(H * sp.vdim), dtype=self.dtype, device=dev)
        ops.linear(self.uv, o, M, sp.vdim, R,
                   nv.Epilogue(kind=ops.GATE, n_main=sp.vdim, out=og.data_ptr(), ldo=og.shape[1], gso=sp.vdim,
                               gate=gate.data_ptr(), ldg=H),
                   groups=H, gsw=sp.vdim * self.uv.shape[2], ldx=H * o.shape[2], gsx=o.shape[2])
        ops.linear(self.o, og, M, self.D, H * sp.vdim, ops.add(x))


class DenseFF:
    def __init__(self, w, spec, D, dtype, dev):
        self.spec, self.D = spec, D
        self.up, self.down = ops.pack(w["up"], dtype, dev), ops.pack(w["down"], dtype, dev)
        self.p = self.q = 0.0
        if spec.act == "xielu":
            a, b = (math.log1p(math.exp(-abs(v))) + max(v, 0.0) for v in w["act"].double().tolist())    # softplus
            self.p, self.q = a, 0.5 + b

    counters = 0

    def run(self, h, x, counts):
        M, ff = x.shape[0], self.spec.ff
        a = torch.empty(M, ops.pad8(ff), dtype=h.dtype, device=h.device)
        ops.linear(self.up, h, M, ff, self.D, ops.store(a, a.shape[1], ff, self.spec.act, self.p, self.q))
        ops.linear(self.down, a, M, self.D, ff, ops.add(x))
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

    def run(self, h, x, counts):
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
            ops.linear(self.shared_down, a, M, D, fs, ops.add(x))
        return y, place, weight
