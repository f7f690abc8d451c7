"""Thin callers of libbitexact_float: packing of weights, allocation of outputs, one function per entry point.

Matrices and activations are kept with their last dimension padded to a multiple of 8 elements (TMA wants row starts on
16-byte boundaries); the padding is storage only, the kernels get the true extents."""

import ctypes

import torch

from .. import _native as nv

DTYPES = {"bfloat16": (torch.bfloat16, 0), "float32": (torch.float32, 1)}
ACTS = {"none": 0, "relu2": 1, "xielu": 2}
STORE, ADD, ROPE, GATE = 0, 1, 2, 3
OUT_T, OUT_F32, OUT_I64 = 0, 1, 2


def pad8(n):
    return (n + 7) // 8 * 8


def pack(w, dtype, dev):
    """[..., N, K] -> contiguous storage [..., N, pad8(K)] of `dtype` on the device, zeros in the padding."""
    out = torch.zeros(*w.shape[:-1], pad8(w.shape[-1]), dtype=dtype, device=dev)
    out[..., : w.shape[-1]] = w.to(dev).to(dtype)
    return out


def code(t):
    return 1 if t.dtype == torch.float32 else 0


def linear(w, x, M, N, K, epi, groups=1, gsw=0, ldx=None, gsx=0, counts=None, tile=0):
    """w [(groups,) N, ldw] and x [M, ldx] tensors of one element type; epi: nv.Epilogue."""
    rc = nv.float_lib().bxf_linear(code(w), w.data_ptr(), w.shape[-1], gsw, x.data_ptr(), x.stride(0) if ldx is None else ldx,
                                   gsx, groups, M, N, K, nv.ptr(counts), ctypes.byref(epi), tile, nv.stream())
    nv.check(rc, "bxf_linear")


def store(out, ldo, n, act="none", act_p=0.0, act_q=0.0, out_type=OUT_T, gso=0, side=None, bias=None):
    """Epilogue of a plain product: channels below n to `out`, the others (with bias) to the float tensor `side`."""
    return nv.Epilogue(kind=STORE, out_type=out_type, act=ACTS[act], n_main=n, act_p=act_p, act_q=act_q,
                       out=out.data_ptr(), ldo=ldo, gso=gso, side=nv.ptr(side), lds=0 if side is None else side.stride(0),
                       bias=nv.ptr(bias))


def add(x):
    return nv.Epilogue(kind=ADD, out=x.data_ptr(), ldo=x.stride(0))


def norm(x, w, b, eps, h=None, ids=None, embed=None, experts=None, zero=None):
    """Layer norm of the residual rows x float [M, D] into h [M, pad8(D)], after x = embed[ids], or after adding the
    experts' outputs (y, place, weight) still due to x. h None: only the latter."""
    M, D = x.shape
    y, place, weight = experts if experts is not None else (None, None, None)
    t = h if h is not None else embed
    rc = nv.float_lib().bxf_norm(0 if t is None else code(t), x.data_ptr(), nv.ptr(ids), nv.ptr(embed),
                                 0 if embed is None else embed.shape[0], nv.ptr(y), nv.ptr(place), nv.ptr(weight),
                                 0 if weight is None else weight.shape[1], nv.ptr(w), nv.ptr(b), eps, nv.ptr(h),
                                 0 if h is None else h.stride(0), nv.ptr(zero), 0 if zero is None else zero.numel(), M, D,
                                 nv.stream())
    nv.check(rc, "bxf_norm")


def row_flags(seq, slot, pos):
    flags = torch.empty(seq.shape[0], dtype=torch.int32, device=seq.device)
    rc = nv.float_lib().bxf_row_flags(seq.data_ptr(), slot.data_ptr(), pos.data_ptr(), flags.data_ptr(), seq.shape[0],
                                      nv.stream())
    nv.check(rc, "bxf_row_flags")
    return flags


def min_gru(w, bias_z, bias_x, h, width, K, state, flags, seq):
    """-> state * silu(gate) [M, pad8(width)]; `state` float [slots, width] is advanced by the rows of every sequence.
    w [3, width, pad8(K)]. One kernel when the rows fit a tile (decoding, short portions), else product and scan."""
    M, lib, dt = h.shape[0], nv.float_lib(), code(w)
    out = torch.empty(M, pad8(width), dtype=w.dtype, device=h.device)
    g = nv.Gru(bias_z=bias_z.data_ptr(), bias_x=bias_x.data_ptr(), state=state.data_ptr(), flags=flags.data_ptr(),
               seq=seq.data_ptr(), out=out.data_ptr(), ldo=out.stride(0))
    if M <= lib.bxf_gru_rows(dt):
        rc = lib.bxf_gru_linear(dt, w.data_ptr(), w.shape[-1], h.data_ptr(), h.stride(0), M, width, K, ctypes.byref(g),
                                nv.stream())
        nv.check(rc, "bxf_gru_linear")
        return out
    y = torch.empty(M, 3 * width, dtype=torch.float32, device=h.device)
    linear(w, h, M, 3 * width, K, store(y, 3 * width, 3 * width, out_type=OUT_F32))
    fold = torch.empty(lib.bxf_gru_chunks(M), width, 2, dtype=torch.float32, device=h.device)
    rc = lib.bxf_gru_scan(dt, y.data_ptr(), fold.data_ptr(), M, width, ctypes.byref(g), nv.stream())
    nv.check(rc, "bxf_gru_scan")
    return out


def route(logits, experts, top, counts):
    """logits float [M, >= experts] -> chosen, weight, rank [M, top]; counts int32 [experts] (zeroed before) is filled."""
    M, dev = logits.shape[0], logits.device
    chosen, rank = (torch.empty(M, top, dtype=torch.int32, device=dev) for _ in range(2))
    weight = torch.empty(M, top, dtype=torch.float32, device=dev)
    rc = nv.float_lib().bxf_route(logits.data_ptr(), logits.stride(0), experts, top, chosen.data_ptr(), weight.data_ptr(),
                                  rank.data_ptr(), counts.data_ptr(), M, nv.stream())
    nv.check(rc, "bxf_route")
    return chosen, weight, rank


def gather(h, D, chosen, rank, counts):
    """-> rows of h in expert order [M * top, ldh], place int32 [M, top]."""
    M, top = chosen.shape
    hp = torch.empty(M * top, h.shape[1], dtype=h.dtype, device=h.device)
    place = torch.empty_like(chosen)
    rc = nv.float_lib().bxf_gather(code(h), h.data_ptr(), h.stride(0), D, chosen.data_ptr(), rank.data_ptr(),
                                   counts.data_ptr(), counts.numel(), top, hp.data_ptr(), place.data_ptr(), M, nv.stream())
    nv.check(rc, "bxf_gather")
    return hp, place


def latent_prepare(y, spec, wq, wkv, freq, pos, slot, cache):
    """-> query latent T [M, pad8(q_rank)], (cos, sin) float [M, rot_dim / 2, 2], gate float [M, heads]; the tokens' cache
    rows are written."""
    M, dev = y.shape[0], y.device
    cq = torch.empty(M, pad8(spec.q_rank), dtype=cache.dtype, device=dev)
    cs = torch.empty(M, spec.rot_dim // 2, 2, dtype=torch.float32, device=dev)
    gate = torch.empty(M, spec.heads, dtype=torch.float32, device=dev)
    rc = nv.float_lib().bxf_latent_prepare(code(cache), y.data_ptr(), y.stride(0), spec.q_rank, spec.kv_rank, spec.rot_dim,
                                           spec.heads, wq.data_ptr(), wkv.data_ptr(), spec.eps, freq.data_ptr(),
                                           pos.data_ptr(), slot.data_ptr(), cq.data_ptr(), cq.stride(0), cache.data_ptr(),
                                           cache.stride(1), cs.data_ptr(), gate.data_ptr(), M, nv.stream())
    nv.check(rc, "bxf_latent_prepare")
    return cq, cs, gate


def latent_attention(q, spec, cache, bt, seq, pos, sink, tiles=None, variant=0):
    """q T [M, heads, >= kv_rank + rot_dim] against the paged cache T [blocks, bs, ldc] -> latent outputs T
    [M, heads, pad8(kv_rank)]."""
    M, H, ldq = q.shape
    lib = nv.float_lib()
    out = torch.empty(M, H, pad8(spec.kv_rank), dtype=q.dtype, device=q.device)
    need = lib.bxf_latent_attention_scratch(M, H, spec.kv_rank)
    scratch = torch.empty(need, dtype=torch.uint8, device=q.device) if need else None
    assert bt.dtype in (torch.int32, torch.int64) and bt.stride(1) == 1 and q.is_contiguous() and cache.is_contiguous()
    rc = lib.bxf_latent_attention(code(q), q.data_ptr(), ldq, M, H, spec.kv_rank, spec.rot_dim, cache.data_ptr(),
                                  cache.shape[2], cache.shape[1], cache.shape[0], bt.data_ptr(), int(bt.dtype == torch.int64),
                                  bt.stride(0), bt.shape[1], seq.data_ptr(), pos.data_ptr(), nv.ptr(tiles),
                                  0 if tiles is None else tiles.shape[0], spec.window, nv.ptr(sink), spec.scale,
                                  out.data_ptr(), out.shape[2], nv.ptr(scratch), need, variant, nv.stream())
    nv.check(rc, "bxf_latent_attention")
    return out
