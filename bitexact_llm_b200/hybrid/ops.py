"""Thin callers of libbitexact_float: packing of weights, allocation of outputs, one function per entry point.

Matrices and activations are kept with their last dimension padded to a multiple of 8 elements (TMA wants row starts on
16-byte boundaries); the padding is storage only, the kernels get the true extents."""

import ctypes

import torch

from .. import _native as nv

DTYPES = {"bfloat16": (torch.bfloat16, 0), "float32": (torch.float32, 1)}
ACTS = {"none": 0, "relu2": 1, "xielu": 2, "gelu": 3, "softcap": 4, "scale": 5}
STORE, ADD, ROPE, GATE, GLU = 0, 1, 2, 3, 4
DECAY_CHANNEL, DECAY_HEAD = 0, 1
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


def store(out, ldo, n, act="none", act_p=0.0, act_q=0.0, out_type=OUT_T, gso=0, side=None, bias=None,
          main_bias=None):
    """Epilogue of a plain product: channels below n to `out`, the others (with bias) to the float tensor `side`."""
    return nv.Epilogue(kind=STORE, out_type=out_type, act=ACTS[act], n_main=n, act_p=act_p, act_q=act_q,
                       out=out.data_ptr(), ldo=ldo, gso=gso, side=nv.ptr(side), lds=0 if side is None else side.stride(0),
                       bias=nv.ptr(bias), main_bias=nv.ptr(main_bias))


def add(x):
    return nv.Epilogue(kind=ADD, out=x.data_ptr(), ldo=x.stride(0))


def sublayer_output(x, add_to):
    """Epilogue of a sublayer's last product: x float [M, D] += it, or x = it."""
    return add(x) if add_to else store(x, x.stride(0), x.shape[1], out_type=OUT_F32)


def glu(out, act):
    """Epilogue of a product whose rows 2 i and 2 i + 1 are a gate and its value: out[m, i] = act(gate) * value."""
    return nv.Epilogue(kind=GLU, act=ACTS[act], out=out.data_ptr(), ldo=out.stride(0))


def interleave(gate, up):
    """[N, K] twice -> [2 N, K], a row of each in turn."""
    return torch.stack([gate, up], 1).reshape(-1, gate.shape[1])


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


def streams(x, eps, start=None, update=None, mix_in=None, w=None, h=None, total=None):
    """Residual streams x float [M, S, D]. start = (ids, embed): every stream is the embedding; update = (y, out, mix): the
    streams after a sublayer with output y. Then h T [M, pad8(D)] = RMS norm (weight w) of the streams weighted by mix_in,
    or total float [M, D] = their sum."""
    M, S, D = x.shape
    ids, embed = start if start is not None else (None, None)
    y, out, mix = update if update is not None else (None, None, None)
    p = nv.StreamsStep(x=x.data_ptr(), ids=nv.ptr(ids), embed=nv.ptr(embed), vocab=0 if embed is None else embed.shape[0],
                       y=nv.ptr(y), out=nv.ptr(out), mix=nv.ptr(mix), in_=nv.ptr(mix_in), w=nv.ptr(w), h=nv.ptr(h),
                       ldh=0 if h is None else h.stride(0), sum=nv.ptr(total), eps=eps, streams=S, D=D)
    t = h if h is not None else embed
    nv.check(nv.float_lib().bxf_streams(0 if t is None else code(t), ctypes.byref(p), M, nv.stream()), "bxf_streams")


def angles(freq, pos):
    """freq double [half] -> (cos, sin) of pos * freq, float [M, half, 2]."""
    cs = torch.empty(pos.shape[0], freq.shape[0], 2, dtype=torch.float32, device=pos.device)
    rc = nv.float_lib().bxf_angles(freq.data_ptr(), freq.shape[0], pos.data_ptr(), cs.data_ptr(), pos.shape[0], nv.stream())
    nv.check(rc, "bxf_angles")
    return cs


def gqa_prepare(y, spec, q_norm, k_norm, cs, slot, cache):
    """y T [M, >= q | k | v] -> queries T [kv_heads, M, heads per group, pad8(dim)]; the tokens' cache rows are written."""
    M, G = y.shape[0], spec.kv_heads
    q = torch.empty(G, M, spec.heads // G, pad8(spec.dim), dtype=y.dtype, device=y.device)
    p = nv.GqaRows(y=y.data_ptr(), ldy=y.stride(0), heads=spec.heads, kv_heads=G, dim=spec.dim, vdim=spec.vdim,
                   rot_dims=spec.rot_dims, page=cache.shape[2], q_norm=nv.ptr(q_norm), k_norm=nv.ptr(k_norm), cs=nv.ptr(cs),
                   slot=slot.data_ptr(), q=q.data_ptr(), ldq=q.shape[3], cache=cache.data_ptr(), ldc=cache.shape[3],
                   voff=pad8(spec.dim), eps=spec.eps)
    nv.check(nv.float_lib().bxf_gqa_prepare(code(y), ctypes.byref(p), M, nv.stream()), "bxf_gqa_prepare")
    return q


def gqa_attention(q, spec, cache, bt, seq, pos, sink, tiles=None, variant=0):
    """q T [kv_heads, M, heads per group, ldq] against the paged cache T [blocks, kv_heads, bs, ldc] -> T [M, pad8(heads vdim)]."""
    G, M, per, ldq = q.shape
    lib, H = nv.float_lib(), spec.heads
    out = torch.empty(M, pad8(H * spec.vdim), dtype=q.dtype, device=q.device)
    need = lib.bxf_gqa_attention_scratch(M, H, G, spec.vdim)
    scratch = torch.empty(need, dtype=torch.uint8, device=q.device) if need else None
    assert bt.dtype in (torch.int32, torch.int64) and bt.stride(1) == 1 and q.is_contiguous() and cache.is_contiguous()
    rc = lib.bxf_gqa_attention(code(q), q.data_ptr(), ldq, M, H, G, spec.dim, spec.vdim, cache.data_ptr(), cache.shape[3],
                               pad8(spec.dim), cache.shape[2], cache.shape[0], bt.data_ptr(), int(bt.dtype == torch.int64),
                               bt.stride(0), bt.shape[1], seq.data_ptr(), pos.data_ptr(), nv.ptr(tiles),
                               0 if tiles is None else tiles.shape[0], spec.window, nv.ptr(sink), spec.scale, out.data_ptr(),
                               out.shape[1], nv.ptr(scratch), need, variant, nv.stream())
    nv.check(rc, "bxf_gqa_attention")
    return out


def conv_of(u, w, b, state, step):
    """bxf_conv of inputs u T [M, channels] (a view into wider rows), w float [taps, channels]."""
    return nv.Conv(u=u.data_ptr(), ldu=u.stride(0), w=w.data_ptr(), b=b.data_ptr(), state=state.data_ptr(),
                   flags=step.flags.data_ptr(), seq=step.seq.data_ptr(), pos=step.pos.data_ptr(), channels=w.shape[1],
                   taps=w.shape[0])


def causal_conv(conv, M, like):
    """-> silu(convolution) T [M, pad8(channels)]."""
    out = torch.empty(M, pad8(conv.channels), dtype=like.dtype, device=like.device)
    rc = nv.float_lib().bxf_causal_conv(code(like), ctypes.byref(conv), out.data_ptr(), out.stride(0), M, nv.stream())
    nv.check(rc, "bxf_causal_conv")
    return out


def recurrence(kind, y, side, state, step, groups, columns, a2=None, a2_b=None, inv_tau=0.0, q_scale=1.0,
               A_log=None, skip=None, tiles=None):
    """state float [slots, heads, K, V] is advanced by the rows of y; columns = where q, k, v begin in y -> outputs T
    [M, pad8(heads V)]. tiles: the chunk kernels walk its runs, else the rows go one by one."""
    M, (_, H, K, V) = y.shape[0], state.shape
    out = torch.empty(M, pad8(H * V), dtype=y.dtype, device=y.device)
    p = nv.RecurrenceRows(kind=kind, heads=H, groups=groups, K=K, V=V, rank=0 if a2 is None else a2.shape[0], q0=columns[0],
                          k0=columns[1], v0=columns[2], batch=int(step.tiles is None), y=y.data_ptr(), ldy=y.stride(0), side=side.data_ptr(),
                          lds=side.stride(0), a2=nv.ptr(a2), a2_b=nv.ptr(a2_b), inv_tau=inv_tau, q_scale=q_scale,
                          A_log=nv.ptr(A_log), skip=nv.ptr(skip), state=state.data_ptr(), flags=step.flags.data_ptr(),
                          seq=step.seq.data_ptr(), out=out.data_ptr(), ldo=out.stride(0))
    lib = nv.float_lib()
    if tiles is None:
        if kind == DECAY_CHANNEL:
            decays = torch.empty(M, H * K, dtype=torch.float32, device=y.device)
            p.decays = decays.data_ptr()
        nv.check(lib.bxf_recurrence(code(y), ctypes.byref(p), M, nv.stream()), "bxf_recurrence")
        return out
    segments = tiles.segments if tiles.segments.shape[0] > tiles.runs.shape[0] else None
    t = nv.ChunkTable(runs=tiles.runs.data_ptr(), chunks=tiles.chunks.data_ptr(), segments=nv.ptr(segments),
                      spans=tiles.spans.data_ptr(), nruns=tiles.runs.shape[0], nchunks=tiles.chunks.shape[0],
                      nsegments=0 if segments is None else segments.shape[0])
    need = lib.bxf_recurrence_chunk_scratch(kind, M, t.nchunks, t.nsegments, H, K, V)
    scratch = torch.empty(need, dtype=torch.uint8, device=y.device) if need else None
    rc = lib.bxf_recurrence_chunks(code(y), ctypes.byref(p), ctypes.byref(t), nv.ptr(scratch), need, M, nv.stream())
    nv.check(rc, "bxf_recurrence_chunks")
    return out


def gated_norm(o, z, n, parts, w, eps, gate_first, conv=None):
    """o, z T [M, >= n] -> T [M, pad8(n)]: RMS norm of `parts` equal parts and the gate silu(z), before or after the norm."""
    out = torch.empty(o.shape[0], pad8(n), dtype=o.dtype, device=o.device)
    p = nv.GateRows(o=o.data_ptr(), z=z.data_ptr(), ldo=o.stride(0), ldz=z.stride(0), w=w.data_ptr(), out=out.data_ptr(),
                    ldout=out.stride(0), n=n, parts=parts, wn=w.shape[0], gate_first=int(gate_first), eps=eps)
    if conv is not None:
        p.conv = conv
    nv.check(nv.float_lib().bxf_gated_norm(code(o), ctypes.byref(p), o.shape[0], nv.stream()), "bxf_gated_norm")
    return out
