"""The Veredra design on the GPU against the plain float64 oracle (oracle/veredra.py): every mechanism alone, whole prompts,
portions, decoding through caches and states, unequal batches, reused pages and slots, greedy generation, the command lines.
Everything runs in both number formats."""

import json
import os
import subprocess
import sys

import numpy as np
import pytest
import torch

import hybrid_models as hm
import veredra_models as vm
from oracle import hybrid as oh
from oracle import veredra as ov
from test_hybrid_gpu import DTYPES, ROOT, TOL, close, logits, packed, rounded, session, steps

pytestmark = pytest.mark.gpu
_cache = {}


def model(name, dtype):
    """(config, oracle weights, engine), built once."""
    if (name, dtype) not in _cache:
        from bitexact_llm_b200.hybrid import veredra
        cfg = vm.CONFIGS[name]
        t = vm.weights(cfg)
        _cache[name, dtype] = (cfg, hm.as_numpy(t), veredra.load(cfg, t, "cuda", dtype))
    return _cache[name, dtype]


def want_logits(name, toks):
    key = (name, tuple(toks))
    if key not in _cache:
        cfg = vm.CONFIGS[name]
        _cache[key] = ov.forward(cfg, hm.as_numpy(vm.weights(cfg)), toks)[0]
    return _cache[key]


def mostly(got, want, dtype):
    """`close`, but in bf16 a position in thirty may be further away: a norm of an output that almost cancels magnifies what
    rounding the operands did to it."""
    if dtype == "float32":
        return close(got, want, dtype)
    got, want = np.asarray(got, np.float64), np.asarray(want, np.float64)
    assert got.shape == want.shape and np.isfinite(got).all()
    ref = np.sqrt((want ** 2).mean(-1)) + 0.1 * np.sqrt((want ** 2).mean())
    err = np.sqrt(((got - want) ** 2).mean(-1)) / ref
    assert (err > TOL[dtype]).sum() <= max(1, len(err) // 30) and err.max() < 0.4, (err.max(), int(err.argmax()), np.sort(err)[-5:])


def tiles_of(runs, heads=()):
    """Tiles of runs = [(sequence, first position, rows)] as the engine makes them."""
    from bitexact_llm_b200 import _native as nv
    from bitexact_llm_b200.hybrid.layers import Tiles
    row, table = 0, []
    for s, p, n in runs:
        table.append((s, row, n, p + n))
        row += n
    return Tiles.of(table, {nv.float_lib().bxf_latent_attention_tile(h) for h in heads}).to("cuda")


# ---------------------------------------------------------------- epilogues

@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("M,ff,K,tile", [(1, 5, 24, 0), (16, 130, 72, 0), (37, 50, 40, 16), (70, 64, 64, 32), (45, 33, 90, 64),
                                         (200, 70, 200, 128), (300, 257, 130, 256)])
def test_gated_product(M, ff, K, tile, dtype):
    from bitexact_llm_b200.hybrid import ops
    rng = np.random.RandomState(M)
    gate, up, x = (rounded(rng.randn(*s), dtype) for s in ((ff, K), (ff, K), (M, K)))
    W = ops.pack(ops.interleave(torch.tensor(gate), torch.tensor(up)), ops.DTYPES[dtype][0], "cuda")
    out = torch.full((M, ops.pad8(ff) + 8), 7.0, dtype=W.dtype, device="cuda")
    ops.linear(W, packed(x, dtype), M, 2 * ff, K, ops.glu(out, "gelu"), tile=tile)
    close(out[:, :ff].float().cpu(), ov.gelu_tanh(x @ gate.T) * (x @ up.T), dtype, 0.3)
    assert (out[:, ff:] == 7.0).all()


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("M,tile", [(3, 0), (40, 16), (70, 64), (150, 128), (300, 256)])
def test_bias_softcap_and_scale(M, tile, dtype):
    from bitexact_llm_b200.hybrid import ops
    rng = np.random.RandomState(M)
    N, E, K = 61, 9, 40
    w, x = rounded(rng.randn(N + E, K), dtype), rounded(rng.randn(M, K), dtype)
    W, X, acc = packed(w, dtype), packed(x, dtype), x @ w.T
    b, side_b = (torch.tensor(rng.randn(n), dtype=torch.float32).cuda() for n in (N, E))
    b64 = b.double().cpu().numpy()
    for act, p, q, f in (("none", 0, 0, lambda v: v), ("gelu", 0, 0, ov.gelu_tanh), ("scale", 0.3, 0, lambda v: 0.3 * v),
                         ("softcap", 0.25, 8.0, lambda v: 8.0 * np.tanh(0.25 * v))):
        out = torch.zeros(M, 64, dtype=W.dtype, device="cuda")
        side = torch.zeros(M, E, device="cuda")
        ops.linear(W, X, M, N + E, K, ops.store(out, 64, N, act, p, q, side=side, bias=side_b, main_bias=b), tile=tile)
        close(out[:, :N].float().cpu(), f(acc[:, :N] + b64), dtype, 0.3)
        close(side.cpu(), acc[:, N:] + side_b.double().cpu().numpy(), "float32")
    fix = torch.zeros(M, N, dtype=torch.long, device="cuda")
    ops.linear(W[:N], X, M, N, K, ops.store(fix, N, N, "softcap", 0.25, 8.0, out_type=ops.OUT_I64), tile=tile)
    close(fix.double().cpu().numpy() / 2 ** 24, 8.0 * np.tanh(0.25 * acc[:, :N]), "float32")


# ---------------------------------------------------------------- residual streams

@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("S,D", [(1, 52), (2, 256), (3, 1030), (4, 64), (5, 77), (8, 2048)])
def test_streams(S, D, dtype):
    from bitexact_llm_b200.hybrid import ops
    T = ops.DTYPES[dtype][0]
    rng = np.random.RandomState(S + D)
    M, V, eps = 7, 20, 1e-2
    emb = torch.tensor(rng.randn(V, D)).to(T).cuda()
    ids = torch.tensor(rng.randint(0, V, M)).cuda()
    coef = [{k: torch.tensor(rng.randn(*s), dtype=torch.float32).cuda() for k, s in (("in", (S,)), ("out", (S,)), ("mix", (S, S)))}
            for _ in range(2)]
    c64 = [{k: v.double().cpu().numpy() for k, v in c.items()} for c in coef]
    w = torch.tensor(1 + 0.3 * rng.randn(D), dtype=torch.float32).cuda()
    y = torch.tensor(rng.randn(M, D), dtype=torch.float32).cuda()
    x = torch.full((M, S, D), float("nan"), device="cuda")
    h = torch.zeros(M, ops.pad8(D), dtype=T, device="cuda")
    norm = lambda v: oh.rms_norm(v, w.double().cpu().numpy(), eps)
    ops.streams(x, eps, (ids, emb), None, coef[0]["in"], w, h)
    xs = np.stack([emb[ids].double().cpu().numpy()] * S)
    assert np.array_equal(x.double().cpu().numpy(), xs.transpose(1, 0, 2))
    close(h[:, :D].float().cpu(), norm(ov.hyper_in(xs, c64[0])), dtype, 0.3)
    ops.streams(x, eps, None, (y, coef[0]["out"], coef[0]["mix"]), coef[1]["in"], w, h)
    xs = ov.hyper_out(xs, c64[0], y.double().cpu().numpy())
    close(x.cpu().numpy().transpose(1, 0, 2), xs, "float32")
    close(h[:, :D].float().cpu(), norm(ov.hyper_in(xs, c64[1])), dtype, 0.3)
    total, keep = torch.empty(M, D, device="cuda"), x.clone()
    ops.streams(x, eps, None, (y, coef[1]["out"], coef[1]["mix"]), total=total)
    close(total.cpu(), ov.hyper_out(xs, c64[1], y.double().cpu().numpy()).sum(0), "float32")
    assert torch.equal(x, keep)


@pytest.mark.parametrize("dtype", DTYPES)
def test_experts_between_streams(dtype):
    """A feed-forward that leaves its experts' outputs due: they must be in y before the streams mix it."""
    from bitexact_llm_b200.hybrid import ops
    from bitexact_llm_b200.hybrid.engine import HybridEngine
    from bitexact_llm_b200.hybrid.spec import ExpertsSpec, GLASpec, LayerSpec, ModelSpec
    cfg = vm.config(50, 48, 2, [vm.gla(2, 8, 16, 4.0, 24, 4)])
    t = vm.weights(cfg)
    g = torch.Generator().manual_seed(3)
    for shared in (0, 16):
        f = {"kind": "moe", "router": {"experts": 3, "top": 3}, "expert": {"ff": 24}, "shared": {"ff": shared} if shared else None}
        ff = {f"e{e}.{n}": torch.randn(*s, generator=g) * 0.2 for e in range(3) for n, s in (("up", (24, 48)), ("down", (48, 24)))}
        ff.update({"router": torch.randn(3, 48, generator=g), "router.b": torch.zeros(3)})
        if shared:
            ff.update({"shared.up": torch.randn(shared, 48, generator=g) * 0.2, "shared.down": torch.randn(48, shared, generator=g) * 0.2})
        ff = {k: v.to(torch.bfloat16) for k, v in ff.items()}
        spec = ModelSpec(50, 48, 1e-5, (LayerSpec(GLASpec(2, 8, 16, 4.0, 1e-5), ExpertsSpec(3, 3, 24, shared)),), streams=2)
        sub = lambda p: oh.sub(t, "l0." + p)
        eng = HybridEngine(spec, {"embed": t["embed"], "head": t["head"], "final": t["final.norm"],
                                  "layers": [{"norm1": t["l0.norm1"], "norm2": t["l0.norm2"], "mixer": sub("mix."), "ff": ff,
                                              "hc1": sub("hc1."), "hc2": sub("hc2.")}]}, "cuda", dtype)
        toks = hm.tokens(cfg, 30, 1)
        w = hm.as_numpy(t)
        xs = np.stack([w["embed"][toks]] * 2)
        for q, body in ((1, lambda h: ov.gla(h, oh.sub(w, "l0.mix."), cfg["layers"][0]["mixer"], 1e-5)[0]),
                        (2, lambda h: oh.moe_ff(h, hm.as_numpy(ff), 3, 3, f["shared"]))):
            hc = oh.sub(w, f"l0.hc{q}.")
            xs = ov.hyper_out(xs, hc, body(oh.rms_norm(ov.hyper_in(xs, hc), 1 + w[f"l0.norm{q}"], 1e-5)))
        close(session(eng).feed([(0, toks)])[0].cpu(), xs.sum(0), dtype)


# ---------------------------------------------------------------- attention

SHAPES = [  # heads, kv heads, dim, vdim, rotated, window, page size
    (6, 2, 24, 40, 16, 19, 4), (5, 5, 10, 13, 6, 33, 8), (16, 2, 64, 80, 32, 130, 16), (12, 4, 128, 64, 128, 65, 64),
    (1, 1, 8, 8, 0, 1, 16), (8, 1, 72, 264, 64, 0, 32), (130, 1, 16, 24, 8, 64, 16), (4, 4, 192, 128, 96, 100, 128)]


def attention_case(H, G, dk, dv, rot, window, dtype, rng, D=40):
    from bitexact_llm_b200.hybrid import ops
    from bitexact_llm_b200.hybrid.layers import Attention
    from bitexact_llm_b200.hybrid.spec import AttentionSpec
    cfg = vm.config(10, D, 1, [vm.attn(H, G, dk, dv, rot, window, None, base=300.0)])
    w = {k[len("l0.mix."):]: v for k, v in vm.weights(cfg, H + dk).items() if k.startswith("l0.mix.")}
    m = cfg["layers"][0]["mixer"]
    sp = AttentionSpec(H, G, dk, dv, rot, 300.0, m["scale"], window, 1e-5)
    return Attention(w, sp, D, ops.DTYPES[dtype][0], "cuda"), hm.as_numpy(w), m


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("H,G,dk,dv,rot,window,bs", SHAPES)
def test_attention_layer(H, G, dk, dv, rot, window, bs, dtype):
    """Whole sequences, portions and single tokens of two sequences over scattered pages."""
    rng = np.random.RandomState(H + dk)
    layer, w, m = attention_case(H, G, dk, dv, rot, window, dtype, rng)
    n, D = 150, 40
    hs = [rounded(rng.randn(n, D), dtype) for _ in range(2)]
    want = [ov.attention(h, w, m, 1e-5) for h in hs]
    blocks = 1 + 2 * ((n + bs - 1) // bs)
    for cuts in ([n], [70, 2, 3, 1, 1, 70, 3]):
        cache, at, got = layer.new_cache(2, blocks, bs), 0, [[], []]
        cache.fill_(0.5)                                              # what earlier requests left
        for k in cuts:
            runs = [(1, at, k), (0, at, k)]
            for tiles in [None] + ([tiles_of(runs, [layer.tile_heads])] if dtype == "bfloat16" and k > 1 else []):
                st = steps(dtype, runs, bs, blocks, 2, tiles)
                x = torch.zeros(2 * k, D, device="cuda")
                layer.run(st, packed(np.concatenate([hs[1][at:at + k], hs[0][at:at + k]]), dtype), x, cache)
                y = torch.full((2 * k, D), 5.0, device="cuda")
                layer.run(st, packed(np.concatenate([hs[1][at:at + k], hs[0][at:at + k]]), dtype), y, cache, add=False)
                close(y.cpu(), x.cpu(), "float32")
            got[1].append(x[:k].cpu())
            got[0].append(x[k:].cpu())
            at += k
        for i in range(2):
            close(torch.cat(got[i]), want[i], dtype)


@pytest.mark.parametrize("dtype", DTYPES)
def test_attention_variants_agree(dtype):
    from bitexact_llm_b200.hybrid import ops
    from bitexact_llm_b200.hybrid.spec import AttentionSpec
    H, G, dk, dv, window, bs = 12, 3, 48, 72, 90, 16
    sp = AttentionSpec(H, G, dk, dv, 0, 1.0, 0.2, window, 1e-5)
    rng = np.random.RandomState(5)
    runs = [(1, 0, 70), (0, 190, 9), (2, 63, 2), (1, 128, 1)]
    st = steps(dtype, runs, bs, 1 + 3 * 16, 3)
    M, P = st.pos.shape[0], H // G
    q, kc, vc = (rounded(rng.randn(*s), dtype) for s in ((G, M, P, dk), (49, G, bs, dk), (49, G, bs, dv)))
    C = packed(np.concatenate([kc, vc], -1), dtype)
    sink = rng.randn(H)
    want = np.zeros((M, H, dv))
    for m in range(M):
        s, i = int(st.seq[m]), int(st.pos[m])
        js = np.arange(max(0, i - window + 1), i + 1)
        pages = st.bt[s].cpu().numpy()[js // bs]
        for h in range(H):
            e = np.exp(kc[pages, h // P, js % bs] @ q[h // P, m, h % P] * 0.2)
            want[m, h] = e @ vc[pages, h // P, js % bs] / (e.sum() + np.exp(sink[h]))
    sinks = torch.tensor(sink, dtype=torch.float32).cuda()
    tiles = tiles_of(runs, [P]).for_heads(P)
    for variant, tt in [(0, None), (0, tiles), (1, None)] + ([(2, None), (2, tiles)] if dtype == "bfloat16" else []):
        out = ops.gqa_attention(packed(q, dtype), sp, C, st.bt, st.seq, st.pos, sinks, tt, variant)
        close(out[:, :H * dv].float().cpu().numpy().reshape(M, H, dv), want, dtype, 0.5)
    one = ops.gqa_attention(packed(q[:, 78:79], dtype), sp, C, st.bt, st.seq[78:79].contiguous(), st.pos[78:79].contiguous(), sinks)
    close(one[:, :H * dv].float().cpu().numpy().reshape(1, H, dv), want[78:79], dtype, 0.5)


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("window", [1, 2, 16, 63, 64, 65, 100])
def test_one_key_stands_out_at_every_distance(window, dtype):
    """One cached key takes nearly all the weight of every query of its group that sees it: a window that is off by one, a page
    or group mix-up or a lost block shows. Also with a sink that outweighs it."""
    from bitexact_llm_b200.hybrid import ops
    from bitexact_llm_b200.hybrid.spec import AttentionSpec
    H, G, d, bs, n = 6, 2, 16, 16, 200
    sp = AttentionSpec(H, G, d, d, 0, 1.0, 1.0, window, 1e-5)
    st = steps(dtype, [(0, 0, n)], bs, 1 + 13, 1)
    q = np.zeros((G, n, H // G, d))
    q[..., 0] = 1.0
    tiles = tiles_of([(0, 0, n)], [H // G]).for_heads(H // G)
    pages = st.bt[0].cpu().numpy()
    for far in (0, 15, 16, 47, 63, 64, 127, 130):
        cache = np.zeros((14, G, bs, 2 * d))
        for j in range(n):
            cache[pages[j // bs], :, j % bs, d] = 1.0
        cache[pages[far // bs], 1, far % bs, 0] = 20.0                # group 1 only
        cache[pages[far // bs], 1, far % bs, d:d + 2] = (0.0, 1.0)    # the marker's value
        for sink, full in ((-30.0, 1.0), (40.0, 0.0)):
            s = torch.full((H,), sink, device="cuda")
            for tt in (None, tiles):
                out = ops.gqa_attention(packed(q, dtype), sp, packed(cache, dtype), st.bt, st.seq, st.pos, s, tt)
                got = out.float().cpu().numpy().reshape(n, G, H // G, d)
                i = np.arange(n)
                seen = ((i >= far) & (i - far < window))[:, None]
                assert np.allclose(got[:, 1, :, 1], seen * full, atol=1e-2), (far, sink)
                assert np.allclose(got[:, 0, :, 1], 0.0)
                if full:
                    assert np.allclose(got[:, 1, :, 0], 1.0 - seen, atol=1e-2) and np.allclose(got[:, 0, :, 0], 1.0, atol=1e-2)


@pytest.mark.parametrize("dtype", DTYPES)
def test_rotation_far_from_the_start(dtype):
    """Queries and keys of far positions, first `rot` entries only, halves paired; angles beyond what 32-bit products hold."""
    from bitexact_llm_b200.hybrid import ops
    from bitexact_llm_b200.hybrid.spec import AttentionSpec
    H, G, d, rot, n = 4, 2, 20, 12, 3
    sp = AttentionSpec(H, G, d, 8, rot, 7.0, 1.0, 0, 1e-5)
    freq = torch.tensor([7.0 ** (-2 * i / rot) for i in range(rot // 2)], dtype=torch.float64, device="cuda")
    rng = np.random.RandomState(1)
    y = rounded(rng.randn(n, (H + G) * d + G * 8), dtype)
    for first in (0, 1, 100003, 3 * 10 ** 7):
        pos = torch.arange(first, first + n, device="cuda")
        slot = torch.tensor([5, 0, -1], device="cuda")                # the last one is padding
        cache = torch.zeros(3, G, 4, 24 + 8, dtype=ops.DTYPES[dtype][0], device="cuda")
        q = ops.gqa_prepare(packed(y, dtype), sp, None, None, ops.angles(freq, pos), slot, cache)
        rot64 = lambda v: ov.rotate_halves(v, 7.0, rot, first)
        q64, k64 = rot64(y[:, :H * d].reshape(n, H, d)), rot64(y[:, H * d:(H + G) * d].reshape(n, G, d))
        close(q.float().cpu().numpy()[..., :d].transpose(1, 0, 2, 3).reshape(n, H, d), q64, dtype, 0.2 if dtype == "bfloat16" else 1.0)
        row = cache[1, :, 1].float().cpu().numpy()
        close(row[:, :d], k64[0], dtype, 0.2 if dtype == "bfloat16" else 1.0)
        assert np.array_equal(row[:, 24:], y[0, (H + G) * d:].reshape(G, 8)) and (cache[2] == 0).all()


# ---------------------------------------------------------------- recurrences

def recurrence_inputs(kind, H, G, K, V, rank, rng, T, dtype, hard=False):
    """(rows y, side, keyword arguments of ops.recurrence, oracle q, k, v, decay, skip)."""
    y = rounded(rng.randn(T, 2 * G * K + H * V), dtype)
    q, k, v = y[:, :G * K].reshape(T, G, K), y[:, G * K:2 * G * K].reshape(T, G, K), y[:, 2 * G * K:].reshape(T, H, V)
    f32 = lambda a: torch.tensor(np.ascontiguousarray(a), dtype=torch.float32).cuda()
    if kind == 0:
        side = rng.randn(T, rank).astype(np.float32)
        a2, b = (rng.randn(H * K, rank) * 0.7).astype(np.float32), (2.0 + rng.randn(H * K)).astype(np.float32)
        if hard:                                                      # rows whose decays reach from none to e^-200
            side[::7] *= 12.0
            side[5::31] -= 40.0
        kw = dict(a2=f32(a2.T), a2_b=f32(b), inv_tau=1.0 if hard else 0.125, q_scale=0.3)
        z = side.astype(np.float64) @ a2.astype(np.float64).T + b
        decay = np.exp(-oh.softplus(-z) * kw["inv_tau"]).reshape(T, H, K)
        return y, side, kw, q * 0.3, k, v, decay, None
    side = rng.randn(T, H).astype(np.float32) - 2.0
    A_log, skip = (rng.randn(H) - 1.0).astype(np.float32), rng.randn(H).astype(np.float32)
    if hard:
        side[::9] += 30.0
        A_log[0] = 3.0
    own = np.arange(H) // (H // G)
    dt = oh.softplus(side.astype(np.float64))
    decay = np.exp(-np.exp(A_log.astype(np.float64)) * dt)[..., None] * np.ones(K)
    return (y, side, dict(A_log=f32(A_log), skip=f32(skip)), q[:, own], k[:, own] * dt[..., None], v, decay,
            skip.astype(np.float64))


REC = [  # kind, heads, groups, key size, value size, rank
    (0, 3, 3, 16, 24, 5), (0, 2, 2, 11, 9, 3), (0, 2, 2, 128, 96, 16), (0, 1, 1, 200, 40, 33), (0, 1, 1, 300, 33, 2),
    (1, 6, 3, 24, 16, 0), (1, 3, 1, 9, 7, 0), (1, 4, 2, 128, 64, 0), (1, 4, 4, 64, 136, 0), (1, 1, 1, 256, 8, 0)]


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("hard", [False, True])
@pytest.mark.parametrize("kind,H,G,K,V,rank", REC)
def test_recurrence(kind, H, G, K, V, rank, hard, dtype):
    """Row by row and in chunks, in portions of several sizes of three sequences side by side, slots that held other states."""
    from bitexact_llm_b200.hybrid import ops
    rng = np.random.RandomState(K + V)
    for cuts in ([200], [2, 3, 1, 64, 65, 1, 64], [130, 70], [3, 600]):
        T = sum(cuts)
        seqs, first = (3, 1, 2), {}
        for s in seqs:
            first[s] = recurrence_inputs(kind, H, G, K, V, rank, np.random.RandomState(s), T, dtype, hard)
        kw = first[3][2]
        if kind == 0:                                                 # one layer: the same weights for every sequence
            for s in seqs[1:]:
                y, side, _, q, k, v, _, _ = first[s]
                z = side.astype(np.float64) @ kw["a2"].double().cpu().numpy() + kw["a2_b"].double().cpu().numpy()
                first[s] = (y, side, kw, q, k, v, np.exp(-oh.softplus(-z) * kw["inv_tau"]).reshape(T, H, K), None)
        else:
            A, sk = kw["A_log"].double().cpu().numpy(), kw["skip"].double().cpu().numpy()
            for s in seqs[1:]:
                y, side, _, q, k, v, _, _ = first[s]
                dt = oh.softplus(side.astype(np.float64))
                first[s] = (y, side, kw, q, k, v, np.exp(-np.exp(A) * dt)[..., None] * np.ones(K), sk)
        want = {}
        for s in seqs:
            y, side, _, q, k, v, decay, skip = first[s]
            o, S = ov.linear_recurrence(q, k, v, decay)
            want[s] = (o + (0 if skip is None else skip[:, None] * v), S)
        chunked = dtype == "bfloat16" and K % 8 == 0 and V % 8 == 0 and K <= 256
        for use_tiles in (False, True) if chunked else (False,):
            state = torch.full((4, H, K, V), 3.0, device="cuda")
            got, at = {s: [] for s in seqs}, 0
            for n in cuts:
                runs = [(s, at, n) for s in seqs]
                st = steps(dtype, runs, 8, 1 + 4 * 80, 4)
                Y = packed(np.concatenate([first[s][0][at:at + n] for s in seqs]), dtype)
                side = torch.tensor(np.concatenate([first[s][1][at:at + n] for s in seqs])).cuda()
                o = ops.recurrence(kind, Y, side, state, st, G, (0, G * K, 2 * G * K), tiles=tiles_of(runs) if use_tiles else None, **kw)
                for i, s in enumerate(seqs):
                    got[s].append(o[i * n:(i + 1) * n, :H * V].float().cpu())
                at += n
            for s in seqs:
                close(torch.cat(got[s]).numpy().reshape(T, H, V), want[s][0], dtype, 0.2 if dtype == "bfloat16" else 1.0)
                close(state[s].cpu(), want[s][1], "float32", 1.0 if dtype == "float32" else 5.0)
            assert (state[0] == 3.0).all()


@pytest.mark.parametrize("dtype", DTYPES)
def test_a_state_lasts_over_a_long_pause(dtype):
    """Decays of almost one: what the first token wrote must come back unharmed a thousand tokens later."""
    from bitexact_llm_b200.hybrid import ops
    T, K, V = 1100, 32, 16
    rng = np.random.RandomState(0)
    y = np.zeros((T, 2 * K + V))
    y[0, K:] = rounded(rng.randn(K + V), dtype)                       # the only key and value
    y[-1, :K] = rounded(rng.randn(K), dtype)                          # the only query
    decay = np.ones((T, 1, K)) / (1 + np.exp(-9.0))
    o, _ = ov.linear_recurrence(y[:, None, :K], y[:, None, K:2 * K], y[:, None, 2 * K:], decay)
    assert abs(o[-1]).max() > 0.1
    kw = dict(a2=torch.zeros(1, K, device="cuda"), a2_b=torch.full((K,), 9.0, device="cuda"), inv_tau=1.0)
    for cuts, tiles in (([T], False), ([300, 1, 799], False), ([T], True), ([65, 1035], True)):
        if tiles and dtype == "float32":
            continue
        state, at = torch.zeros(1, 1, K, V, device="cuda"), 0
        for n in cuts:
            out = ops.recurrence(0, packed(y[at:at + n], dtype), torch.zeros(n, 1, device="cuda"), state,
                                 steps(dtype, [(0, at, n)], 8, 1 + 138, 1), 1, (0, K, 2 * K),
                                 tiles=tiles_of([(0, at, n)]) if tiles else None, **kw)
            at += n
        close(out[-1:, :V].float().cpu(), o[-1], dtype, 0.15 if dtype == "bfloat16" else 1.0)


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("taps,channels", [(1, 24), (2, 40), (3, 17), (4, 64), (4, 1032), (6, 32)])
def test_causal_convolution(taps, channels, dtype):
    """Portions down to single tokens, of sequences side by side, through the state that the gated norm advances."""
    from bitexact_llm_b200.hybrid import ops
    T = ops.DTYPES[dtype][0]
    rng = np.random.RandomState(taps + channels)
    n_all = 60
    w, b = rng.randn(channels, taps).astype(np.float32), rng.randn(channels).astype(np.float32)
    W, Bv = torch.tensor(w.T.copy()).cuda(), torch.tensor(b).cuda()
    us = {s: rounded(rng.randn(n_all, channels), dtype) for s in (2, 0)}
    want = {s: oh.silu(ov.causal_conv(u, w.astype(np.float64), b.astype(np.float64))) for s, u in us.items()}
    for cuts in ([60], [1] * 60, [2] * 30, [1, 2, 3, 20, 34]):
        state = torch.full((3, max(1, taps - 1), channels), 9.0, dtype=T, device="cuda")
        at, got = 0, {2: [], 0: []}
        for n in cuts:
            st = steps(dtype, [(2, at, n), (0, at, n)], 8, 1 + 3 * 8, 3)
            u = packed(np.concatenate([us[2][at:at + n], us[0][at:at + n]]), dtype)
            c = ops.conv_of(u, W, Bv, state, st)
            out = ops.causal_conv(c, 2 * n, u)
            one = torch.ones(2 * n, 8, dtype=T, device="cuda")
            ops.gated_norm(one, one, 8, 1, torch.ones(8, device="cuda"), 1e-5, True, conv=c)       # advances the state
            got[2].append(out[:n, :channels].float().cpu())
            got[0].append(out[n:, :channels].float().cpu())
            at += n
        for s in us:
            close(torch.cat(got[s]), want[s], dtype, 0.3)
        assert (state[1] == 9.0).all()


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("n,parts,wn", [(24, 3, 8), (45, 5, 9), (96, 1, 96), (1536, 2, 1536), (1100, 1, 1100), (4096, 32, 128), (77, 7, 77)])
@pytest.mark.parametrize("gate_first", [True, False])
def test_gated_norm(n, parts, wn, gate_first, dtype):
    from bitexact_llm_b200.hybrid import ops
    rng = np.random.RandomState(n)
    M, eps = 5, 0.02
    o, z, w = rounded(rng.randn(M, n), dtype), rounded(rng.randn(M, n), dtype), rng.randn(wn).astype(np.float32)
    o[1] *= 1e-3                                                      # eps counts
    o = rounded(o, dtype)
    got = ops.gated_norm(packed(o, dtype), packed(z, dtype), n, parts, torch.tensor(w).cuda(), eps, gate_first)
    s, w64 = oh.silu(z), np.tile(w.astype(np.float64), n // wn)
    v = (o * s if gate_first else o).reshape(M, parts, -1)
    want = oh.rms_norm(v, 1.0, eps).reshape(M, n) * w64 * (1.0 if gate_first else s)
    close(got[:, :n].float().cpu(), want, dtype, 0.3)


LAYERS = [("looped", 1), ("looped", 2), ("looped", 3), ("odd", 0), ("odd", 2), ("one", 0), ("one", 1), ("wide", 1), ("wide", 2)]


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("name,layer", LAYERS)
@pytest.mark.parametrize("cuts", [[200], [1] * 25, [2, 3, 2, 61, 64, 5, 63], [129, 71]])
def test_recurrent_layer_in_portions(name, layer, cuts, dtype):
    cfg, w64, eng = model(name, dtype)
    kind, m = cfg["layers"][layer]["type"], cfg["layers"][layer]["mixer"]
    from bitexact_llm_b200.hybrid.engine import MIXERS
    mixer = MIXERS[type(eng.spec.layers[layer].mixer)](
        {k[len(f"l{layer}.mix."):]: v for k, v in vm.weights(cfg).items() if k.startswith(f"l{layer}.mix.")},
        eng.spec.layers[layer].mixer, cfg["width"], eng.dtype, "cuda")
    rng = np.random.RandomState(layer)
    T, D, eps = sum(cuts), cfg["width"], cfg["norm"]["eps"]
    hs = [rounded(rng.randn(T, D), dtype) for _ in range(3)]
    f = ov.mamba2 if kind == "mamba2" else ov.gla
    want, ends = zip(*[f(h, oh.sub(w64, f"l{layer}.mix."), m, eps) for h in hs])
    cache = mixer.new_cache(4, 2, 4)
    parts = cache if isinstance(cache, tuple) else (cache,)
    for c in parts:
        c.fill_(3.0)                                                  # what an earlier request left
    got, at = [[], [], []], 0
    for n in cuts:                                                    # three sequences side by side, slots 3, 1, 2
        runs = [(s, at, n) for s in (3, 1, 2)]
        st = steps(dtype, runs, 4, 1 + 4 * 51, 4, tiles_of(runs) if dtype == "bfloat16" and n > 1 else None)
        x = torch.zeros(3 * n, D, device="cuda")
        mixer.run(st, packed(np.concatenate([v[at:at + n] for v in hs]), dtype), x, cache)
        for i in range(3):
            got[i].append(x[i * n:(i + 1) * n].cpu())
        at += n
    for i, s in enumerate((3, 1, 2)):
        mostly(torch.cat(got[i]), want[i], dtype)
        close(parts[0][s].cpu(), ends[i], dtype)
    assert all((c[0] == 3.0).all() for c in parts)


# ---------------------------------------------------------------- whole models

@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("name", list(vm.CONFIGS))
def test_residual_after_every_layer_run(name, dtype):
    cfg, w64, eng = model(name, dtype)
    toks = hm.tokens(cfg, 90, 5)
    _, after = ov.forward(cfg, w64, toks)
    runs = eng.layers
    assert len(runs) == len(after) == eng.L
    try:
        for k in range(1, len(runs) + 1):
            eng.layers = runs[:k]
            mostly(session(eng).feed([(0, toks)])[0].cpu(), after[k - 1], dtype)
    finally:
        eng.layers = runs


PORTIONS = {"whole": [260], "tokens": [1] * 260, "twos": [2] * 130, "threes_and_sevens": [3, 7] * 26,
            "pages": [16, 15, 17, 1, 64, 63, 65, 19], "long_then_tokens": [200] + [1] * 60}


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("name", list(vm.CONFIGS))
@pytest.mark.parametrize("cut", list(PORTIONS))
def test_portions_and_decoding(name, cut, dtype):
    cfg, _, eng = model(name, dtype)
    toks = hm.tokens(cfg, 260, 1)
    ses = session(eng, 3, 272, bs=16 if cut == "pages" else None, perm_seed=4)
    at, rows = 0, []
    for n in PORTIONS[cut]:
        rows += ses.feed([(1, toks[at:at + n])])
        at += n
    mostly(logits(eng, torch.cat(rows)), want_logits(name, toks), dtype)


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("name", list(vm.CONFIGS))
def test_mixed_batches_match_each_request_alone(name, dtype):
    """Prompts, portions and single tokens of several requests in one call, slots and pages handed on between them."""
    cfg, _, eng = model(name, dtype)
    lens = {"a": 150, "b": 1, "c": 67, "d": 3, "e": 200}
    toks = {k: hm.tokens(cfg, n, i + 10) for i, (k, n) in enumerate(lens.items())}
    plan = [[("a", 40), ("b", 1), ("c", 2)], [("a", 2), ("c", 33)], [("a", 1), ("c", 1), ("d", 3)], [("c", 31), ("a", 57)],
            [("e", 100), ("a", 1)], [("a", 49), ("e", 1)]] + [[("e", 1)]] * 3 + [[("e", 96)]]
    ses = session(eng, 3, 208, bs=16, pages=26)
    slot, at, got, idle = {}, {k: 0 for k in lens}, {k: [] for k in lens}, [2, 0, 1]
    for entries in plan:
        for k, _ in entries:
            if k not in slot:
                slot[k] = idle.pop()
        for (k, n), r in zip(entries, ses.feed([(slot[k], toks[k][at[k]:at[k] + n]) for k, n in entries])):
            got[k].append(r)
            at[k] += n
            if at[k] == lens[k]:
                ses.release(slot[k])
                idle.append(slot.pop(k))
    assert at == lens and len(ses.free) == 26
    for k in lens:
        mostly(logits(eng, torch.cat(got[k])), want_logits(name, toks[k]), dtype)


@pytest.mark.parametrize("name", list(vm.CONFIGS))
def test_the_batch_changes_nothing_beyond_rounding(name):
    cfg, _, eng = model(name, "float32")
    a, b = hm.tokens(cfg, 120, 30), hm.tokens(cfg, 45, 31)
    alone = logits(eng, session(eng).feed([(0, a)])[0])
    ses = session(eng, 4)
    both = ses.feed([(2, b), (3, a)])[1]
    assert np.abs(logits(eng, both) - alone).max() < 1e-4 * np.abs(alone).max()


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("name", ["looped", "wide"])
def test_large_decoding_batch(name, dtype):
    """Eighty sequences of unequal lengths step together: one row each, neighbours in the kernels' row groups."""
    cfg, _, eng = model(name, dtype)
    n, more = 80, 3
    toks = {s: hm.tokens(cfg, 1 + s % 7 + more, 100 + s) for s in range(n)}
    ses = session(eng, n, 32)
    order = [(7 * s) % n for s in range(n)]
    got = {s: [x] for s, x in zip(order, ses.feed([(s, toks[s][:-more]) for s in order]))}
    for k in range(more):
        for s, x in zip(order, ses.feed([(s, [toks[s][k - more]]) for s in order])):
            got[s].append(x)
    for s in (0, 1, 5, 6, 7, 33, 63, 64, 79):
        mostly(logits(eng, torch.cat(got[s])), want_logits(name, toks[s]), dtype)


@pytest.mark.parametrize("name", list(vm.CONFIGS))
def test_greedy_generation_of_an_unequal_batch(name):
    from bitexact_llm_b200.decode import generate
    cfg, w64, eng = model(name, "float32")
    prompts = [hm.tokens(cfg, n, 40 + n) for n in (37, 1, 20)]
    ids = torch.zeros(3, 37, dtype=torch.long)
    for i, p in enumerate(prompts):
        ids[i, : len(p)] = torch.tensor(p)
    toks, _ = generate(eng, ids, 12, lens=torch.tensor([len(p) for p in prompts]), perm_seed=7)
    assert toks.tolist() == [ov.greedy(cfg, w64, p, 12) for p in prompts]


@pytest.mark.parametrize("dtype", DTYPES)
def test_long_decoding(dtype):
    from bitexact_llm_b200.decode import generate
    cfg, w64, eng = model("looped", dtype)
    prompt = hm.tokens(cfg, 5, 77)
    toks, _ = generate(eng, torch.tensor([prompt]), 400, hashes=False)
    seq = prompt + toks[0].tolist()
    want, _ = ov.forward(cfg, w64, seq[:-1])
    rows, ses = [], session(eng, 1, 512)
    for t in seq[:-1]:
        rows += ses.feed([(0, [t])])
    lg = logits(eng, torch.cat(rows))
    mostly(lg, want, dtype)
    assert (lg[4:].argmax(-1) == np.array(seq[5:])).mean() > 0.99


@pytest.mark.parametrize("name", ["looped", "wide"])
def test_decode_graph_matches_the_eager_loop(name):
    from bitexact_llm_b200.decode import GraphDecoder, Session, generate
    cfg, _, eng = model(name, "bfloat16")
    ids = torch.tensor([hm.tokens(cfg, 30, 50 + i) for i in range(4)])
    want, _ = generate(eng, ids, 12, 7, 10, hashes=False)
    ses = Session(eng, 4, 64)
    h = ses.prefill(ids)
    rows = torch.zeros(4, 4, dtype=torch.long, device="cuda")
    rows[:, 0], rows[:, 2], rows[:, 3] = torch.arange(4), 7, 10
    dec = GraphDecoder(ses, rows, h, warmup=0)
    got = torch.stack([dec.step().clone() for _ in range(12)], 1).cpu()
    assert torch.equal(got, want)


@pytest.mark.parametrize("dtype", DTYPES)
def test_padding_rows_touch_nothing(dtype):
    cfg, _, eng = model("looped", dtype)
    toks = hm.tokens(cfg, 20, 9)
    want = logits(eng, session(eng).feed([(0, toks)])[0])
    ses = session(eng, 2, 64)
    ids = torch.tensor(toks + [0] * 5).cuda()
    pos = torch.tensor(list(range(20)) + [0] * 5).cuda()
    seq = torch.tensor([1] * 20 + [0] * 5).cuda()
    slot = torch.where(torch.arange(25).cuda() < 20, ses._slots(seq, pos), torch.full_like(pos, -1))
    ses.feed([(0, [3, 4])])
    states = lambda: [t[0].clone() for c in ses.kvs if not (torch.is_tensor(c) and c.shape[0] != 2) for t in (c if isinstance(c, tuple) else (c,))]
    before = states()
    assert len(before) == 7                                           # two mamba runs of two parts, three gated linear ones
    x = eng.forward(ses.kvs, ids, pos, slot, ses.bt, seq)
    mostly(logits(eng, x[:20]), want, dtype)
    assert all(torch.equal(a, b) for a, b in zip(before, states()))


# ---------------------------------------------------------------- commands

def test_trace_run_and_generate_commands(tmp_path):
    cfg = vm.CONFIGS["odd"]
    t = vm.weights(cfg, 3)
    w64 = hm.as_numpy(t)
    folder = hm.save_folder(tmp_path / "m", cfg, t)
    a, b = hm.tokens(cfg, 50, 1), hm.tokens(cfg, 20, 2)
    trace = [{"step": 0, "entries": [{"id": "a", "tokens": a[:30], "want": [0, 29]}], "end": []},
             {"step": 1, "entries": [{"id": "b", "tokens": b, "want": []}, {"id": "a", "tokens": a[30:31], "want": [0]}], "end": ["b"]},
             {"step": 2, "entries": [{"id": "a", "tokens": a[31:], "want": [18, 0]}], "end": ["a"]},
             {"step": 5, "entries": [{"id": "c", "tokens": b[:2], "want": [1]}], "end": ["c"]}]
    want_a, want_b = ov.forward(cfg, w64, a)[0], ov.forward(cfg, w64, b)[0]
    expect = {0: want_a[[0, 29]], 1: want_a[[30]], 2: want_a[[49, 31]], 5: want_b[[1]]}
    for dtype in DTYPES:
        out = tmp_path / dtype
        out.mkdir()
        r = subprocess.run([os.path.join(ROOT, "bin", "trace_run"), "--model", folder, "--dtype", dtype, "--out", str(out),
                            "--max-tokens", "70"], input="".join(json.dumps(s) + "\n" for s in trace), capture_output=True, text=True)
        assert r.returncode == 0, r.stderr
        assert [ln for ln in r.stdout.splitlines() if ln.startswith("done")] == ["done 0", "done 1", "done 2", "done 5"]
        for s, e in expect.items():
            mostly(np.fromfile(out / f"{s}.f32", "<f4").reshape(e.shape), e, dtype)
    r = subprocess.run([sys.executable, "-m", "bitexact_llm_b200", "generate", "--model", folder, "--dtype", "float32", "--max-new",
                        "6", "--prompt", ",".join(map(str, a[:9])), "--prompt", ",".join(map(str, b[:4]))],
                       cwd=ROOT, capture_output=True, text=True)
    assert r.returncode == 0, r.stderr
    assert [[int(v) for v in ln.split(",")] for ln in r.stdout.split()] == [ov.greedy(cfg, w64, a[:9], 6), ov.greedy(cfg, w64, b[:4], 6)]
