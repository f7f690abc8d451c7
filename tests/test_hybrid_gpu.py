"""Hybrid float models on the GPU against the plain float64 oracle (oracle/hybrid.py): every mechanism alone, whole
prompts, portions, decoding through the caches, unequal batches, reused pages and slots, greedy generation, the command
lines.  Everything runs in both number formats."""

import json
import os
import subprocess
import sys

import numpy as np
import pytest
import torch

import hybrid_models as hm
from oracle import hybrid as oh

pytestmark = pytest.mark.gpu
ROOT = os.path.dirname(os.path.dirname(os.path.abspath(__file__)))
DTYPES = ("float32", "bfloat16")
TOL = {"float32": 2e-4, "bfloat16": 0.06}                 # rms of the difference over rms of the values, per row
_cache = {}


def config(name, dtype):
    return hm.CONFIGS[name] if dtype == "float32" else hm.settled(hm.CONFIGS[name])


def model(name, dtype):
    """(config, oracle weights, engine), built once."""
    if (name, dtype) not in _cache:
        from bitexact_llm_b200.hybrid import fedatar
        cfg = config(name, dtype)
        t = hm.weights(cfg)
        _cache[name, dtype] = (cfg, hm.as_numpy(t), fedatar.load(cfg, t, "cuda", dtype))
    return _cache[name, dtype]


def want_logits(name, dtype, toks):
    key = (name, dtype, tuple(toks))
    if key not in _cache:
        cfg, w64, _ = model(name, dtype)
        _cache[key] = oh.forward(cfg, w64, toks)[0]
    return _cache[key]


def close(got, want, dtype, scale=1.0):
    got, want = np.asarray(got, np.float64), np.asarray(want, np.float64)
    assert got.shape == want.shape and np.isfinite(got).all()
    g, w = got.reshape(-1, got.shape[-1]), want.reshape(-1, want.shape[-1])
    err = np.sqrt(((g - w) ** 2).mean(-1))
    ref = np.sqrt((w ** 2).mean(-1)) + 0.1 * np.sqrt((w ** 2).mean())
    worst = (err / ref).max()
    assert worst < TOL[dtype] * scale, (worst, int((err / ref).argmax()))


def session(eng, n_seqs=1, max_len=512, **kw):
    from bitexact_llm_b200.decode import Session
    return Session(eng, n_seqs, max_len, **kw)


def logits(eng, x):
    out = eng.logits_float(x).cpu().numpy()
    eng.check()
    return out


def packed(w, dtype):
    from bitexact_llm_b200.hybrid import ops
    return ops.pack(torch.as_tensor(w), ops.DTYPES[dtype][0], "cuda")


def rounded(a, dtype):
    """The values a tensor of the format holds."""
    t = torch.as_tensor(a)
    return (t.float() if dtype == "float32" else t.to(torch.bfloat16)).double().numpy()


# ---------------------------------------------------------------- products and their epilogues

@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("M,N,K,tile", [(1, 5, 7, 0), (1, 300, 2048, 0), (16, 129, 72, 0), (33, 260, 1030, 0), (70, 64, 64, 0),
                                        (200, 140, 200, 0), (200, 140, 200, 16), (300, 257, 520, 256), (300, 257, 520, 128)])
def test_linear_sizes_and_tiles(M, N, K, tile, dtype):
    from bitexact_llm_b200.hybrid import ops
    rng = np.random.RandomState(M + N + K)
    w, x = rounded(rng.randn(N, K), dtype), rounded(rng.randn(M, K), dtype)
    W, X = packed(w, dtype), packed(x, dtype)
    out = torch.full((M, N + 3), 7.0, device="cuda")
    ops.linear(W, X, M, N, K, ops.store(out, N + 3, N, out_type=ops.OUT_F32), tile=tile)
    close(out[:, :N].cpu(), x @ w.T, "float32")
    assert (out[:, N:] == 7.0).all()                                  # nothing beside the output
    fix = torch.zeros(M, N, dtype=torch.long, device="cuda")
    ops.linear(W, X, M, N, K, ops.store(fix, N, N, out_type=ops.OUT_I64), tile=tile)
    assert torch.equal(fix, torch.round(out[:, :N].double() * 2 ** 24).long())
    ops.linear(W, X, M, N, K, ops.add(out), tile=tile)
    close(out[:, :N].cpu(), 2 * (x @ w.T), "float32")


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("counts", [[3, 0, 1, 9], [0, 0, 0, 5], [40, 1, 0, 33], [300, 2, 130, 77], [1] * 70])
def test_ragged_groups(counts, dtype):
    from bitexact_llm_b200.hybrid import ops
    rng = np.random.RandomState(len(counts) + sum(counts))
    G, M, N, K = len(counts), sum(counts), 150, 90
    w, x = rounded(rng.randn(G, N, K), dtype), rounded(rng.randn(M, K), dtype)
    W, X = packed(w, dtype), packed(x, dtype)
    out = torch.full((M, N), 7.0, device="cuda")
    c = torch.tensor(counts, dtype=torch.int32, device="cuda")
    group = np.repeat(np.arange(G), counts)
    ref = np.einsum("mk,mnk->mn", x, w[group])
    for tile in ((0,) if dtype == "float32" else (0, 16, 64, 128, 256)):
        out.fill_(7.0)
        ops.linear(W, X, M, N, K, ops.store(out, N, N, out_type=ops.OUT_F32), groups=G, gsw=N * W.shape[2], counts=c, tile=tile)
        close(out.cpu(), ref, "float32")


@pytest.mark.parametrize("dtype", DTYPES)
def test_activations_side_output_and_gate(dtype):
    from bitexact_llm_b200 import _native as nv
    from bitexact_llm_b200.hybrid import ops
    rng = np.random.RandomState(0)
    M, N, E, K = 37, 50, 9, 40
    w, x, b = rounded(rng.randn(N + E, K), dtype), rounded(rng.randn(M, K), dtype), rng.randn(E)
    W, X = packed(w, dtype), packed(x, dtype)
    acc = x @ w.T
    for act, f in (("none", lambda v: v), ("relu2", oh.relu2), ("xielu", lambda v: oh.xielu(v, 0.2, -1.3))):
        out = torch.zeros(M, 56, dtype=W.dtype, device="cuda")
        side = torch.zeros(M, E, device="cuda")
        p, q = np.log1p(np.exp(0.2)), 0.5 + np.log1p(np.exp(-1.3))
        ops.linear(W, X, M, N + E, K, ops.store(out, 56, N, act, p, q, side=side, bias=torch.tensor(b, dtype=torch.float32).cuda()))
        close(out[:, :N].float().cpu(), f(acc[:, :N]), dtype)
        close(side.cpu(), acc[:, N:] + b, "float32")
    H, V = 3, 16                                                      # groups = heads, one gate each
    w, x = rounded(rng.randn(H, V, 24), dtype), rounded(rng.randn(M, H, 24), dtype)
    gate = torch.rand(M, H, device="cuda")
    W, X = packed(w, dtype), packed(x, dtype)
    out = torch.zeros(M, H * V, dtype=W.dtype, device="cuda")
    ops.linear(W, X, M, V, 24, nv.Epilogue(kind=ops.GATE, n_main=V, out=out.data_ptr(), ldo=H * V, gso=V, gate=gate.data_ptr(), ldg=H),
               groups=H, gsw=V * W.shape[2], ldx=H * 24, gsx=24)
    close(out.float().cpu(), (np.einsum("mhk,hvk->mhv", x, w) * gate.cpu().numpy()[..., None]).reshape(M, -1), dtype)


# ---------------------------------------------------------------- norms, routing, rotation

@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("D", [52, 256, 1030])
def test_norm_embedding_and_expert_sum(D, dtype):
    from bitexact_llm_b200.hybrid import ops
    T = ops.DTYPES[dtype][0]
    rng = np.random.RandomState(D)
    M, V, top = 9, 30, 3
    emb = torch.tensor(rng.randn(V, D) + 3.0).to(T).cuda()            # a mean the variance must not see
    w, b = (torch.tensor(rng.randn(D), dtype=torch.float32).cuda() for _ in range(2))
    ids = torch.tensor(rng.randint(0, V, M)).cuda()
    x, h = torch.empty(M, D, device="cuda"), torch.zeros(M, ops.pad8(D), dtype=T, device="cuda")
    zero = torch.full((5,), 3, dtype=torch.int32, device="cuda")
    ops.norm(x, w, b, 1e-3, h, ids=ids, embed=emb, zero=zero)
    x0 = emb[ids].double().cpu().numpy()
    assert np.array_equal(x.double().cpu().numpy(), x0) and int(zero.abs().sum()) == 0
    n64 = lambda v: oh.layer_norm(v, w.double().cpu().numpy(), b.double().cpu().numpy(), 1e-3)
    close(h[:, :D].float().cpu(), n64(x0), dtype)
    y = torch.tensor(rng.randn(M * top, D), dtype=torch.float32).cuda()
    place = torch.randperm(M * top).int().view(M, top).cuda()
    wt = torch.rand(M, top, device="cuda")
    ops.norm(x, w, b, 1e-3, h, experts=(y, place, wt))
    x1 = x0 + (y.cpu().double().numpy()[place.cpu().numpy()] * wt.cpu().double().numpy()[..., None]).sum(1)
    close(x.cpu(), x1, "float32")
    close(h[:, :D].float().cpu(), n64(x1), dtype)
    keep = x.clone()
    ops.norm(x, None, None, 1e-3, experts=(y, place, wt))             # only the sum
    close(x.cpu(), keep.double().cpu().numpy() + (x1 - x0), "float32")


@pytest.mark.parametrize("E,top", [(1, 1), (5, 2), (64, 8), (100, 32), (1024, 6)])
def test_routing_and_gathering(E, top):
    from bitexact_llm_b200.hybrid import ops
    rng = np.random.RandomState(E)
    M = 41
    z = rng.randn(M, E).astype(np.float32)
    z[3] = 0.25                                                       # all equal: the lowest indices
    z[4] = -50.0
    lg = torch.tensor(z).cuda()
    counts = torch.zeros(E, dtype=torch.int32, device="cuda")
    chosen, weight, rank = ops.route(lg, E, top, counts)
    idx, wt = oh.route(np.eye(E), np.zeros((E, E)), np.zeros(E), top)
    z64 = z.astype(np.float64)
    idx = np.argsort(-z64, -1, kind="stable")[:, :top]
    e = np.exp(np.take_along_axis(z64, idx, -1) - z64.max(-1, keepdims=True))
    assert np.array_equal(chosen.cpu().numpy(), idx)
    assert np.allclose(weight.cpu().numpy(), e / e.sum(-1, keepdims=True), atol=1e-6)
    assert np.array_equal(counts.cpu().numpy(), np.bincount(idx.ravel(), minlength=E))
    h = torch.randn(M, 24, device="cuda")
    hp, place = ops.gather(h, 20, chosen, rank, counts)
    assert sorted(place.flatten().tolist()) == list(range(M * top))
    order = np.empty(M * top, int)
    order[place.cpu().numpy().ravel()] = idx.ravel()
    assert (np.diff(order) >= 0).all()
    assert torch.equal(hp[place.long(), :20], h[:, None, :20].expand(M, top, 20))


# ---------------------------------------------------------------- layers alone

def steps(eng_dtype, runs, bs, n_blocks, n_seqs, tiles=None):
    """Step of runs = [(sequence, first position, tokens)]; sequence s owns pages 1 + s * n .. in reverse order."""
    from bitexact_llm_b200.hybrid import ops
    from bitexact_llm_b200.hybrid.layers import Step
    per = (n_blocks - 1) // n_seqs
    bt = torch.stack([torch.arange(1 + s * per, 1 + (s + 1) * per).flip(0) for s in range(n_seqs)]).int().cuda()
    seq = torch.cat([torch.full((n,), s) for s, _, n in runs]).cuda()
    pos = torch.cat([torch.arange(p, p + n) for _, p, n in runs]).cuda()
    slot = bt[seq, pos // bs].long() * bs + pos % bs
    return Step(pos, slot, seq, bt, ops.row_flags(seq, slot, pos), tiles)


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("cuts", [[400], [1] * 30, [2, 3, 2, 61, 64, 65, 5, 128, 70], [129, 271]])
def test_mingru_layer_in_portions(cuts, dtype):
    from bitexact_llm_b200.hybrid import ops
    from bitexact_llm_b200.hybrid.layers import MinGRU
    from bitexact_llm_b200.hybrid.spec import MinGRUSpec
    cfg = hm.CONFIGS["odd"]
    w = {k[len("l0.mix."):]: v for k, v in hm.weights(cfg).items() if k.startswith("l0.mix.")}
    D, W, T = cfg["width"], 90, sum(cuts)
    layer = MinGRU(w, MinGRUSpec(W), D, ops.DTYPES[dtype][0], "cuda")
    rng = np.random.RandomState(T)
    hs = [rounded(rng.randn(T, D), dtype) for _ in range(3)]
    w64 = hm.as_numpy(w)
    want, ends = zip(*[oh.mingru(h, w64["z"], w64["z.b"], w64["x"], w64["x.b"], w64["g"], w64["o"]) for h in hs])
    cache = layer.new_cache(4, 2, 4)
    cache.fill_(3.0)                                                  # what an earlier request left
    got, at = [[], [], []], 0
    for n in cuts:                                                    # three sequences side by side, slots 3, 1, 2
        h = packed(np.concatenate([v[at:at + n] for v in hs]), dtype)
        st = steps(dtype, [(s, at, n) for s in (3, 1, 2)], 4, 1 + 4 * 101, 4)
        x = torch.zeros(3 * n, D, device="cuda")
        layer.run(st, h, x, cache)
        for i in range(3):
            got[i].append(x[i * n:(i + 1) * n].cpu())
        at += n
    for i, s in enumerate((3, 1, 2)):
        close(torch.cat(got[i]), want[i], dtype)
        close(cache[s].cpu()[None], ends[i][None], dtype)
    assert (cache[0] == 3.0).all()


def test_mingru_holds_its_state_over_a_long_pause():
    """Gates almost shut: the value written at the first token must survive hundreds of tokens, also over tiles."""
    from bitexact_llm_b200.hybrid import ops
    from bitexact_llm_b200.hybrid.layers import MinGRU
    from bitexact_llm_b200.hybrid.spec import MinGRUSpec
    D, W, T = 16, 24, 700
    w = {"z": torch.zeros(W, D), "x": torch.zeros(W, D), "g": torch.zeros(W, D), "o": torch.zeros(D, W),
         "z.b": torch.full((W,), -6.0), "x.b": torch.zeros(W)}
    w["z"][:, 0] = 14.0                                               # entry 0 of the input opens the gate
    w["x"][:, 1] = torch.linspace(-2, 2, W)
    w["g"][:, 2] = 1.0
    w["o"][:, :D] = torch.eye(D)
    h = np.zeros((T, D))
    h[0, :2] = 1.0
    h[:, 2] = 1.0
    want, _ = oh.mingru(h, *(w[k].double().numpy() for k in ("z", "z.b", "x", "x.b", "g", "o")))
    assert abs(want[500]).max() > 0.1 * abs(want[0]).max()
    for dtype in DTYPES:
        layer = MinGRU(w, MinGRUSpec(W), D, ops.DTYPES[dtype][0], "cuda")
        for cuts in ([T], [1, 699], [300, 400]):
            cache, x, at = layer.new_cache(1, 2, 8), torch.zeros(T, D, device="cuda"), 0
            for n in cuts:
                layer.run(steps(dtype, [(0, at, n)], 8, 1 + 90, 1), packed(h[at:at + n], dtype), x[at:at + n], cache)
                at += n
            close(x.cpu(), want, dtype, 0.3)


SHAPES = [  # heads, latent, rotated, window, page size
    (3, 48, 8, 19, 4), (1, 23, 2, 0, 16), (5, 50, 6, 33, 8), (12, 128, 32, 130, 16), (16, 272, 16, 65, 32), (40, 96, 32, 64, 16),
    (130, 64, 8, 20, 16), (4, 512, 64, 100, 64), (8, 320, 64, 0, 128)]


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("H,R,rot,window,bs", SHAPES)
def test_latent_attention_core(H, R, rot, window, bs, dtype):
    """The kernels on given queries and cache rows: every variant, rows and tiles, contexts of several lengths."""
    from bitexact_llm_b200.hybrid import ops
    from bitexact_llm_b200.hybrid.spec import LatentAttentionSpec
    from bitexact_llm_b200 import _native as nv
    T = ops.DTYPES[dtype][0]
    sp = LatentAttentionSpec(H, 1, rot, 1, 1, R, 1.0, 0.11, window, 1e-5)
    rng = np.random.RandomState(H + R)
    runs = [(1, 0, 70), (0, 190, 9), (2, 63, 2), (1, 128, 1)]         # (sequence, first position, rows)
    per = (256 + bs - 1) // bs
    st = steps(dtype, runs, bs, 1 + 3 * per, 3)
    M = st.pos.shape[0]
    q, cache = rounded(rng.randn(M, H, R + rot), dtype), rounded(rng.randn(1 + 3 * per, bs, R + rot), dtype)
    Q, C = packed(q, dtype), packed(cache, dtype)
    sink = rng.randn(H)
    want = np.zeros((M, H, R))
    for m in range(M):
        s, i = int(st.seq[m]), int(st.pos[m])
        js = np.arange(max(0, i - window + 1) if window else 0, i + 1)
        rows = cache[st.bt[s].cpu().numpy()[js // bs], js % bs]
        e = np.exp(q[m] @ rows.T * 0.11)
        want[m] = e @ rows[:, :R] / (e.sum(-1) + np.exp(sink))[:, None]
    sinks = torch.tensor(sink, dtype=torch.float32).cuda()
    n = nv.float_lib().bxf_latent_attention_tile(H)
    tiles, row = [], 0
    for s, p, k in runs:
        tiles += [(s, row + a, min(n, k - a)) for a in range(0, k, n)]
        row += k
    tiles = torch.tensor(tiles, dtype=torch.int32).cuda()
    tc = dtype == "bfloat16" and bs >= 8
    for variant, tt in [(0, None), (0, tiles), (1, None)] + ([(2, None), (2, tiles)] if tc else []):
        out = ops.latent_attention(Q, sp, C, st.bt, st.seq, st.pos, sinks, tt, variant)
        close(out[..., :R].float().cpu(), want, dtype, 0.5)
        if variant == 2 and tt is None:                               # one row alone: its keys are split over CTAs
            for m in (0, 72, 78, M - 1):
                one = ops.latent_attention(Q[m:m + 1].contiguous(), sp, C, st.bt, st.seq[m:m + 1].contiguous(),
                                           st.pos[m:m + 1].contiguous(), sinks, None, 2)
                close(one[..., :R].float().cpu(), want[m:m + 1], dtype, 0.5)
    assert nv.float_device_status() == 0


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("window", [16, 40, 63, 64, 65, 100])
def test_one_key_stands_out_at_every_distance(window, dtype):
    """One cached key gets nearly all the weight of every query that sees it, and none of the others': a window that is
    off by one, a page mix-up or a lost block shows as the marker's presence or absence. Also with a dominating sink."""
    from bitexact_llm_b200.hybrid import ops
    from bitexact_llm_b200.hybrid.spec import LatentAttentionSpec
    T = ops.DTYPES[dtype][0]
    H, R, rot, bs, n = 4, 64, 16, 16, 260
    sp = LatentAttentionSpec(H, 1, rot, 1, 1, R, 1.0, 1.0, window, 1e-5)
    st = steps(dtype, [(0, 0, n)], bs, 1 + 17, 1)
    q = np.zeros((n, H, R + rot))
    q[..., R] = 1.0                                                   # reads the rotated part's first entry
    tiles = torch.tensor([(0, a, min(32, n - a)) for a in range(0, n, 32)], dtype=torch.int32).cuda()
    for far in (0, 15, 16, 47, 63, 64, 127, 130):
        rows = np.zeros((n, R + rot))
        rows[:, 0] = 1.0
        rows[far, :2] = (0.0, 1.0)                                    # the marker's value
        rows[far, R] = 20.0
        cache = np.zeros((18, bs, R + rot))
        b = st.bt[0].cpu().numpy()
        for j in range(n):
            cache[b[j // bs], j % bs] = rows[j]
        for sink, full in ((-30.0, 1.0), (40.0, 0.0)):
            s = torch.full((H,), sink, device="cuda")
            for tt in (None, tiles):
                out = ops.latent_attention(packed(q, dtype), sp, packed(cache, dtype), st.bt, st.seq, st.pos, s, tt)
                got = out[..., 1].float().cpu().numpy()
                i = np.arange(n)
                seen = (i >= far) & (i - far < window)
                assert np.allclose(got, (seen * full)[:, None], atol=1e-2), (far, sink)
                if full:
                    assert np.allclose(out[..., 0].float().cpu().numpy(), (1.0 - seen)[:, None], atol=1e-2)


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("name,layer", [("plain", 0), ("plain", 3), ("odd", 1), ("odd", 2), ("wide", 1), ("wide", 3)])
def test_latent_attention_layer(name, layer, dtype):
    from bitexact_llm_b200.hybrid.spec import LatentAttentionSpec
    cfg, w64, eng = model(name, dtype)
    mixer, m = eng.layers[layer][1], cfg["layers"][layer]["mixer"]
    assert isinstance(mixer.spec, LatentAttentionSpec)
    n, D = 150, cfg["width"]
    rng = np.random.RandomState(layer)
    h = rounded(rng.randn(n, D), dtype)
    want = oh.latent_attention(h, oh.sub(w64, f"l{layer}.mix."), m, cfg["norm"]["eps"])
    for cuts in ([n], [70, 2, 3, 1, 1, 70, 3]):
        cache, x, at = mixer.new_cache(1, 12, 16), torch.zeros(n, D, device="cuda"), 0
        for k in cuts:
            st = steps(dtype, [(0, at, k)], 16, 12, 1)
            tt = eng.tile_table([(0, 0, k, at + k)], 16)
            st.tiles = None if tt is None or k == 1 else tt.to("cuda")
            mixer.run(st, packed(h[at:at + k], dtype), x[at:at + k], cache)
            at += k
        close(x.cpu(), want, dtype)


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("name,layer", [("plain", 0), ("plain", 1), ("odd", 0), ("odd", 1), ("wide", 0), ("wide", 1), ("wide", 2)])
@pytest.mark.parametrize("n", [1, 2, 45, 300])
def test_feed_forward_layers(name, layer, n, dtype):
    from bitexact_llm_b200.hybrid import ops
    cfg, w64, eng = model(name, dtype)
    ff, f = eng.layers[layer][3], cfg["layers"][layer]["mlp"]
    rng = np.random.RandomState(n)
    h = rounded(rng.randn(n, cfg["width"]), dtype)
    w = oh.sub(w64, f"l{layer}.mlp.")
    x = torch.ones(n, cfg["width"], device="cuda")
    counts = torch.zeros(max(1, ff.counters), dtype=torch.int32, device="cuda")
    due = ff.run(packed(h, dtype), x, counts[: ff.counters])
    if f["kind"] == "dense":
        assert due is None
        want = oh.dense_ff(h, w["up"], w["down"], w["act"])
    else:
        ops.norm(x, None, None, 1e-5, experts=due)
        want = oh.moe_ff(h, w, f["router"]["experts"], f["router"]["top"], f.get("shared"))
    close(x.cpu().numpy() - 1.0, want, dtype)


# ---------------------------------------------------------------- whole models

@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("name", list(hm.CONFIGS))
def test_residual_stream_after_every_layer(name, dtype):
    cfg, w64, eng = model(name, dtype)
    toks = hm.tokens(cfg, 90, 5)
    _, streams = oh.forward(cfg, w64, toks)
    all_layers, L = eng.layers, eng.L
    try:
        for k in range(1, L + 1):
            eng.layers, eng.L = all_layers[:k], k
            close(session(eng).feed([(0, toks)])[0].cpu(), streams[k - 1], dtype)
    finally:
        eng.layers, eng.L = all_layers, L


PORTIONS = {"whole": [260], "tokens": [1] * 260, "twos": [2] * 130, "threes_and_sevens": [3, 7] * 26,
            "pages": [16, 15, 17, 1, 64, 63, 65, 19], "long_then_tokens": [200] + [1] * 60}


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("name", list(hm.CONFIGS))
@pytest.mark.parametrize("cut", list(PORTIONS))
def test_portions_and_decoding(name, cut, dtype):
    cfg, _, eng = model(name, dtype)
    toks = hm.tokens(cfg, 260, 1)
    want = want_logits(name, dtype, toks)
    ses = session(eng, 3, 272, bs=16 if cut == "pages" else None, perm_seed=4)
    at, rows = 0, []
    for n in PORTIONS[cut]:
        rows += ses.feed([(1, toks[at:at + n])])
        at += n
    close(logits(eng, torch.cat(rows)), want, dtype)


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("name", list(hm.CONFIGS))
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
        close(logits(eng, torch.cat(got[k])), want_logits(name, dtype, toks[k]), dtype)


@pytest.mark.parametrize("name", list(hm.CONFIGS))
def test_the_batch_changes_nothing_beyond_rounding(name):
    cfg, _, eng = model(name, "float32")
    a, b = hm.tokens(cfg, 120, 30), hm.tokens(cfg, 45, 31)
    alone = logits(eng, session(eng).feed([(0, a)])[0])
    ses = session(eng, 4)
    both = ses.feed([(2, b), (3, a)])[1]
    assert np.abs(logits(eng, both) - alone).max() < 1e-4 * np.abs(alone).max()


@pytest.mark.parametrize("name", list(hm.CONFIGS))
def test_greedy_generation_of_an_unequal_batch(name):
    """`generate`: chunked prompts, the decode loop and the sampler, token for token the oracle's greedy continuation."""
    from bitexact_llm_b200.decode import generate
    cfg, w64, eng = model(name, "float32")
    prompts = [hm.tokens(cfg, n, 40 + n) for n in (37, 1, 20)]
    ids = torch.zeros(3, 37, dtype=torch.long)
    for i, p in enumerate(prompts):
        ids[i, : len(p)] = torch.tensor(p)
    toks, shas = generate(eng, ids, 24, lens=torch.tensor([len(p) for p in prompts]), perm_seed=7)
    assert toks.tolist() == [oh.greedy(cfg, w64, p, 24) for p in prompts]
    assert all(len(s) == 24 for s in shas)


@pytest.mark.parametrize("dtype", DTYPES)
def test_long_decoding(dtype):
    from bitexact_llm_b200.decode import generate
    cfg, w64, eng = model("plain", dtype)
    prompt = hm.tokens(cfg, 5, 77)
    toks, _ = generate(eng, torch.tensor([prompt]), 500, hashes=False)
    seq = prompt + toks[0].tolist()
    want, _ = oh.forward(cfg, w64, seq[:-1])
    rows, at = [], 0
    ses = session(eng, 1, 512)
    for t in seq[:-1]:
        rows += ses.feed([(0, [t])])
    lg = logits(eng, torch.cat(rows))
    close(lg, want, dtype)
    assert (lg[4:].argmax(-1) == np.array(seq[5:])).mean() > 0.99      # the graph of kernels the loop ran, same tokens


@pytest.mark.parametrize("name", ["plain", "wide"])
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
    # capture itself runs nothing: the state is where the prompts left it
    got = torch.stack([dec.step().clone() for _ in range(12)], 1).cpu()
    assert torch.equal(got, want)


def test_sampler_is_keyed_by_seed_and_index():
    from bitexact_llm_b200.decode import generate
    cfg, _, eng = model("plain", "bfloat16")
    ids = torch.tensor([hm.tokens(cfg, 10, 3)] * 3)
    a, _ = generate(eng, ids, 8, 1, 1, seeds=[5, 6, 5], hashes=False)
    assert a[0].tolist() == a[2].tolist() != a[1].tolist()


def test_padding_rows_touch_nothing():
    cfg, _, eng = model("plain", "float32")
    toks = hm.tokens(cfg, 20, 9)
    want = logits(eng, session(eng).feed([(0, toks)])[0])
    ses = session(eng, 2, 64)
    ids = torch.tensor(toks + [0] * 5).cuda()
    pos = torch.tensor(list(range(20)) + [0] * 5).cuda()
    seq = torch.tensor([1] * 20 + [0] * 5).cuda()
    slot = torch.where(torch.arange(25).cuda() < 20, ses._slots(seq, pos), torch.full_like(pos, -1))
    ses.feed([(0, [3, 4])])
    before = [c[0].clone() for c in ses.kvs if c.dim() == 2]
    x = eng.forward(ses.kvs, ids, pos, slot, ses.bt, seq)
    close(logits(eng, x[:20]), want, "float32")
    assert all(torch.equal(a, c[0]) for a, c in zip(before, [c for c in ses.kvs if c.dim() == 2]))


# ---------------------------------------------------------------- commands

def test_trace_run_and_generate_commands(tmp_path):
    cfg = hm.settled(hm.CONFIGS["odd"])
    t = hm.weights(cfg, 3)
    w64 = hm.as_numpy(t)
    folder = hm.save_folder(tmp_path / "m", cfg, t)
    a, b = hm.tokens(cfg, 50, 1), hm.tokens(cfg, 20, 2)
    trace = [{"step": 0, "entries": [{"id": "a", "tokens": a[:30], "want": [0, 29]}], "end": []},
             {"step": 1, "entries": [{"id": "b", "tokens": b, "want": []}, {"id": "a", "tokens": a[30:31], "want": [0]}], "end": ["b"]},
             {"step": 2, "entries": [{"id": "a", "tokens": a[31:], "want": [18, 0]}], "end": ["a"]},
             {"step": 5, "entries": [{"id": "c", "tokens": b[:2], "want": [1]}], "end": ["c"]}]
    want_a, want_b = oh.forward(cfg, w64, a)[0], oh.forward(cfg, w64, b)[0]
    expect = {0: want_a[[0, 29]], 1: want_a[[30]], 2: want_a[[49, 31]], 5: want_b[[1]]}
    for dtype in DTYPES:
        out = tmp_path / dtype
        out.mkdir()
        r = subprocess.run([os.path.join(ROOT, "bin", "trace_run"), "--model", folder, "--dtype", dtype, "--out", str(out),
                            "--max-tokens", "70"], input="".join(json.dumps(s) + "\n" for s in trace), capture_output=True, text=True)
        assert r.returncode == 0, r.stderr
        assert [ln for ln in r.stdout.splitlines() if ln.startswith("done")] == ["done 0", "done 1", "done 2", "done 5"]
        for s, e in expect.items():
            close(np.fromfile(out / f"{s}.f32", "<f4").reshape(e.shape), e, dtype)
    r = subprocess.run([sys.executable, "-m", "bitexact_llm_b200", "generate", "--model", folder, "--dtype", "float32", "--max-new",
                        "6", "--prompt", ",".join(map(str, a[:9])), "--prompt", ",".join(map(str, b[:4]))],
                       cwd=ROOT, capture_output=True, text=True)
    assert r.returncode == 0, r.stderr
    assert [[int(v) for v in ln.split(",")] for ln in r.stdout.split()] == [oh.greedy(cfg, w64, a[:9], 6), oh.greedy(cfg, w64, b[:4], 6)]
