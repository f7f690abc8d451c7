"""The Veredra design, host side: configuration reading, the registry, the unrolled loop, the tables of a prompt portion, the
argument checks of the library, and the oracle's mechanisms against scalar loops."""

import ctypes
import json
import math

import numpy as np
import pytest
import torch

import hybrid_models as hm
import veredra_models as vm
from oracle import veredra as ov


def test_config_reader_takes_every_size_and_branch():
    from bitexact_llm_b200.hybrid import veredra
    from bitexact_llm_b200.hybrid.spec import AttentionSpec, GatedSpec, GLASpec, Mamba2Spec
    s = veredra.read_config(vm.CONFIGS["looped"])
    assert (s.vocab, s.width, s.eps, s.streams, s.logit_scale, s.logit_softcap) == (130, 72, 1e-3, 3, 0.5, 4.0)
    assert s.runs == (0, 1, 2, 1, 2, 3)
    assert s.layers[0].mixer == AttentionSpec(heads=6, kv_heads=2, dim=24, vdim=40, rot_dims=16, rot_base=10000.0,
                                              scale=24 ** -0.5, window=19, eps=1e-3)
    assert s.layers[1].mixer == GLASpec(heads=3, dim=16, vdim=24, tau=8.0, eps=1e-3) and s.layers[1].ff == GatedSpec(88)
    assert s.layers[2].mixer == Mamba2Spec(heads=6, vdim=16, state=24, groups=3, taps=4, norm_groups=2, eps=1e-3)
    assert s.layers[2].ff is None
    s = veredra.read_config(vm.CONFIGS["odd"])
    assert s.runs == (0, 1, 2) and s.layers[1].mixer.scale == 0.4 and s.layers[1].mixer.rot_base == 500.0
    assert veredra.read_config(vm.CONFIGS["wide"]).runs == (0, 1, 2, 2, 2, 3)

    def changed(f):
        c = json.loads(json.dumps(vm.CONFIGS["looped"]))
        f(c)
        return c
    for f in (lambda c: c["layers"][0].update(type="other"), lambda c: c["layers"][0]["mlp"].update(kind="moe"),
              lambda c: c["loop"].update(stop=9)):
        with pytest.raises(ValueError):
            veredra.read_config(changed(f))
    assert veredra.read_config(changed(lambda c: c["layers"][0]["mixer"].pop("mask"))).layers[0].mixer.window == 0
    assert veredra.read_config(changed(lambda c: c["layers"][0]["mixer"].pop("rot"))).layers[0].mixer.rot_dims == 0
    assert veredra.read_config(changed(lambda c: c["loop"].update(times=0))).runs == (0, 3)


def test_weights_are_grouped_by_sublayer():
    from bitexact_llm_b200.hybrid import veredra
    cfg = vm.CONFIGS["looped"]
    w = veredra.read_weights(veredra.read_config(cfg), vm.weights(cfg))
    assert set(w["layers"][1]["mixer"]) == {"q", "k", "v", "g", "o", "a1", "a2", "a2.b", "norm"}
    assert set(w["layers"][0]["ff"]) == {"gate", "up", "down"} and w["layers"][0]["hc2"]["mix"].shape == (3, 3)
    assert w["layers"][2]["norm2"] is None and w["layers"][2]["hc2"] is None
    one = json.loads(json.dumps(vm.CONFIGS["one"]))
    t = {k: v for k, v in vm.weights(one).items() if ".hc" not in k}
    assert veredra.read_weights(veredra.read_config(one), t)["layers"][0]["hc1"]["mix"].item() == 1.0


def test_registry_and_dtypes(tmp_path):
    from bitexact_llm_b200 import registry
    assert registry.family(vm.CONFIGS["one"]) is registry.VeredraFamily
    folder = hm.save_folder(tmp_path / "m", vm.CONFIGS["one"], {})
    with pytest.raises(registry.UnsupportedDtype):
        registry.load(folder, dtype="exact")


def test_tables_of_a_portion():
    from bitexact_llm_b200.hybrid.layers import Tiles
    t = Tiles.of([(4, 0, 130, 500), (2, 130, 1, 1), (0, 131, 64, 64)], {16, 50})
    assert t.runs.tolist() == [[0, 130, 0], [130, 1, 3], [131, 64, 4]]
    assert t.chunks.tolist() == [[0, 64], [64, 64], [128, 2], [130, 1], [131, 64]]
    assert t.attention[50].tolist() == [[4, 0, 50], [4, 50, 50], [4, 100, 30], [2, 130, 1], [0, 131, 50], [0, 181, 14]]
    assert t.segments.tolist() == t.runs.tolist() and t.spans.tolist() == [[0, 0, 1], [130, 1, 1], [131, 2, 1]]
    long = Tiles.of([(0, 0, 600, 600), (1, 600, 3, 3)], ())
    assert long.segments.tolist() == [[0, 256, 0], [256, 256, 4], [512, 88, 8], [600, 3, 10]]
    assert long.spans.tolist() == [[0, 0, 3], [600, 3, 1]]
    assert Tiles.of([(0, 0, 5000, 5000)], ()).segments[1].tolist() == [512, 512, 8]
    assert len(t.attention[16]) == 9 + 1 + 4 and Tiles.of([(0, 0, 2, 2)], ()).attention == {}


def test_library_checks_its_arguments():
    from bitexact_llm_b200 import _native as nv
    from bitexact_llm_b200 import build
    build.build(target="float")
    lib = nv.float_lib()
    sizes = {nv.StreamsStep: 112, nv.GqaRows: 120, nv.Conv: 72, nv.RecurrenceRows: 160, nv.ChunkTable: 48, nv.GateRows: 152}
    assert all(ctypes.sizeof(c) == n for c, n in sizes.items())                  # as asserted in float_capi.cu
    ref = ctypes.byref
    p = nv.StreamsStep(x=16, streams=9, D=8, sum=16)
    assert lib.bxf_streams(0, ref(p), 1, None) == nv.BX_EARG                     # too many streams
    p = nv.StreamsStep(x=16, streams=2, D=8, y=16, sum=16)
    assert lib.bxf_streams(0, ref(p), 1, None) == nv.BX_EARG                     # an output without its weights
    g = nv.GqaRows(y=16, ldy=64, heads=3, kv_heads=2, dim=8, vdim=8, slot=16, q=16, ldq=8, cache=16, ldc=16, voff=8, page=16)
    assert lib.bxf_gqa_prepare(0, ref(g), 1, None) == nv.BX_EARG                 # unequal groups
    r = nv.RecurrenceRows(kind=0, heads=2, groups=1, K=8, V=8, rank=1, y=16, side=16, a2=16, a2_b=16, state=16, flags=16, seq=16,
                          out=16, ldo=16)
    assert lib.bxf_recurrence(0, ref(r), 1, None) == nv.BX_EARG                  # channel decays have a key per head
    r.groups, r.K = 2, 513
    assert lib.bxf_recurrence(0, ref(r), 1, None) == nv.BX_ELIMIT
    t = nv.ChunkTable(runs=16, chunks=16, nruns=1, nchunks=1)
    assert lib.bxf_recurrence_chunks(0, ref(r), ref(t), 16, 1 << 20, 1, None) == nv.BX_ELIMIT
    r.K, t.nsegments = 8, 2
    assert lib.bxf_recurrence_chunks(0, ref(r), ref(t), 16, 1 << 20, 1, None) == nv.BX_EARG             # segments without a table
    assert [lib.bxf_recurrence_chunk_rows(*a) for a in ((0, 128, 64), (0, 12, 64), (0, 16, 12), (0, 264, 8), (1, 128, 64))] == [64, 0, 0, 0, 0]
    epi = nv.Epilogue(kind=4, out=16)
    assert lib.bxf_linear(0, 16, 8, 0, 16, 8, 0, 1, 1, 7, 8, None, ref(epi), 0, None) == nv.BX_EARG    # pairs
    gate = nv.GateRows(o=16, z=16, ldo=8, ldz=8, w=16, out=16, ldout=8, n=8, parts=3, wn=8)
    assert lib.bxf_gated_norm(0, ref(gate), 1, None) == nv.BX_EARG               # unequal parts


# ---- the oracle's mechanisms against scalar loops ----

def test_oracle_attention_by_hand():
    rng = np.random.RandomState(1)
    cfg = {"heads": 4, "kv_heads": 2, "dim": 6, "vdim": 3, "rot": {"base": 50.0, "dims": 4}, "scale": 0.7, "mask": {"size": 3}}
    T, D, eps = 6, 5, 1e-2
    w = {"q": rng.randn(24, D), "k": rng.randn(12, D), "v": rng.randn(6, D), "q.b": rng.randn(24), "k.b": rng.randn(12),
         "v.b": rng.randn(6), "q.norm": rng.randn(24), "k.norm": rng.randn(12), "sink": rng.randn(4), "o": rng.randn(D, 12)}
    h = rng.randn(T, D)
    y = ov.attention(h, w, cfg, eps)

    def rot(v, p):
        out = list(v)
        for i in range(2):
            a = p * 50.0 ** (-2 * i / 4)
            out[i], out[i + 2] = v[i] * math.cos(a) - v[i + 2] * math.sin(a), v[i + 2] * math.cos(a) + v[i] * math.sin(a)
        return np.array(out)

    def normed(n, j):
        v = w[n] @ h[j] + w[n + ".b"]
        return v / math.sqrt((v ** 2).mean() + eps) * w[n + ".norm"]
    for i in range(T):
        heads = []
        for a in range(4):
            g = a // 2
            js = [j for j in range(T) if 0 <= i - j < 3]
            q = rot(normed("q", i)[6 * a:6 * a + 6], i)
            e = [math.exp(0.7 * (q @ rot(normed("k", j)[6 * g:6 * g + 6], j))) for j in js]
            den = sum(e) + math.exp(w["sink"][a])
            heads.append(sum(x * (w["v"] @ h[j] + w["v.b"])[3 * g:3 * g + 3] for x, j in zip(e, js)) / den)
        assert np.allclose(y[i], w["o"] @ np.concatenate(heads))


def test_oracle_mamba2_by_hand():
    rng = np.random.RandomState(2)
    cfg = {"heads": 4, "vdim": 3, "state": 2, "groups": 2, "conv": 3, "norm_groups": 2}
    T, D, eps, inner, ch = 5, 4, 1e-2, 12, 20
    w = {"in": rng.randn(2 * inner + 8 + 4, D), "conv": rng.randn(ch, 3), "conv.b": rng.randn(ch), "dt_bias": rng.randn(4),
         "A_log": rng.randn(4), "D": rng.randn(4), "norm": rng.randn(inner), "o": rng.randn(D, inner)}
    h = rng.randn(T, D)
    out, S_end = ov.mamba2(h, w, cfg, eps)
    u = [w["in"] @ h[t] for t in range(T)]
    silu = lambda v: v / (1 + math.exp(-v))
    S = np.zeros((4, 2, 3))
    for t in range(T):
        c = [silu(w["conv.b"][k] + sum(w["conv"][k, j] * u[t - 2 + j][inner + k] for j in range(3) if t - 2 + j >= 0)) for k in range(ch)]
        y = []
        for a in range(4):
            g = a // 2
            dt = math.log(1 + math.exp(u[t][2 * inner + 8 + a] + w["dt_bias"][a]))
            x, B, C = np.array(c[3 * a:3 * a + 3]), np.array(c[12 + 2 * g:14 + 2 * g]), np.array(c[16 + 2 * g:18 + 2 * g])
            S[a] = math.exp(-math.exp(w["A_log"][a]) * dt) * S[a] + dt * np.outer(B, x)
            y += list(S[a].T @ C + w["D"][a] * x)
        y = np.array([v * silu(u[t][k]) for k, v in enumerate(y)])
        y = np.concatenate([y[k:k + 6] / math.sqrt((y[k:k + 6] ** 2).mean() + eps) for k in (0, 6)]) * w["norm"]
        assert np.allclose(out[t], w["o"] @ y)
    assert np.allclose(S, S_end)


def test_oracle_gla_by_hand():
    rng = np.random.RandomState(3)
    cfg = {"heads": 2, "dim": 3, "vdim": 4, "tau": 5.0}
    T, D, eps = 4, 5, 1e-2
    w = {"q": rng.randn(6, D), "k": rng.randn(6, D), "v": rng.randn(8, D), "g": rng.randn(8, D), "a1": rng.randn(2, D),
         "a2": rng.randn(6, 2), "a2.b": rng.randn(6), "norm": rng.randn(4), "o": rng.randn(D, 8)}
    h = rng.randn(T, D)
    out, S_end = ov.gla(h, w, cfg, eps)
    S = np.zeros((2, 3, 4))
    for t in range(T):
        z = w["a2"] @ (w["a1"] @ h[t]) + w["a2.b"]
        o = []
        for a in range(2):
            decay = (1 / (1 + np.exp(-z[3 * a:3 * a + 3]))) ** (1 / 5.0)
            S[a] = decay[:, None] * S[a] + np.outer((w["k"] @ h[t])[3 * a:3 * a + 3], (w["v"] @ h[t])[4 * a:4 * a + 4])
            v = S[a].T @ ((w["q"] @ h[t])[3 * a:3 * a + 3] * 3 ** -0.5)
            o += list(v / math.sqrt((v ** 2).mean() + eps) * w["norm"])
        g = w["g"] @ h[t]
        assert np.allclose(out[t], w["o"] @ (np.array(o) * g / (1 + np.exp(-g))))
    assert np.allclose(S, S_end)


def test_oracle_streams_and_feed_forward_by_hand():
    rng = np.random.RandomState(4)
    hc = {"in": rng.randn(3), "out": rng.randn(3), "mix": rng.randn(3, 3)}
    xs, y = rng.randn(3, 2, 4), rng.randn(2, 4)
    u, new = ov.hyper_in(xs, hc), ov.hyper_out(xs, hc, y)
    for t in range(2):
        for d in range(4):
            assert np.isclose(u[t, d], sum(hc["in"][s] * xs[s, t, d] for s in range(3)))
            for to in range(3):
                assert np.isclose(new[to, t, d], sum(hc["mix"][s, to] * xs[s, t, d] for s in range(3)) + hc["out"][to] * y[t, d])
    z = np.array([-2.0, 0.0, 1.5])
    want = [0.5 * v * (1 + math.tanh(math.sqrt(2 / math.pi) * (v + 0.044715 * v ** 3))) for v in z]
    assert np.allclose(ov.gelu_tanh(z), want)
    w = {"gate": rng.randn(5, 4), "up": rng.randn(5, 4), "down": rng.randn(4, 5)}
    h = rng.randn(1, 4)
    assert np.allclose(ov.gated_ff(h, w)[0], w["down"] @ (ov.gelu_tanh(w["gate"] @ h[0]) * (w["up"] @ h[0])))


def test_oracle_loop_runs_layers_again_with_states_of_their_own():
    assert ov.layer_order(vm.CONFIGS["looped"]) == [0, 1, 2, 1, 2, 3] and ov.layer_order(vm.CONFIGS["odd"]) == [0, 1, 2]
    cfg = json.loads(json.dumps(vm.CONFIGS["wide"]))
    w, toks = hm.as_numpy(vm.weights(cfg)), hm.tokens(cfg, 6, 0)
    lg, after = ov.forward(cfg, w, toks)
    cfg["layers"][2:3] = [cfg["layers"][2]] * 3                       # the loop written out, weights repeated
    cfg["loop"] = None
    flat = {}
    for k, v in w.items():
        if k[0] == "l" and k[1].isdigit():
            i, rest = int(k[1:k.index(".")]), k[k.index("."):]
            for j in ([i] if i < 2 else [2, 3, 4] if i == 2 else [5]):
                flat[f"l{j}{rest}"] = v
        else:
            flat[k] = v
    lg2, after2 = ov.forward(cfg, flat, toks)
    assert np.array_equal(lg, lg2) and np.array_equal(after, after2) and abs(lg).max() < cfg["logit_softcap"]
