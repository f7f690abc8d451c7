"""Hybrid float models, host side: weight files, configuration reading, the registry, the page pool of a session, the
command lines' argument handling, the C ABI of the float library, and the oracle against hand-written loops."""

import ctypes
import json
import math
import os
import re
import subprocess
import sys

import numpy as np
import pytest
import torch

import hybrid_models as hm
from oracle import hybrid as oh

ROOT = os.path.dirname(os.path.dirname(os.path.abspath(__file__)))


def test_safetensors_round_trip_and_bad_files(tmp_path):
    from bitexact_llm_b200.weights import load_safetensors, save_safetensors
    t = {"a": torch.randn(3, 5).to(torch.bfloat16), "b": torch.arange(7, dtype=torch.int32), "c": torch.tensor([1.5]),
         "empty": torch.empty(0, 4)}
    p = str(tmp_path / "m.safetensors")
    save_safetensors(t, p)
    u = load_safetensors(p)
    assert list(u) == list(t) and all(torch.equal(u[k], t[k]) and u[k].dtype == t[k].dtype for k in t)
    raw = open(p, "rb").read()
    open(p, "wb").write(raw[:-1])                                     # the last tensor's data is cut off
    with pytest.raises(ValueError):
        load_safetensors(p)
    open(p, "wb").write(raw[:5])
    with pytest.raises(ValueError):
        load_safetensors(p)


def test_config_reader_takes_every_size_and_branch():
    from bitexact_llm_b200.hybrid import fedatar
    from bitexact_llm_b200.hybrid.spec import DenseSpec, ExpertsSpec, LatentAttentionSpec, MinGRUSpec
    s = fedatar.read_config(hm.CONFIGS["odd"])
    assert (s.vocab, s.width, s.eps) == (77, 52, 1e-5)
    assert s.layers[0].mixer == MinGRUSpec(90)
    assert s.layers[0].ff == ExpertsSpec(experts=7, top=3, ff=33, shared_ff=19)
    assert s.layers[1].mixer == LatentAttentionSpec(heads=5, dim=10, rot_dim=6, vdim=13, q_rank=27, kv_rank=50, rot_base=1e6,
                                                    scale=0.31, window=33, eps=1e-5)
    assert s.layers[2].mixer.window == 0 and s.layers[2].ff is None
    p = fedatar.read_config(hm.CONFIGS["plain"])
    assert p.layers[0].ff.shared_ff == 0 and p.layers[1].ff == DenseSpec(104) and p.layers[2].ff is None
    bad = json.loads(json.dumps(hm.CONFIGS["plain"]))
    bad["layers"][0]["type"] = "other"
    with pytest.raises(ValueError):
        fedatar.read_config(bad)
    bad = json.loads(json.dumps(hm.CONFIGS["plain"]))
    bad["layers"][0]["mixer"]["rot"]["dims"] = 4
    with pytest.raises(ValueError):
        fedatar.read_config(bad)


def test_registry_chooses_the_family_by_config(tmp_path):
    from bitexact_llm_b200 import registry
    assert registry.family(hm.CONFIGS["plain"]) is registry.FedatarFamily
    assert registry.family({"architectures": ["LlamaForCausalLM"]}) is registry.LlamaFamily
    with pytest.raises(ValueError):
        registry.family({"architecture": "Nothing"})
    folder = hm.save_folder(tmp_path / "m", hm.CONFIGS["plain"], {})
    with pytest.raises(registry.UnsupportedDtype):
        registry.load(folder, dtype="int8")


def test_trace_run_refuses_32_bit_for_an_integer_model(tmp_path):
    (tmp_path / "config.json").write_text(json.dumps({"architectures": ["LlamaForCausalLM"]}))
    r = subprocess.run([os.path.join(ROOT, "bin", "trace_run"), "--model", str(tmp_path), "--dtype", "float32", "--out",
                        str(tmp_path), "--max-tokens", "8"], stdin=subprocess.DEVNULL, capture_output=True)
    assert r.returncode == 3


class CountingEngine:
    """The host side of an engine: residual row = (token, position, slot), no device work."""
    dev, D, L, tiles_from = torch.device("cpu"), 3, 1, 0

    def __init__(self):
        self.calls, self.tables = [], []

    def new_cache(self, n_seqs, n_blocks, bs):
        return [torch.full((n_blocks * bs,), -1, dtype=torch.long)]

    def tile_table(self, runs, bs):
        self.tables.append(list(runs))

    def forward(self, caches, ids, pos, slot, bt, rmap, tiles=None):
        self.calls.append(ids.shape[0])
        caches[0][slot] = ids
        return torch.stack([ids, pos, slot], 1).float()


def test_session_pool_takes_pages_on_demand_and_reuses_them():
    from bitexact_llm_b200.decode import Session
    eng = CountingEngine()
    ses = Session(eng, 3, 40, bs=4, pages=12)
    a, b = ses.feed([(0, list(range(10))), (2, [50, 51])])
    assert a[:, 1].tolist() == list(range(10)) and b[:, 1].tolist() == [0, 1] and eng.calls == [12]
    assert len(ses.held[0]) == 3 and len(ses.held[2]) == 1 and len(ses.free) == 8
    assert not set(ses.held[0]) & set(ses.held[2]) and 0 not in ses.held[0]
    (c,) = ses.feed([(0, [7])])
    assert c[0, 1] == 10 and c[0, 2] == ses.held[0][2] * 4 + 2         # position 10: third page, third token
    with pytest.raises(MemoryError):
        ses.feed([(1, list(range(36)))])
    with pytest.raises(ValueError):
        ses.feed([(1, list(range(41)))])
    held = list(ses.held[0])
    ses.release(0)
    assert ses.lens.tolist() == [0, 0, 2] and len(ses.free) == 11
    ses.feed([(1, list(range(8)))])
    assert set(ses.held[1]) <= set(held) and ses.lens.tolist() == [0, 8, 2]


def test_session_feed_cuts_long_portions_into_forward_calls():
    from bitexact_llm_b200.decode import Session
    eng = CountingEngine()
    ses = Session(eng, 2, 64, bs=8)
    a, b = ses.feed([(1, list(range(23))), (0, list(range(100, 105)))], chunk_rows=10)
    assert eng.calls == [10, 10, 8] and a[:, 0].tolist() == list(range(23)) and b[:, 0].tolist() == list(range(100, 105))
    assert eng.tables == [[(1, 0, 10, 10)], [(1, 0, 10, 20)], [(1, 0, 3, 23), (0, 3, 5, 5)]]
    assert ses.lens.tolist() == [5, 23]


def test_float_library_exports_every_declared_symbol_and_checks_arguments():
    from bitexact_llm_b200 import _native as nv
    from bitexact_llm_b200 import build
    h = ctypes.CDLL(build.build(target="float"))
    with open(os.path.join(ROOT, "include", "bitexact_float.h")) as f:
        names = sorted(set(re.findall(r"\b(bxf_[a-z0-9_]+)\s*\(", f.read())))
    assert all(hasattr(h, n) for n in names) and nv.exported_symbols(float_models=True) == names
    lib = nv.float_lib()
    epi = nv.Epilogue(kind=0, n_main=8, out=16)
    assert lib.bxf_linear(0, None, 8, 0, 16, 8, 0, 1, 1, 8, 8, None, ctypes.byref(epi), 0, None) == nv.BX_EARG
    assert lib.bxf_linear(0, 16, 12, 0, 16, 8, 0, 1, 1, 8, 8, None, ctypes.byref(epi), 0, None) == nv.BX_EARG   # ld % 8
    assert lib.bxf_linear(0, 16, 8, 0, 16, 8, 0, 1, 1, 9, 8, None, ctypes.byref(epi), 0, None) == nv.BX_EARG    # no side
    assert lib.bxf_route(16, 8, 8, 9, 16, 16, 16, 16, 1, None) == nv.BX_ELIMIT
    g = nv.Gru()
    assert lib.bxf_gru_linear(0, 16, 8, 16, 8, 4, 8, 8, ctypes.byref(g), None) == nv.BX_EARG
    assert lib.bxf_latent_attention_tile(12) == 10 and lib.bxf_latent_attention_tile(200) == 1
    assert ctypes.sizeof(nv.Epilogue) == 136 and ctypes.sizeof(nv.Gru) == 56      # as asserted in float_capi.cu


def test_sources_of_the_targets_are_separate():
    from bitexact_llm_b200 import build
    names = lambda t: {os.path.basename(f) for f in build.sources(t)}
    assert "fl_gemm.cuh" in names("float") and "fl_gemm.cuh" not in names("integer")
    assert "capi.cu" in names("integer") and "capi.cu" not in names("float") and "bx_ptx.cuh" in names("float")


# ---- the oracle's mechanisms against scalar loops ----

def test_oracle_mingru_by_hand():
    rng = np.random.RandomState(0)
    T, D, W = 5, 3, 4
    h = rng.randn(T, D)
    wz, wx, wg, wo, bz, bx = rng.randn(W, D), rng.randn(W, D), rng.randn(W, D), rng.randn(D, W), rng.randn(W), rng.randn(W)
    y, s_end = oh.mingru(h, wz, bz, wx, bx, wg, wo)
    sig = lambda v: 1.0 / (1.0 + math.exp(-v))
    s = [0.0] * W
    for t in range(T):
        o = []
        for j in range(W):
            z, u, g = (sum(w[j, d] * h[t, d] for d in range(D)) for w in (wz, wx, wg))
            z, u = sig(z + bz[j]), u + bx[j]
            s[j] = (1 - z) * s[j] + z * (u + 0.5 if u >= 0 else sig(u))
            o.append(s[j] * g * sig(g))
        assert np.allclose(y[t], wo @ np.array(o))
    assert np.allclose(s, s_end)
    y1, s1 = oh.mingru(h[:2], wz, bz, wx, bx, wg, wo)
    y2, s2 = oh.mingru(h[2:], wz, bz, wx, bx, wg, wo, state=s1)
    assert np.allclose(np.concatenate([y1, y2]), y) and np.allclose(s2, s_end)


def test_oracle_attention_by_hand():
    rng = np.random.RandomState(1)
    cfg = {"heads": 2, "dim": 3, "rot_dim": 4, "vdim": 2, "kv_rank": 5, "rot": {"base": 50.0, "dims": 4}, "scale": 0.7,
           "mask": {"size": 3}}
    T, D, Q, eps = 6, 4, 3, 1e-4
    w = {"dq": rng.randn(Q, D), "dq.norm": rng.randn(Q), "uq": rng.randn(14, Q), "dkv": rng.randn(9, D),
         "dkv.norm": rng.randn(5), "uk": rng.randn(6, 5), "uv": rng.randn(4, 5), "sink": rng.randn(2), "g": rng.randn(2, D),
         "o": rng.randn(D, 4)}
    h = rng.randn(T, D)
    y = oh.latent_attention(h, w, cfg, eps)

    def rot(v, p):
        out = list(v)
        for i in range(2):
            a = p * 50.0 ** (-2 * i / 4)
            out[2 * i], out[2 * i + 1] = v[2 * i] * math.cos(a) - v[2 * i + 1] * math.sin(a), \
                v[2 * i + 1] * math.cos(a) + v[2 * i] * math.sin(a)
        return np.array(out)

    def rms(v, g):
        return v / math.sqrt((v ** 2).mean() + eps) * g
    lat = [rms((w["dkv"] @ h[j])[:5], w["dkv.norm"]) for j in range(T)]
    kr = [rot((w["dkv"] @ h[j])[5:], j) for j in range(T)]
    for i in range(T):
        q = w["uq"] @ rms(w["dq"] @ h[i], w["dq.norm"])
        heads = []
        for k in range(2):
            qn, qr = q[7 * k:7 * k + 3], rot(q[7 * k + 3:7 * k + 7], i)
            js = [j for j in range(T) if 0 <= i - j < 3]
            e = [math.exp(0.7 * (qn @ (w["uk"][3 * k:3 * k + 3] @ lat[j]) + qr @ kr[j])) for j in js]
            den = sum(e) + math.exp(w["sink"][k])
            o = sum(a * (w["uv"][2 * k:2 * k + 2] @ lat[j]) for a, j in zip(e, js)) / den
            heads.append(o / (1 + math.exp(-(w["g"][k] @ h[i]))))
        assert np.allclose(y[i], w["o"] @ np.concatenate(heads))


def test_oracle_feed_forwards_by_hand():
    z = np.array([-3.0, -1e-3, 0.0, 1e-3, 2.0])
    sp = lambda v: math.log(1 + math.exp(v))
    want = [sp(0.3) * v * v + v / 2 if v > 0 else (0.5 + sp(-0.2)) * (math.exp(v) - 1 - v) + v / 2 for v in z]
    assert np.allclose(oh.xielu(z, 0.3, -0.2), want)
    assert np.array_equal(oh.relu2(np.array([-2.0, 3.0])), [0.0, 9.0])
    idx, wt = oh.route(np.eye(3), np.array([[1.0, 0, 0], [0, 2.0, 0], [0, 0, 3.0], [1.0, 0, 0]]), np.array([0, 0.5, 0, 0.25]), 2)
    assert idx.tolist() == [[3, 0], [1, 3], [2, 1]]
    assert np.allclose(wt[0], [math.exp(1.25) / (math.exp(1.25) + math.e), math.e / (math.exp(1.25) + math.e)])


def test_module_help_lists_the_commands():
    r = subprocess.run([sys.executable, "-m", "bitexact_llm_b200"], cwd=ROOT, capture_output=True, text=True)
    assert r.returncode == 2 and "generate" in r.stderr and "trace" in r.stderr
