"""Small random models of the hybrid float designs for the tests: configurations of several shapes (sizes that are not
multiples of 8 or 64, layers without a feed-forward, experts with and without a shared one, different windows, orders
and constants) and their weights, plus the folder form the registry loads."""

import json
import os

import torch

from bitexact_llm_b200.weights import save_safetensors


def gru(width, mlp):
    return {"type": "mingru", "mixer": {"width": width}, "mlp": mlp}


def attn(heads, dim, rot, vdim, q_rank, kv_rank, window, mlp, base=10000.0, scale=None):
    m = {"heads": heads, "dim": dim, "rot_dim": rot, "vdim": vdim, "q_rank": q_rank, "kv_rank": kv_rank,
         "rot": {"base": base, "dims": rot}, "scale": scale or (dim + rot) ** -0.5}
    if window:
        m["mask"] = {"size": window}
    return {"type": "latent_attention", "mixer": m, "mlp": mlp}


def dense(ff):
    return {"kind": "dense", "ff": ff}


def moe(experts, top, ff, shared):
    f = {"kind": "moe", "router": {"experts": experts, "top": top}, "expert": {"ff": ff}}
    if shared:
        f["shared"] = {"ff": shared}
    return f


def config(vocab, width, layers, eps=1e-5):
    return {"architecture": "Fedatar", "vocab": vocab, "width": width, "norm": {"eps": eps}, "layers": layers}


CONFIGS = {
    # attention first, a layer without a feed-forward, one expert chosen
    "plain": config(130, 72, [attn(3, 24, 8, 40, 56, 48, 19, moe(5, 1, 48, 0)), gru(88, dense(104)), gru(40, None),
                              attn(2, 16, 4, 24, 32, 80, 70, dense(64), base=500.0)], eps=1e-3),
    # nothing divides anything
    "odd": config(77, 52, [gru(90, moe(7, 3, 33, 19)), attn(5, 10, 6, 13, 27, 50, 33, moe(3, 2, 21, 45), base=1e6, scale=0.31),
                           attn(1, 9, 2, 7, 11, 23, 0, None)]),
    # wider: several tiles and key blocks per tile, heads that do not divide 128
    "wide": config(300, 256, [gru(384, moe(16, 4, 96, 160)), attn(12, 48, 32, 48, 96, 128, 130, moe(9, 2, 72, 64)),
                              gru(320, dense(384)), attn(16, 64, 16, 32, 128, 272, 65, dense(256), base=2e5)]),
}


def settled(cfg):
    """The same model with every expert chosen: no choice that rounding could turn (the bf16 runs of whole models)."""
    c = json.loads(json.dumps(cfg))
    for ly in c["layers"]:
        if ly["mlp"] and ly["mlp"]["kind"] == "moe":
            ly["mlp"]["router"]["top"] = ly["mlp"]["router"]["experts"]
    return c


def weights(cfg, seed=0):
    """bf16 tensors under the design's names; gains such that every mechanism moves the logits."""
    g = torch.Generator().manual_seed(seed)
    D, t = cfg["width"], {}

    def mat(name, n, k, gain=1.0):
        t[name] = torch.randn(n, k, generator=g) * (gain / k ** 0.5)

    def vec(name, n, mean=0.0, std=0.3):
        t[name] = mean + std * torch.randn(n, generator=g)

    def norm(name, n=D):
        vec(name, n, 1.0, 0.2)
        vec(name + ".b", n)

    t["embed"] = torch.randn(cfg["vocab"], D, generator=g)
    mat("head", cfg["vocab"], D)
    norm("final.norm")
    for i, ly in enumerate(cfg["layers"]):
        p, m = f"l{i}.", ly["mixer"]
        norm(p + "norm1")
        if ly["type"] == "mingru":
            w = m["width"]
            for n in ("z", "x", "g"):
                mat(p + "mix." + n, w, D, 1.5)
            vec(p + "mix.z.b", w, -1.5, 1.0)
            vec(p + "mix.x.b", w)
            mat(p + "mix.o", D, w, 1.5)
        else:
            H, dn, dr, dv, R, Q = (m[k] for k in ("heads", "dim", "rot_dim", "vdim", "kv_rank", "q_rank"))
            mat(p + "mix.dq", Q, D)
            vec(p + "mix.dq.norm", Q, 1.0, 0.2)
            mat(p + "mix.uq", H * (dn + dr), Q, 2.0)
            mat(p + "mix.dkv", R + dr, D)
            vec(p + "mix.dkv.norm", R, 1.0, 0.2)
            mat(p + "mix.uk", H * dn, R, 2.0)
            mat(p + "mix.uv", H * dv, R)
            vec(p + "mix.sink", H, 0.5, 1.0)
            mat(p + "mix.g", H, D)
            mat(p + "mix.o", D, H * dv, 2.0)
        f = ly["mlp"]
        if f is None:
            continue
        norm(p + "norm2")
        if f["kind"] == "dense":
            mat(p + "mlp.up", f["ff"], D)
            mat(p + "mlp.down", D, f["ff"])
            t[p + "mlp.act"] = torch.tensor([0.4, -0.7]) + 0.1 * i
        else:
            E = f["router"]["experts"]
            for e in range(E):
                mat(p + f"mlp.e{e}.up", f["expert"]["ff"], D)
                mat(p + f"mlp.e{e}.down", D, f["expert"]["ff"])
            mat(p + "mlp.router", E, D, 2.0)
            vec(p + "mlp.router.b", E)
            if f.get("shared"):
                mat(p + "mlp.shared.up", f["shared"]["ff"], D)
                mat(p + "mlp.shared.down", D, f["shared"]["ff"])
    return {k: v.to(torch.bfloat16) for k, v in t.items()}


def as_numpy(t):
    return {k: v.double().numpy() for k, v in t.items()}


def save_folder(path, cfg, tensors):
    os.makedirs(path, exist_ok=True)
    with open(os.path.join(path, "config.json"), "w") as f:
        json.dump(cfg, f)
    save_safetensors(tensors, os.path.join(path, "model.safetensors"))
    return str(path)


def tokens(cfg, n, seed):
    g = torch.Generator().manual_seed(seed)
    return torch.randint(0, cfg["vocab"], (n,), generator=g).tolist()
