"""Small random Veredra models for the tests: sizes that are not multiples of 8 or 64, one and several streams, one and
several key/value heads, groups and convolution taps, loops and none, and their weights."""

import torch


def attn(heads, kv_heads, dim, vdim, rot, window, ff, base=10000.0, scale=None):
    return {"type": "attention", "mlp": ff and {"kind": "dense", "ff": ff},
            "mixer": {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "rot": {"base": base, "dims": rot},
                      "scale": scale or dim ** -0.5, "mask": {"size": window}}}


def mamba(heads, vdim, state, groups, taps, norm_groups, ff):
    return {"type": "mamba2", "mlp": ff and {"kind": "dense", "ff": ff},
            "mixer": {"heads": heads, "vdim": vdim, "state": state, "groups": groups, "conv": taps, "norm_groups": norm_groups}}


def gla(heads, dim, vdim, tau, ff, rank):
    return {"type": "gla", "mlp": ff and {"kind": "dense", "ff": ff}, "rank": rank,
            "mixer": {"heads": heads, "dim": dim, "vdim": vdim, "tau": tau}}


def config(vocab, width, streams, layers, loop=None, eps=1e-5, scale=1.0, cap=30.0):
    return {"architecture": "Veredra", "vocab": vocab, "width": width, "streams": streams, "layers": layers, "loop": loop,
            "norm": {"eps": eps}, "logit_scale": scale, "logit_softcap": cap}


CONFIGS = {
    "looped": config(130, 72, 3, [attn(6, 2, 24, 40, 16, 19, 104), gla(3, 16, 24, 8.0, 88, 8), mamba(6, 16, 24, 3, 4, 2, None),
                                  gla(2, 40, 16, 16.0, None, 5)], {"start": 1, "stop": 3, "times": 2}, eps=1e-3, scale=0.5, cap=4.0),
    # nothing divides anything
    "odd": config(77, 52, 4, [mamba(3, 7, 9, 1, 2, 3, 45), attn(5, 5, 10, 13, 6, 33, 61, base=500.0, scale=0.4),
                              gla(2, 11, 9, 1.0, 33, 3)], scale=3.0, cap=9.0),
    # one of everything, also one run and one tap
    "one": config(40, 40, 1, [gla(1, 8, 8, 4.0, 48, 1), mamba(1, 16, 8, 1, 1, 1, 24), attn(1, 1, 8, 8, 8, 1, None)],
                  {"start": 0, "stop": 2, "times": 1}, eps=1e-2),
    # wider: several tiles, key blocks and value slices
    "wide": config(300, 256, 2, [attn(16, 2, 64, 80, 32, 130, 384, base=1e6), mamba(8, 64, 128, 2, 4, 1, 320),
                                 gla(4, 128, 96, 16.0, None, 16), attn(12, 4, 128, 64, 128, 65, 256, base=2e5)],
                   {"start": 2, "stop": 3, "times": 3}, eps=1e-6, scale=2.0, cap=20.0),
}


def weights(cfg, seed=0):
    """bf16 tensors under the design's names; gains such that every mechanism moves the logits and states last, and such that
    the norms of recurrent outputs seldom divide by next to nothing."""
    g = torch.Generator().manual_seed(seed)
    D, S, t = cfg["width"], cfg["streams"], {}

    def mat(name, n, k, gain=1.0):
        t[name] = torch.randn(n, k, generator=g) * (gain / k ** 0.5)

    def vec(name, n, mean=0.0, std=0.3):
        t[name] = mean + std * torch.randn(n, generator=g)

    t["embed"] = torch.randn(cfg["vocab"], D, generator=g)
    mat("head", cfg["vocab"], D)
    vec("final.norm", D, 0.0, 0.2)
    for i, ly in enumerate(cfg["layers"]):
        p, m = f"l{i}.", ly["mixer"]
        for q in (1, 2) if ly["mlp"] else (1,):
            vec(f"{p}norm{q}", D, 0.0, 0.2)
            vec(f"{p}hc{q}.in", S, 1.0 / S, 0.3)
            vec(f"{p}hc{q}.out", S, 0.5, 0.3)
            t[f"{p}hc{q}.mix"] = 0.9 * torch.eye(S) + 0.15 * torch.randn(S, S, generator=g)
        p += "mix."
        if ly["type"] == "attention":
            H, G, dk, dv = m["heads"], m["kv_heads"], m["dim"], m["vdim"]
            for n, rows in (("q", H * dk), ("k", G * dk), ("v", G * dv)):
                mat(p + n, rows, D)
                vec(f"{p}{n}.b", rows)
            vec(p + "q.norm", H * dk, 1.2, 0.2)
            vec(p + "k.norm", G * dk, 1.2, 0.2)
            vec(p + "sink", H, 0.5, 1.0)
            mat(p + "o", D, H * dv, 2.0)
        elif ly["type"] == "mamba2":
            H, inner, bc = m["heads"], m["heads"] * m["vdim"], 2 * m["groups"] * m["state"]
            mat(p + "in", 2 * inner + bc + H, D, 1.5)
            mat(p + "conv", inner + bc, m["conv"], 1.5)
            vec(p + "conv.b", inner + bc)
            vec(p + "dt_bias", H, -2.0, 1.0)
            vec(p + "A_log", H, -1.5, 1.0)
            vec(p + "D", H, 1.2)
            vec(p + "norm", inner, 1.0, 0.2)
            mat(p + "o", D, inner)
        else:
            H, dk, dv, r = m["heads"], m["dim"], m["vdim"], ly["rank"]
            for n, rows, k in (("q", H * dk, D), ("k", H * dk, D), ("v", H * dv, D), ("g", H * dv, D), ("a1", r, D), ("a2", H * dk, r)):
                mat(p + n, rows, k, 1.5)
            t[p + "k"] = 0.6 * t[p + "k"] + 0.6 * t[p + "q"]          # q . k away from zero: its sign survives rounding
            vec(p + "a2.b", H * dk, 1.0, 1.0)
            vec(p + "norm", dv, 1.0, 0.2)
            mat(p + "o", D, H * dv)
        if ly["mlp"]:
            p, ff = f"l{i}.mlp.", ly["mlp"]["ff"]
            mat(p + "gate", ff, D)
            mat(p + "up", ff, D)
            mat(p + "down", D, ff)
    return {k: v.to(torch.bfloat16) for k, v in t.items()}
