"""Plain float64 restatement of the Veredra design: gated linear attention, Mamba-2 and sliding-window attention layers on
several residual streams.  Oracle: test infrastructure only, shares no code with the product package.

Same conventions as oracle/hybrid.py: one function per mechanism, one sequence at a time, the whole sequence h [T, .] at
once and token by token where there is a state, matrices [out, in], `mat(h, W)` is h W^T.
"""

import numpy as np

from .hybrid import F, mat, rms_norm, sigmoid, silu, sink_softmax, softplus, sub, window_mask


def gelu_tanh(z):
    return 0.5 * z * (1.0 + np.tanh(np.sqrt(2.0 / np.pi) * (z + 0.044715 * z ** 3)))


def rotate_halves(v, base, dims, first=0):
    """v [T, ..., n]: entries i and i + dims / 2 of the first `dims` turn by position * base^(-2i / dims)."""
    half = dims // 2
    out = v.copy()
    pos = np.arange(first, first + v.shape[0], dtype=F).reshape((-1,) + (1,) * (v.ndim - 1))
    ang = pos * base ** (-2.0 * np.arange(half, dtype=F) / dims)
    a, b = v[..., :half], v[..., half:dims]
    out[..., :half] = a * np.cos(ang) - b * np.sin(ang)
    out[..., half:dims] = b * np.cos(ang) + a * np.sin(ang)
    return out


def attention(h, w, cfg, eps):
    T, H, G, dk, dv = h.shape[0], cfg["heads"], cfg["kv_heads"], cfg["dim"], cfg["vdim"]
    rot = cfg["rot"]
    q = rms_norm(mat(h, w["q"]) + w["q.b"], w["q.norm"], eps).reshape(T, H, dk)
    k = rms_norm(mat(h, w["k"]) + w["k.b"], w["k.norm"], eps).reshape(T, G, dk)
    v = (mat(h, w["v"]) + w["v.b"]).reshape(T, G, dv)
    q, k = rotate_halves(q, rot["base"], rot["dims"]), rotate_halves(k, rot["base"], rot["dims"])
    own = np.arange(H) // (H // G)                                    # the key/value head of each query head
    s = np.einsum("ihd,jhd->hij", q, k[:, own]) * cfg["scale"]
    p = sink_softmax(s, window_mask(T, (cfg.get("mask") or {}).get("size")), w["sink"])
    return mat(np.einsum("hij,jhd->ihd", p, v[:, own]).reshape(T, H * dv), w["o"])


def causal_conv(u, w, b):
    """u [T, C], w [C, taps] (last column: the current token), zeros before the start."""
    taps = w.shape[1]
    pad = np.concatenate([np.zeros((taps - 1, u.shape[1])), u])
    return b + sum(pad[j:j + u.shape[0]] * w[:, j] for j in range(taps))


def linear_recurrence(q, k, v, decay):
    """S_t = diag(decay_t) S_(t-1) + k_t v_t^T, o_t = S_t^T q_t; q, k, decay [T, H, n], v [T, H, m] -> (o, last S [H, n, m])."""
    T, H, n = k.shape
    S = np.zeros((H, n, v.shape[2]))
    o = np.empty((T, H, v.shape[2]))
    for t in range(T):
        S = decay[t][:, :, None] * S + k[t][:, :, None] * v[t][:, None, :]
        o[t] = np.einsum("hnm,hn->hm", S, q[t])
    return o, S


def mamba2(h, w, cfg, eps):
    """-> (output [T, D], state after the last token [heads, N, vdim])."""
    T, H, P, N, G = h.shape[0], cfg["heads"], cfg["vdim"], cfg["state"], cfg["groups"]
    inner = H * P
    u = mat(h, w["in"])
    z, xbc, dt = u[:, :inner], u[:, inner:2 * inner + 2 * G * N], u[:, 2 * inner + 2 * G * N:]
    xbc = silu(causal_conv(xbc, w["conv"], w["conv.b"]))
    x = xbc[:, :inner].reshape(T, H, P)
    own = np.arange(H) // (H // G)
    B = xbc[:, inner:inner + G * N].reshape(T, G, N)[:, own]
    C = xbc[:, inner + G * N:].reshape(T, G, N)[:, own]
    dt = softplus(dt + w["dt_bias"])                                  # [T, H]
    decay = np.exp(-np.exp(w["A_log"]) * dt)[:, :, None] * np.ones(N)
    y, S = linear_recurrence(C, B * dt[:, :, None], x, decay)
    y = (y + w["D"][:, None] * x).reshape(T, inner) * silu(z)
    parts = y.reshape(T, cfg["norm_groups"], -1)
    y = rms_norm(parts, 1.0, eps).reshape(T, inner) * w["norm"]
    return mat(y, w["o"]), S


def gla(h, w, cfg, eps):
    """-> (output [T, D], state after the last token [heads, dim, vdim])."""
    T, H, n, m = h.shape[0], cfg["heads"], cfg["dim"], cfg["vdim"]
    q = mat(h, w["q"]).reshape(T, H, n) * n ** -0.5
    k, v = mat(h, w["k"]).reshape(T, H, n), mat(h, w["v"]).reshape(T, H, m)
    z = mat(mat(h, w["a1"]), w["a2"]) + w["a2.b"]
    decay = np.exp(-softplus(-z) / cfg["tau"]).reshape(T, H, n)       # sigmoid(z)^(1/tau)
    o, S = linear_recurrence(q, k, v, decay)
    o = rms_norm(o, w["norm"], eps).reshape(T, H * m)
    return mat(o * silu(mat(h, w["g"])), w["o"]), S


def gated_ff(h, w):
    return mat(gelu_tanh(mat(h, w["gate"])) * mat(h, w["up"]), w["down"])


def hyper_in(xs, hc):
    """xs [streams, T, D] -> the sublayer's input before its norm."""
    return np.einsum("s,std->td", hc["in"], xs)


def hyper_out(xs, hc, y):
    """Every stream from the old streams (mix[from, to]) and the sublayer's output."""
    return np.einsum("st,snd->tnd", hc["mix"], xs) + hc["out"][:, None, None] * y


def layer_order(cfg):
    n, loop = len(cfg["layers"]), cfg.get("loop")
    if not loop:
        return list(range(n))
    a, b = loop["start"], loop["stop"]
    return list(range(a)) + list(range(a, b)) * loop["times"] + list(range(b, n))


MIXERS = {"attention": lambda *a: attention(*a), "mamba2": lambda *a: mamba2(*a)[0], "gla": lambda *a: gla(*a)[0]}


def forward(cfg, w, tokens):
    """-> (logits [T, vocab], sum of the streams after every layer run [runs, T, D]) of one sequence."""
    w = {k: np.asarray(v, F) for k, v in w.items()}
    eps = cfg["norm"]["eps"]
    xs = np.stack([w["embed"][np.asarray(tokens)]] * cfg["streams"])
    after = []
    for i in layer_order(cfg):
        ly, p = cfg["layers"][i], f"l{i}."
        hc = sub(w, p + "hc1.")
        y = MIXERS[ly["type"]](rms_norm(hyper_in(xs, hc), 1.0 + w[p + "norm1"], eps), sub(w, p + "mix."), ly["mixer"], eps)
        xs = hyper_out(xs, hc, y)
        if ly["mlp"] is not None:
            hc = sub(w, p + "hc2.")
            xs = hyper_out(xs, hc, gated_ff(rms_norm(hyper_in(xs, hc), 1.0 + w[p + "norm2"], eps), sub(w, p + "mlp.")))
        after.append(xs.sum(0))
    z = mat(rms_norm(xs.sum(0), 1.0 + w["final.norm"], eps), w["head"]) * cfg["logit_scale"]
    return cfg["logit_softcap"] * np.tanh(z / cfg["logit_softcap"]), np.stack(after)


def greedy(cfg, w, tokens, n):
    toks = list(tokens)
    for _ in range(n):
        toks.append(int(forward(cfg, w, toks)[0][-1].argmax()))
    return toks[len(tokens):]
