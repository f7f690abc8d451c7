"""Plain float64 restatement of the hybrid float models (recurrent minGRU layers, latent attention, dense and expert
feed-forwards; the Fedatar design).  Oracle: test infrastructure only, shares no code with the product package.

One function per mechanism, one sequence at a time, no cache: every function sees the whole sequence h [T, .] and
returns what each of its positions gets.  Weights come as a dict name -> float array (the names of the weight file).
Notation: rows are tokens, matrices are [out, in], `mat(h, W)` is h W^T.
"""

import numpy as np

F = np.float64


def mat(h, w):
    return h @ w.T


def sigmoid(v):
    return 0.5 * (1.0 + np.tanh(0.5 * v))


def silu(v):
    return v * sigmoid(v)


def softplus(v):
    return np.maximum(v, 0.0) + np.log1p(np.exp(-np.abs(v)))


def rms_norm(v, w, eps):
    return v / np.sqrt((v * v).mean(-1, keepdims=True) + eps) * w


def layer_norm(v, w, b, eps):
    c = v - v.mean(-1, keepdims=True)
    return c / np.sqrt((c * c).mean(-1, keepdims=True) + eps) * w + b


def rotate_pairs(v, base, dims, first=0):
    """v [T, ..., n]: pairs (2i, 2i + 1) of the first `dims` entries turn by position * base^(-2i / dims); row t is
    position first + t."""
    out = v.copy()
    pos = np.arange(first, first + v.shape[0], dtype=F).reshape((-1,) + (1,) * (v.ndim - 1))
    ang = pos * base ** (-np.arange(0, dims, 2, dtype=F) / dims)
    c, s = np.cos(ang), np.sin(ang)
    a, b = v[..., 0:dims:2], v[..., 1:dims:2]
    out[..., 0:dims:2] = a * c - b * s
    out[..., 1:dims:2] = b * c + a * s
    return out


def xielu(z, p, q):
    """p z^2 + z / 2 on the right, (1/2 + q) (e^z - 1 - z) + z / 2 on the left, p and q through softplus."""
    neg = np.minimum(z, 0.0)
    return np.where(z > 0, softplus(p) * z * z, (0.5 + softplus(q)) * (np.expm1(neg) - neg)) + 0.5 * z


def relu2(z):
    return np.maximum(z, 0.0) ** 2


def mingru(h, w_z, b_z, w_x, b_x, w_g, w_o, state=None):
    """-> (output [T, D], state after the last token [width])."""
    z = sigmoid(mat(h, w_z) + b_z)
    u = mat(h, w_x) + b_x
    cand = np.where(u >= 0, u + 0.5, sigmoid(u))
    s = np.zeros(w_z.shape[0], F) if state is None else state.astype(F)
    ss = np.empty_like(z)
    for t in range(h.shape[0]):
        s = (1.0 - z[t]) * s + z[t] * cand[t]
        ss[t] = s
    return mat(ss * silu(mat(h, w_g)), w_o), s


def window_mask(T, size):
    """[query, key] True where the key is visible: 0 <= i - j (< size, when there is one)."""
    d = np.arange(T)[:, None] - np.arange(T)[None, :]
    return (d >= 0) & ((d < size) if size else True)


def sink_softmax(s, mask, sink):
    """s [H, T, T]; weights over the visible keys, exp(sink) added to every denominator (sink [H])."""
    s = np.where(mask, s, -np.inf)
    m = np.maximum(s.max(-1, keepdims=True), sink[:, None, None])
    e = np.exp(s - m)
    return e / (e.sum(-1, keepdims=True) + np.exp(sink[:, None, None] - m))


def latent_attention(h, w, cfg, eps):
    """w: name -> array of one mixer ('dq', 'dq.norm', ...); cfg: the mixer's sizes and constants."""
    T, H, dn, dr, dv, R = h.shape[0], cfg["heads"], cfg["dim"], cfg["rot_dim"], cfg["vdim"], cfg["kv_rank"]
    rot = cfg["rot"]
    q = mat(rms_norm(mat(h, w["dq"]), w["dq.norm"], eps), w["uq"]).reshape(T, H, dn + dr)
    qn, qr = q[..., :dn], rotate_pairs(q[..., dn:], rot["base"], rot["dims"])
    kv = mat(h, w["dkv"])
    c = rms_norm(kv[:, :R], w["dkv.norm"], eps)
    kr = rotate_pairs(kv[:, R:], rot["base"], rot["dims"])
    kn, v = mat(c, w["uk"]).reshape(T, H, dn), mat(c, w["uv"]).reshape(T, H, dv)
    s = (np.einsum("ihd,jhd->hij", qn, kn) + np.einsum("ihd,jd->hij", qr, kr)) * cfg["scale"]
    p = sink_softmax(s, window_mask(T, (cfg.get("mask") or {}).get("size")), w["sink"])
    o = np.einsum("hij,jhd->ihd", p, v) * sigmoid(mat(h, w["g"]))[..., None]
    return mat(o.reshape(T, H * dv), w["o"])


def dense_ff(h, up, down, act):
    return mat(xielu(mat(h, up), act[0], act[1]), down)


def route(h, w_router, b_router, top):
    """-> (chosen experts [T, top], their weights [T, top]); equal logits: the lower index first."""
    z = mat(h, w_router) + b_router
    idx = np.argsort(-z, axis=-1, kind="stable")[:, :top]
    zc = np.take_along_axis(z, idx, -1)
    e = np.exp(zc - zc.max(-1, keepdims=True))
    return idx, e / e.sum(-1, keepdims=True)


def moe_ff(h, w, n_experts, top, shared):
    idx, wt = route(h, w["router"], w["router.b"], top)
    out = np.zeros_like(h)
    for e in range(n_experts):
        g = (wt * (idx == e)).sum(-1)
        rows = np.nonzero((idx == e).any(-1))[0]
        out[rows] += g[rows, None] * mat(relu2(mat(h[rows], w[f"e{e}.up"])), w[f"e{e}.down"])
    if shared:
        out += mat(relu2(mat(h, w["shared.up"])), w["shared.down"])
    return out


def sub(w, prefix):
    return {k[len(prefix):]: v for k, v in w.items() if k.startswith(prefix)}


def forward(cfg, w, tokens):
    """-> (logits [T, vocab], residual stream after every layer [L, T, D]) of one sequence."""
    w = {k: np.asarray(v, F) for k, v in w.items()}
    eps = cfg["norm"]["eps"]
    x = w["embed"][np.asarray(tokens)]
    streams = []
    for i, ly in enumerate(cfg["layers"]):
        p = f"l{i}."
        m = sub(w, p + "mix.")
        h = layer_norm(x, w[p + "norm1"], w[p + "norm1.b"], eps)
        if ly["type"] == "mingru":
            y, _ = mingru(h, m["z"], m["z.b"], m["x"], m["x.b"], m["g"], m["o"])
        else:
            y = latent_attention(h, m, ly["mixer"], eps)
        x = x + y
        f = ly["mlp"]
        if f is not None:
            h = layer_norm(x, w[p + "norm2"], w[p + "norm2.b"], eps)
            m = sub(w, p + "mlp.")
            if f["kind"] == "dense":
                y = dense_ff(h, m["up"], m["down"], m["act"])
            else:
                y = moe_ff(h, m, f["router"]["experts"], f["router"]["top"], f.get("shared"))
            x = x + y
        streams.append(x)
    return mat(layer_norm(x, w["final.norm"], w["final.norm.b"], eps), w["head"]), np.stack(streams)


def greedy(cfg, w, tokens, n):
    toks = list(tokens)
    for _ in range(n):
        toks.append(int(forward(cfg, w, toks)[0][-1].argmax()))
    return toks[len(tokens):]
