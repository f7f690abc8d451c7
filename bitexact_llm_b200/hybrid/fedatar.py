"""The Fedatar design: a decoder-only hybrid of minGRU and latent-attention layers (config key 'layers' gives the order),
pre-norm layer norms with bias, dense xIELU feed-forwards or routed squared-relu experts with a shared one.

`read_config` turns config.json into a ModelSpec, `read_weights` groups the tensors of the weight file (names
'l<i>.norm1', 'l<i>.mix.*', 'l<i>.mlp.*', 'embed', 'final.norm', 'head'; a norm's bias carries '.b')."""

from .engine import HybridEngine
from .spec import DenseSpec, ExpertsSpec, LatentAttentionSpec, LayerSpec, MinGRUSpec, ModelSpec

ARCHITECTURE = "Fedatar"
DTYPES = ("bfloat16", "float32")


def _mixer(kind, m, eps):
    if kind == "mingru":
        return MinGRUSpec(width=m["width"])
    if kind == "latent_attention":
        rot = m["rot"]
        if rot.get("dims", m["rot_dim"]) != m["rot_dim"]:
            raise ValueError("latent_attention: the rotated part is rotated as a whole (rot.dims = rot_dim)")
        return LatentAttentionSpec(heads=m["heads"], dim=m["dim"], rot_dim=m["rot_dim"], vdim=m["vdim"], q_rank=m["q_rank"],
                                   kv_rank=m["kv_rank"], rot_base=float(rot["base"]), scale=float(m["scale"]),
                                   window=int((m.get("mask") or {}).get("size") or 0), eps=eps)
    raise ValueError(f"unknown mixer {kind!r}")


def _ff(f):
    if f is None:
        return None
    if f["kind"] == "dense":
        return DenseSpec(ff=f["ff"])
    if f["kind"] == "moe":
        shared = f.get("shared")
        return ExpertsSpec(experts=f["router"]["experts"], top=f["router"]["top"], ff=f["expert"]["ff"],
                           shared_ff=shared["ff"] if shared else 0)
    raise ValueError(f"unknown feed-forward {f['kind']!r}")


def read_config(cfg):
    eps = float(cfg["norm"]["eps"])
    return ModelSpec(vocab=cfg["vocab"], width=cfg["width"], eps=eps,
                     layers=tuple(LayerSpec(_mixer(ly["type"], ly["mixer"], eps), _ff(ly.get("mlp"))) for ly in cfg["layers"]))


def read_weights(spec, t):
    pair = lambda name: (t[name], t[name + ".b"])
    under = lambda p: {k[len(p):]: v for k, v in t.items() if k.startswith(p)}
    layers = []
    for i, ly in enumerate(spec.layers):
        p = f"l{i}."
        layers.append({"norm1": pair(p + "norm1"), "norm2": pair(p + "norm2") if ly.ff is not None else None,
                       "mixer": under(p + "mix."), "ff": under(p + "mlp.")})
    return {"embed": t["embed"], "head": t["head"], "final": pair("final.norm"), "layers": layers}


def load(cfg, tensors, dev="cuda", dtype="bfloat16", n_layers=None):
    spec = read_config(cfg)
    return HybridEngine(spec, read_weights(spec, tensors), dev, dtype, n_layers)
