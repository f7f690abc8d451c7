"""The Veredra design: gated linear attention, Mamba-2 and sliding-window attention layers in any order, some of them run
several times in a row, on several residual streams (hyper-connections), RMS norms stored around zero, feed-forwards gated by
the tanh form of gelu, scaled and soft-capped logits.

`read_config` turns config.json into a ModelSpec, `read_weights` groups the tensors of the weight file (names 'l<i>.norm1',
'l<i>.mix.*', 'l<i>.mlp.*', 'l<i>.hc1.*', 'embed', 'final.norm', 'head')."""

import torch

from .engine import HybridEngine
from .spec import AttentionSpec, GatedSpec, GLASpec, LayerSpec, Mamba2Spec, ModelSpec

ARCHITECTURE = "Veredra"
DTYPES = ("bfloat16", "float32")


def _mixer(kind, m, eps):
    if kind == "attention":
        rot = m.get("rot") or {"base": 1.0, "dims": 0}
        return AttentionSpec(heads=m["heads"], kv_heads=m["kv_heads"], dim=m["dim"], vdim=m["vdim"], rot_dims=int(rot["dims"]),
                             rot_base=float(rot["base"]), scale=float(m["scale"]),
                             window=int((m.get("mask") or {}).get("size") or 0), eps=eps)
    if kind == "mamba2":
        return Mamba2Spec(heads=m["heads"], vdim=m["vdim"], state=m["state"], groups=m["groups"], taps=m["conv"],
                          norm_groups=m["norm_groups"], eps=eps)
    if kind == "gla":
        return GLASpec(heads=m["heads"], dim=m["dim"], vdim=m["vdim"], tau=float(m["tau"]), eps=eps)
    raise ValueError(f"unknown mixer {kind!r}")


def _ff(f):
    if f is None:
        return None
    if f["kind"] == "dense":
        return GatedSpec(ff=f["ff"])
    raise ValueError(f"unknown feed-forward {f['kind']!r}")


def _runs(n, loop):
    if not loop:
        return tuple(range(n))
    a, b = loop["start"], loop["stop"]
    if not 0 <= a <= b <= n or loop["times"] < 0:
        raise ValueError("loop: layers start .. stop - 1 of the model, run 'times' times")
    return tuple(range(a)) + tuple(range(a, b)) * loop["times"] + tuple(range(b, n))


def read_config(cfg):
    eps = float(cfg["norm"]["eps"])
    layers = tuple(LayerSpec(_mixer(ly["type"], ly["mixer"], eps), _ff(ly.get("mlp"))) for ly in cfg["layers"])
    return ModelSpec(vocab=cfg["vocab"], width=cfg["width"], eps=eps, layers=layers, runs=_runs(len(layers), cfg.get("loop")),
                     streams=int(cfg.get("streams") or 1), logit_scale=float(cfg.get("logit_scale") or 1.0),
                     logit_softcap=float(cfg.get("logit_softcap") or 0.0))


def read_weights(spec, t):
    under = lambda p: {k[len(p):]: v for k, v in t.items() if k.startswith(p)}
    one = {"in": torch.ones(1), "out": torch.ones(1), "mix": torch.ones(1, 1)}       # the plain residual sum
    layers = []
    for i, ly in enumerate(spec.layers):
        p = f"l{i}."
        streams = lambda q: under(f"{p}hc{q}.") or (one if spec.streams == 1 else None)
        layers.append({"norm1": t[p + "norm1"], "norm2": t[p + "norm2"] if ly.ff is not None else None, "mixer": under(p + "mix."),
                       "ff": under(p + "mlp."), "hc1": streams(1), "hc2": streams(2) if ly.ff is not None else None})
    return {"embed": t["embed"], "head": t["head"], "final": t["final.norm"], "layers": layers}


def load(cfg, tensors, dev="cuda", dtype="bfloat16", n_layers=None):
    spec = read_config(cfg)
    return HybridEngine(spec, read_weights(spec, tensors), dev, dtype, n_layers)
