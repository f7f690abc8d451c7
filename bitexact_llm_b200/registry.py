"""Model registry: config.json of a model folder -> engine. Every entry builds an engine with the token-row contract of
`engine_base`, so the decode loop, the command line and the trace runner treat all of them alike.

  Fedatar            hybrid.fedatar   dtype bfloat16 (default) or float32
  Veredra            hybrid.veredra   dtype bfloat16 (default) or float32
  LlamaForCausalLM   integer engines  dtype exact (default: original bf16 weights as limbs) or int8

A folder holds config.json and model.safetensors; the integer engines also take constants.bx (`constfile`), which
saves the decomposition of the weights."""

import glob
import json
import os

from .weights import load_safetensors


class UnsupportedDtype(ValueError):
    """The model family has no engine for the requested number format."""


def _tensors(folder):
    files = sorted(glob.glob(os.path.join(folder, "*.safetensors")))
    if not files:
        raise FileNotFoundError(f"{folder}: no .safetensors file")
    out = {}
    for f in files:
        out.update(load_safetensors(f))
    return out


class FedatarFamily:
    dtypes, libraries = ("bfloat16", "float32"), ("float",)
    serving_dtype = "bfloat16"

    @staticmethod
    def load(folder, cfg, dev, dtype, max_len):
        from .hybrid import fedatar
        return fedatar.load(cfg, _tensors(folder), dev, dtype)


class VeredraFamily(FedatarFamily):
    @staticmethod
    def load(folder, cfg, dev, dtype, max_len):
        from .hybrid import veredra
        return veredra.load(cfg, _tensors(folder), dev, dtype)


class LlamaFamily:
    dtypes, libraries = ("exact", "int8"), ("integer",)
    serving_dtype = "exact"

    @staticmethod
    def load(folder, cfg, dev, dtype, max_len):
        from . import constfile
        path = os.path.join(folder, "constants.bx")
        if os.path.exists(path):
            c = constfile.load(path, dev)
        else:
            if dtype == "exact":
                from .exact import consts
            else:
                from .int8 import consts
            sd = {k: v.to(dev) for k, v in _tensors(folder).items()}
            c = consts.build(cfg, sd, n_pos=max_len)
        if dtype == "exact":
            from .vllm_plugin.exact_run import ExactEngine
            return ExactEngine(c, dev)
        from .int8.engine import IntEngine
        return IntEngine(c, dev)


FAMILIES = {"Fedatar": FedatarFamily, "Veredra": VeredraFamily, "LlamaForCausalLM": LlamaFamily}


def read_config(folder):
    with open(os.path.join(folder, "config.json")) as f:
        return json.load(f)


def family(cfg):
    """The registry entry of a config: its 'architecture', or the first known of its 'architectures'."""
    names = [cfg["architecture"]] if "architecture" in cfg else list(cfg.get("architectures", []))
    for n in names:
        if n in FAMILIES:
            return FAMILIES[n]
    raise ValueError(f"unknown architecture {names}; known: {sorted(FAMILIES)}")


def load(folder, dev="cuda", dtype=None, max_len=2048):
    """-> engine. dtype None: the family's serving format; max_len sizes position tables where a family has them."""
    cfg = read_config(folder)
    fam = family(cfg)
    dtype = fam.serving_dtype if dtype is None else dtype
    if dtype not in fam.dtypes:
        raise UnsupportedDtype(f"{dtype}: this model runs in {', '.join(fam.dtypes)}")
    return fam.load(folder, cfg, dev, dtype, max_len)
