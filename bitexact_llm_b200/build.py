"""Build the CUDA libraries in-tree with nvcc for sm_100a:  python -m bitexact_llm_b200.build [target ...] [--force] [-v]

Targets: `integer` (libbitexact_b200.so, the integer engines and the sampler) and `float` (libbitexact_float.so, the
float models). Without a target both are built."""

import os
import subprocess
import sys

HERE = os.path.dirname(os.path.abspath(__file__))
SRC = os.path.join(HERE, "csrc")
INCLUDE = os.path.join(os.path.dirname(HERE), "include")
# target -> (translation unit, library)
TARGETS = {"integer": ("capi.cu", "libbitexact_b200.so"), "float": ("float_capi.cu", "libbitexact_float.so")}
OUT = os.path.join(HERE, "_lib", TARGETS["integer"][1])


def library(target):
    return os.path.join(HERE, "_lib", TARGETS[target][1])


def sources(target="integer"):
    """What the target is compiled from (the integer library uses none of the fl_*.cuh headers)."""
    tu = TARGETS[target][0]
    names = [f for f in os.listdir(SRC) if f == tu or (f.endswith(".cuh") and (target == "float" or not f.startswith("fl_")))]
    heads = ["bitexact_b200.h"] + (["bitexact_float.h"] if target == "float" else [])
    return sorted(os.path.join(SRC, f) for f in names) + [os.path.join(INCLUDE, h) for h in heads]


def up_to_date(target="integer"):
    out = library(target)
    if not os.path.exists(out):
        return False
    t = os.path.getmtime(out)
    return all(os.path.getmtime(s) <= t for s in sources(target))


def build(force=False, verbose=False, target="integer"):
    out = library(target)
    if not force and up_to_date(target):
        return out
    os.makedirs(os.path.dirname(out), exist_ok=True)
    nvcc = os.environ.get("NVCC", "/usr/local/cuda/bin/nvcc")
    part = f"{out}.{os.getpid()}"                       # moved into place when complete
    cmd = [nvcc, "-gencode", "arch=compute_100a,code=sm_100a", "-O3", "-lineinfo", "-std=c++17",
           "-shared", "-Xcompiler", "-fPIC", "-o", part, os.path.join(SRC, TARGETS[target][0])]
    if verbose:
        cmd[1:1] = ["-Xptxas", "-v"]
    r = subprocess.run(cmd, capture_output=True, text=True)
    if r.returncode != 0:
        raise RuntimeError("nvcc failed:\n" + r.stdout + r.stderr)
    os.replace(part, out)
    if verbose:
        print(r.stdout + r.stderr)
    return out


if __name__ == "__main__":
    for name in [a for a in sys.argv[1:] if a in TARGETS] or list(TARGETS):
        print(build(force="--force" in sys.argv, verbose="-v" in sys.argv, target=name))
