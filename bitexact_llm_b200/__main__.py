"""Command line:

    python -m bitexact_llm_b200 generate --model DIR --prompt 5,17,3 [--prompt ...] [--max-new N] [--dtype D]
                                         [--temperature T] [--seed S]
    python -m bitexact_llm_b200 trace --model DIR --dtype D --out DIR --max-tokens N   (see trace_run.py)

`generate` loads the folder through the model registry, decodes the prompts (token ids) as one batch and prints one line of
generated ids per prompt: greedy at temperature 0 (default), else the integer Gumbel sampler keyed by (seed + row, index)."""

import argparse
import sys


def generate(argv):
    ap = argparse.ArgumentParser(prog="bitexact_llm_b200 generate")
    ap.add_argument("--model", required=True)
    ap.add_argument("--prompt", action="append", required=True, help="token ids with commas between them")
    ap.add_argument("--max-new", type=int, default=16)
    ap.add_argument("--dtype", default=None, help="number format of the engine (default: the model family's own)")
    ap.add_argument("--temperature", type=float, default=0.0)
    ap.add_argument("--seed", type=int, default=0)
    args = ap.parse_args(argv)
    import torch

    from . import build, registry
    from .decode import generate as run
    from .vllm_plugin.sampler import temp_ratio
    prompts = [[int(v) for v in p.split(",")] for p in args.prompt]
    longest = max(map(len, prompts))
    fam = registry.family(registry.read_config(args.model))
    for target in sorted(set(fam.libraries) | {"integer"}):          # the sampler lives in the integer library
        build.build(target=target)
    eng = registry.load(args.model, dtype=args.dtype, max_len=longest + args.max_new)
    ids = torch.zeros(len(prompts), longest, dtype=torch.long)
    for i, p in enumerate(prompts):
        ids[i, : len(p)] = torch.tensor(p)
    tn, td = temp_ratio(args.temperature)
    toks, _ = run(eng, ids, args.max_new, tn, td, seeds=[args.seed + i for i in range(len(prompts))], hashes=False,
                  lens=torch.tensor([len(p) for p in prompts]))
    for row in toks.tolist():
        print(",".join(map(str, row)))
    return 0


def main(argv):
    if argv[:1] == ["generate"]:
        return generate(argv[1:])
    if argv[:1] == ["trace"]:
        from .trace_run import main as trace
        return trace(argv[1:])
    print(__doc__, file=sys.stderr)
    return 2


if __name__ == "__main__":
    sys.exit(main(sys.argv[1:]))
