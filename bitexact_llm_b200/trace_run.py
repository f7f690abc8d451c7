"""Replays a trace of token ids through a model and writes logits:

    bin/trace_run --model DIR --dtype bfloat16|float32 --out DIR --max-tokens N

Standard input holds one step per line, {"step": 0, "entries": [{"id": "a", "tokens": [5, 17], "want": [0, 1]}],
"end": ["a"]}: the next tokens of each request, the places among them whose logits are written to DIR/<step>.f32 (float32,
[wanted, vocab], in the order given), and the requests that are over after the step. After every step the line
"done <step>" is printed. The steps go through `decode.Session`: the engine, caches and kernels that serve the model.

Exit codes: 0 at the end of the input, 3 when the model has no engine in the number format asked for."""

import argparse
import json
import os
import sys

SLOTS = 64          # requests alive at a time


def parse(argv=None):
    ap = argparse.ArgumentParser(prog="trace_run", description=__doc__.split("\n")[0])
    ap.add_argument("--model", required=True)
    ap.add_argument("--dtype", required=True, choices=["bfloat16", "float32"])
    ap.add_argument("--out", required=True)
    ap.add_argument("--max-tokens", type=int, default=4096, help="tokens that live requests hold at any time")
    return ap.parse_args(argv)


class Replay:
    """Requests by name over the sequences of a session."""

    def __init__(self, session):
        self.ses = session
        self.seq = {}
        self.idle = list(range(session.B))[::-1]

    def step(self, entries):
        """-> float32 logits [wanted, vocab] of the step, or None."""
        import torch
        for e in entries:
            if e["id"] not in self.seq:
                self.seq[e["id"]] = self.idle.pop()
        rows = self.ses.feed([(self.seq[e["id"]], e["tokens"]) for e in entries])
        want = [r[torch.tensor(e["want"], device=r.device)] for e, r in zip(entries, rows) if e["want"]]
        return self.ses.eng.logits_float(torch.cat(want)).cpu() if want else None

    def end(self, name):
        s = self.seq.pop(name)
        self.ses.release(s)
        self.idle.append(s)


def main(argv=None):
    args = parse(argv)
    from . import build, registry
    fam = registry.family(registry.read_config(args.model))
    dtype = args.dtype
    if dtype not in fam.dtypes:
        if dtype == "float32":
            print("trace_run: this model has no 32-bit engine", file=sys.stderr)
            return 3
        dtype = fam.serving_dtype
    for target in fam.libraries:
        build.build(target=target)
    from .decode import Session
    n = max(1, args.max_tokens)
    eng = registry.load(args.model, dtype=dtype, max_len=n)
    replay = Replay(Session(eng, SLOTS, n, pages=(n + eng.page - 1) // eng.page + SLOTS))
    for line in sys.stdin:
        if not line.strip():
            continue
        s = json.loads(line)
        logits = replay.step(s["entries"])
        if logits is not None:
            eng.check()
            with open(os.path.join(args.out, f"{s['step']}.f32"), "wb") as f:
                f.write(logits.numpy().astype("<f4").tobytes())
        for name in s["end"]:
            replay.end(name)
        print(f"done {s['step']}", flush=True)
    eng.check()
    return 0


if __name__ == "__main__":
    sys.exit(main())
