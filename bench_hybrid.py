"""Throughput of the hybrid float models: Fedatar beside the integer Llama, `python bench.py --workload hybrid`, and Veredra
beside Fedatar, `python bench.py --workload veredra`.

Three sizes that resemble a real model's layers (random weights): 16 layers of width 2048 and of width 1024, 4 layers of
width 4096; minGRU and latent-attention layers alternate, the first feed-forward is dense, the others have 8 experts (two
per token) and a shared one, sized so that a token's active weights per layer are those of a Llama layer of that width
(three matrices of 4 x width; at 4096 the integer kernels' limit, 14336). Beside it the integer Llama of the same width, depth
and vocabulary, in exact mode and in int8 mode. Veredra: `veredra_config` (a gated feed-forward of the same weights). Prompts: 4 x 2048 tokens through `Session.prefill`; decoding: batches of 1, 16 and 256
after 512-token prompts, the whole step (forward, head, sampler at T = 0.7) replayed from one CUDA graph.
Every number is device time from CUDA events after warm-up; the weights exceed L2. One JSON line per model and size."""

import json
import statistics

VOCAB = 128256
SIZES = {"w2048": (2048, 16), "w1024": (1024, 16), "w4096": (4096, 4)}
DECODE_BATCHES = (1, 16, 256)
PROMPT, PREFILL_BATCH, PREFILL_LEN = 512, 4, 2048


def hybrid_config(width, layers, vocab=VOCAB):
    def ff(i):
        if i == 0:
            return {"kind": "dense", "ff": 6 * width}
        return {"kind": "moe", "router": {"experts": 8, "top": 2}, "expert": {"ff": 2 * width}, "shared": {"ff": 2 * width}}

    def mixer(i):
        if i % 2 == 0:
            return "mingru", {"width": width}
        return "latent_attention", {"heads": width // 64, "dim": 64, "rot_dim": 32, "vdim": 64, "q_rank": 3 * width // 8,
                                    "kv_rank": 256, "rot": {"base": 1e6, "dims": 32}, "scale": 96 ** -0.5,
                                    "mask": {"size": 1024}}
    out = []
    for i in range(layers):
        kind, m = mixer(i)
        out.append({"type": kind, "mixer": m, "mlp": ff(i)})
    return {"architecture": "Fedatar", "vocab": vocab, "width": width, "norm": {"eps": 1e-6}, "layers": out}


def random_weights(cfg, dev, seed=0):
    """bf16 tensors under the design's names, generated on the device."""
    import torch
    g = torch.Generator(device=dev).manual_seed(seed)
    D, t = cfg["width"], {}

    def mat(name, n, k):
        t[name] = (torch.randn(n, k, generator=g, device=dev) * k ** -0.5).to(torch.bfloat16)

    def vec(name, n, mean=0.0):
        t[name] = (mean + 0.1 * torch.randn(n, generator=g, device=dev)).to(torch.bfloat16)

    def norm(name):
        vec(name, D, 1.0)
        vec(name + ".b", D)

    mat("embed", cfg["vocab"], D)
    mat("head", cfg["vocab"], D)
    norm("final.norm")
    for i, ly in enumerate(cfg["layers"]):
        p, m, f = f"l{i}.", ly["mixer"], ly["mlp"]
        norm(p + "norm1")
        norm(p + "norm2")
        if ly["type"] == "mingru":
            for n in "zxg":
                mat(p + "mix." + n, m["width"], D)
            vec(p + "mix.z.b", m["width"], -1.0)
            vec(p + "mix.x.b", m["width"])
            mat(p + "mix.o", D, m["width"])
        else:
            H, R = m["heads"], m["kv_rank"]
            for n, a, b in (("dq", m["q_rank"], D), ("uq", H * (m["dim"] + m["rot_dim"]), m["q_rank"]), ("dkv", R + m["rot_dim"], D),
                            ("uk", H * m["dim"], R), ("uv", H * m["vdim"], R), ("g", H, D), ("o", D, H * m["vdim"])):
                mat(p + "mix." + n, a, b)
            vec(p + "mix.dq.norm", m["q_rank"], 1.0)
            vec(p + "mix.dkv.norm", R, 1.0)
            vec(p + "mix.sink", H)
        if f["kind"] == "dense":
            mat(p + "mlp.up", f["ff"], D)
            mat(p + "mlp.down", D, f["ff"])
            vec(p + "mlp.act", 2)
        else:
            names = [(f"e{e}", f["expert"]["ff"]) for e in range(f["router"]["experts"])] + [("shared", f["shared"]["ff"])]
            for n, ff in names:
                mat(p + f"mlp.{n}.up", ff, D)
                mat(p + f"mlp.{n}.down", D, ff)
            mat(p + "mlp.router", f["router"]["experts"], D)
            vec(p + "mlp.router.b", f["router"]["experts"])
    return t


def veredra_config(width, layers, vocab=VOCAB):
    """Gated linear attention, attention and Mamba-2 in turn, two streams, no layer repeated; a gated feed-forward of 4 x width."""
    mixers = [("gla", {"heads": max(1, width // 256), "dim": 128, "vdim": 256, "tau": 16.0}),
              ("attention", {"heads": width // 128, "kv_heads": width // 512, "dim": 128, "vdim": 128, "scale": 128 ** -0.5,
                             "rot": {"base": 1e6, "dims": 128}, "mask": {"size": 1024}}),
              ("mamba2", {"heads": width // 32, "vdim": 64, "state": 128, "groups": 8, "conv": 4, "norm_groups": 8})]
    out = [{"type": mixers[i % 3][0], "mixer": mixers[i % 3][1], "mlp": {"kind": "dense", "ff": 4 * width}} for i in range(layers)]
    return {"architecture": "Veredra", "vocab": vocab, "width": width, "streams": 2, "norm": {"eps": 1e-6}, "logit_scale": 1.0,
            "logit_softcap": 30.0, "loop": None, "layers": out}


def veredra_weights(cfg, dev, seed=0):
    """bf16 tensors under the design's names, generated on the device."""
    import torch
    g = torch.Generator(device=dev).manual_seed(seed)
    D, S, t = cfg["width"], cfg["streams"], {}

    def mat(name, n, k):
        t[name] = (torch.randn(n, k, generator=g, device=dev) * k ** -0.5).to(torch.bfloat16)

    def vec(name, n, mean=0.0):
        t[name] = (mean + 0.1 * torch.randn(n, generator=g, device=dev)).to(torch.bfloat16)

    mat("embed", cfg["vocab"], D)
    mat("head", cfg["vocab"], D)
    vec("final.norm", D)
    for i, ly in enumerate(cfg["layers"]):
        p, m, ff = f"l{i}.", ly["mixer"], ly["mlp"]["ff"]
        for q in (1, 2):
            vec(f"{p}norm{q}", D)
            vec(f"{p}hc{q}.in", S, 1.0 / S)
            vec(f"{p}hc{q}.out", S, 0.7)
            t[f"{p}hc{q}.mix"] = torch.eye(S, device=dev).to(torch.bfloat16)
        for n, a, b in (("gate", ff, D), ("up", ff, D), ("down", D, ff)):
            mat(f"{p}mlp.{n}", a, b)
        p += "mix."
        H = m["heads"]
        if ly["type"] == "attention":
            for n, rows in (("q", H * m["dim"]), ("k", m["kv_heads"] * m["dim"]), ("v", m["kv_heads"] * m["vdim"])):
                mat(p + n, rows, D)
                vec(f"{p}{n}.b", rows)
                if n != "v":
                    vec(f"{p}{n}.norm", rows, 1.0)
            vec(p + "sink", H)
            mat(p + "o", D, H * m["vdim"])
        elif ly["type"] == "gla":
            nk, nv = H * m["dim"], H * m["vdim"]
            for n, rows, k in (("q", nk, D), ("k", nk, D), ("v", nv, D), ("g", nv, D), ("a1", 16, D), ("a2", nk, 16)):
                mat(p + n, rows, k)
            vec(p + "a2.b", nk, 2.0)
            vec(p + "norm", m["vdim"], 1.0)
            mat(p + "o", D, nv)
        else:
            inner, bc = H * m["vdim"], 2 * m["groups"] * m["state"]
            mat(p + "in", 2 * inner + bc + H, D)
            mat(p + "conv", inner + bc, m["conv"])
            for n, size, mean in (("conv.b", inner + bc, 0.0), ("dt_bias", H, -3.0), ("A_log", H, 0.0), ("D", H, 1.0), ("norm", inner, 1.0)):
                vec(p + n, size, mean)
            mat(p + "o", D, inner)
    return t


def veredra_engine(width, layers, dev="cuda"):
    from bitexact_llm_b200.hybrid import veredra
    cfg = veredra_config(width, layers)
    return veredra.load(cfg, veredra_weights(cfg, dev), dev, "bfloat16")


def hybrid_engine(width, layers, dev="cuda"):
    from bitexact_llm_b200.hybrid import fedatar
    cfg = hybrid_config(width, layers)
    return fedatar.load(cfg, random_weights(cfg, dev), dev, "bfloat16")


def llama_engine(width, layers, mode, dev="cuda"):
    from bitexact_llm_b200.exact import consts
    cfg = dict(consts.LLAMA_1B, hidden_size=width, intermediate_size=min(4 * width, 14336), num_hidden_layers=layers,
               num_attention_heads=width // 64, num_key_value_heads=max(1, width // 256), head_dim=64)
    sd = consts.random_state_dict(cfg, seed=0, device=dev)
    if mode == "exact":
        from bitexact_llm_b200.vllm_plugin.exact_run import ExactEngine
        return ExactEngine(consts.build(cfg, sd, n_pos=PREFILL_LEN + 64), dev)
    from bitexact_llm_b200.int8 import consts as consts8
    from bitexact_llm_b200.int8.engine import IntEngine
    return IntEngine(consts8.build(cfg, sd, n_pos=PREFILL_LEN + 64), dev)


def event_ms(fn, n):
    import torch
    torch.cuda.synchronize()
    a, b = torch.cuda.Event(enable_timing=True), torch.cuda.Event(enable_timing=True)
    a.record()
    for _ in range(n):
        fn()
    b.record()
    torch.cuda.synchronize()
    return a.elapsed_time(b) / n


def measure(eng, steps, warmup):
    """-> {"prefill_tok_s": .., "decode": {batch: {"tok_s", "ms_per_step"}}} of one engine."""
    import torch

    from bitexact_llm_b200.decode import GraphDecoder, Session
    g = torch.Generator().manual_seed(1)
    ids = torch.randint(0, eng.V, (PREFILL_BATCH, PREFILL_LEN), generator=g)
    ses = Session(eng, PREFILL_BATCH, PREFILL_LEN)

    def prompt():
        ses.lens.zero_()
        ses.prefill(ids, chunk_rows=PREFILL_BATCH * PREFILL_LEN)
    for _ in range(max(3, warmup)):
        prompt()
    ms = statistics.median(event_ms(prompt, 1) for _ in range(7))
    out = {"prefill_tok_s": PREFILL_BATCH * PREFILL_LEN / ms * 1e3, "prefill_ms": ms, "decode": {}}
    del ses
    for B in DECODE_BATCHES:
        ids = torch.randint(0, eng.V, (B, PROMPT), generator=g)
        ses = Session(eng, B, PROMPT + 4 * steps + warmup + 16)
        h = ses.prefill(ids, chunk_rows=8192)
        rows = torch.zeros(B, 4, dtype=torch.long, device=eng.dev)
        rows[:, 0], rows[:, 2], rows[:, 3] = torch.arange(B), 7, 10
        dec = GraphDecoder(ses, rows, h, warmup=2)
        for _ in range(max(3, warmup)):
            dec.step()
        ms = statistics.median(event_ms(dec.step, steps) for _ in range(3))
        out["decode"][B] = {"tok_s": B / ms * 1e3, "ms_per_step": ms}
        del dec, ses
    eng.check()
    return out


def run(args):
    import torch

    from bitexact_llm_b200 import build
    for target in build.TARGETS:
        build.build(target=target)
    for name, (width, layers) in SIZES.items():
        models = {"Veredra bf16": lambda: veredra_engine(width, layers), "Fedatar bf16": lambda: hybrid_engine(width, layers),
                  "Llama exact": lambda: llama_engine(width, layers, "exact"),
                  "Llama int8": lambda: llama_engine(width, layers, "int8")}
        for model, make in list(models.items())[:2] if args.workload == "veredra" else list(models.items())[1:]:
            eng = make()
            torch.cuda.empty_cache()
            r = measure(eng, args.steps, args.warmup)
            print(json.dumps({"workload": args.workload, "size": name, "width": width, "layers": layers, "model": model,
                              "data": "synthetic", **r}), flush=True)
            del eng
            torch.cuda.empty_cache()
