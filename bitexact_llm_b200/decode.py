"""A minimal decode loop over any token-row engine (`engine_base`): paged-cache bookkeeping, chunked prompt processing,
greedy / Gumbel-max sampling and per-position logits hashes (the reference's `generate` / `logits_sha`,
src/bitexact/generate.py:21-50, on a batch of sequences with one block-table row each)."""

import hashlib

import torch

from .vllm_plugin import sampler


def logits_sha(row):
    """SHA-256 (hex) of one int64 logits row: equal hashes <=> bit-identical logits."""
    return hashlib.sha256(row.contiguous().cpu().numpy().tobytes()).hexdigest()


class Session:
    """B sequences with one block-table row each (page 0 is the null page; a recurrent layer's state of sequence b is slot
    b of its cache). By default every sequence owns a run of pages for max_len tokens. With `pages`, the cache has that
    many pages for all sequences together: `feed` takes them as a sequence grows and `release` gives them back."""

    def __init__(self, eng, B, max_len, bs=None, perm_seed=None, pages=None):
        bs = eng.page if bs is None else bs
        self.eng, self.B, self.bs = eng, B, bs
        self.nblk = (max_len + bs - 1) // bs
        nb = 1 + (B * self.nblk if pages is None else pages)
        dev = eng.dev
        self.kvs = eng.new_cache(B, nb, bs)
        blocks = torch.arange(1, nb, dtype=torch.int64)
        if perm_seed is not None:                                  # scattered pages
            g = torch.Generator().manual_seed(perm_seed)
            blocks = blocks[torch.randperm(nb - 1, generator=g)]
        self.free = None
        if pages is None:
            self.bt = blocks.view(B, self.nblk).to(torch.int32).to(dev)
        else:
            self.bt = torch.zeros(B, self.nblk, dtype=torch.int32, device=dev)
            self.free = blocks.tolist()[::-1]
            self.held = [[] for _ in range(B)]
        self.lens = torch.zeros(B, dtype=torch.long, device=dev)
        self.rows = torch.arange(B, device=dev)

    def _reserve(self, seq, n):
        """Pages for positions 0 .. n - 1 of the sequence."""
        need = (n + self.bs - 1) // self.bs
        if need > self.nblk:
            raise ValueError(f"sequence {seq}: {n} tokens are beyond the session's max_len")
        if self.free is None or need <= len(self.held[seq]):
            return
        have = len(self.held[seq])
        if need - have > len(self.free):
            raise MemoryError("the session has no free pages")
        new = [self.free.pop() for _ in range(need - have)]
        self.held[seq] += new
        self.bt[seq, have:need] = torch.tensor(new, dtype=torch.int32).to(self.bt.device)

    def release(self, seq):
        """The sequence is finished: its pages go back to the pool and its row may serve another one. Nothing is cleared:
        keys beyond a sequence's length carry no weight, and a recurrent state starts from zero at position 0."""
        if self.free is not None:
            self.free += self.held[seq][::-1]
            self.held[seq] = []
            self.bt[seq] = 0
        self.lens[seq] = 0

    @torch.no_grad()
    def feed(self, entries, chunk_rows=4096):
        """entries: [(sequence, its next tokens)], every sequence at most once; any mix of prompt portions and single
        decode tokens goes through one forward call per chunk_rows rows. Returns the residual rows [n, D] per entry."""
        dev = self.eng.dev
        lens = self.lens.tolist()
        todo = [[int(s), torch.as_tensor(t, dtype=torch.long), lens[s]] for s, t in entries]
        assert len({s for s, _, _ in todo}) == len(todo), "a sequence may appear once per call"
        for s, t, n in todo:
            self._reserve(s, n + len(t))
        out, i = [[] for _ in todo], 0
        while i < len(todo):
            runs, at = [], 0                                       # (entry, sequence, first position, tokens)
            while i < len(todo) and at < chunk_rows:
                s, t, n = todo[i]
                take = min(len(t), chunk_rows - at)
                if take:
                    runs.append((i, s, n, t[:take]))
                    at += take
                todo[i][1], todo[i][2] = t[take:], n + take
                if take == len(t):
                    i += 1
            if not runs:
                continue
            seq = torch.cat([torch.full((len(t),), s) for _, s, _, t in runs]).to(dev)
            pos = torch.cat([torch.arange(n, n + len(t)) for _, _, n, t in runs]).to(dev)
            ids = torch.cat([t for _, _, _, t in runs]).to(dev)
            tt, row = [], 0
            for _, s, n, t in runs:
                tt.append((s, row, len(t), n + len(t)))
                row += len(t)
            longest = max(c for _, _, q, c in tt if q > 1) if any(q > 1 for _, _, q, _ in tt) else 0
            tt = self.eng.tile_table(tt, self.bs) if longest > self.eng.tiles_from else None
            x = self.eng.forward(self.kvs, ids, pos, self._slots(seq, pos), self.bt, seq,
                                 tiles=None if tt is None else tt.to(dev))
            row = 0
            for e, s, n, t in runs:
                out[e].append(x[row:row + len(t)])
                row += len(t)
                self.lens[s] = n + len(t)
        return [torch.cat(o) if o else torch.empty(0, self.eng.D, device=dev) for o in out]

    def _slots(self, seq, pos):
        return self.bt[seq, pos // self.bs].long() * self.bs + pos % self.bs

    @torch.no_grad()
    def import_kv(self, seq, k, v, layers=None):
        """Loads keys / values of positions 0 .. n - 1 of sequence `seq` (int64 [n, HKV, HD] at 17 / 19 fractional
        bits, within three limbs) into the paged cache of the given layers (default: all) and sets the sequence's
        length to n: a prefix computed elsewhere, e.g. by another engine or an earlier session."""
        from .vllm_plugin import tri_paged
        dev = self.eng.dev
        k, v = k.to(dev).long().contiguous(), v.to(dev).long().contiguous()
        n = k.shape[0]
        pos = torch.arange(n, device=dev)
        slot = self._slots(torch.full_like(pos, int(seq)), pos)
        for i in (range(self.eng.L) if layers is None else layers):
            tri_paged.store(self.kvs[i], slot, k, v)
        self.lens[seq] = n

    @torch.no_grad()
    def prefill(self, prompts, lens=None, chunk_rows=4096, tiles=True):
        """prompts: int64 [B, P] right-padded, lens [B] the true lengths (default: all P). Token rows are processed
        in position chunks so that every row's keys are in the cache before it attends; with `tiles` the attention
        of a chunk runs on the prefill tile kernel (runs of 32 / G consecutive tokens share their K / V staging),
        else every token is a row of the decode kernel. Same integers either way. Returns the final residual row of
        each sequence [B, D]."""
        B, P = prompts.shape
        dev = self.eng.dev
        prompts = prompts.to(dev)
        lens_host = [P] * B if lens is None else [int(v) for v in lens.tolist()]
        lens = torch.full((B,), P, dtype=torch.long, device=dev) if lens is None else lens.to(dev).long()
        if self.free is not None:
            for b in range(B):
                self._reserve(b, lens_host[b])
        tile_from = 0 if tiles == "always" else self.eng.tiles_from
        step = max(1, chunk_rows // B)
        last = None
        for p0 in range(0, P, step):
            p1 = min(P, p0 + step)
            grid = torch.arange(p0, p1, device=dev).expand(B, -1)
            live = grid < lens[:, None]
            if not bool(live.any()):
                break
            pos = grid[live]                                                      # sequence-major rows
            seq = self.rows[:, None].expand(-1, p1 - p0)[live]
            tt = None
            if tiles and p1 > tile_from:                                        # sequence-major rows: runs per sequence
                pre, row0 = [], 0
                for b in range(B):
                    n = max(0, min(p1, lens_host[b]) - p0)
                    if n:
                        pre.append((b, row0, n, p0 + n))
                    row0 += n
                tt = self.eng.tile_table(pre, self.bs)
                tt = None if tt is None else tt.to(dev)
            x = self.eng.forward(self.kvs, prompts[:, p0:p1][live], pos, self._slots(seq, pos), self.bt, seq, tiles=tt)
            fin = pos == lens[seq] - 1
            if last is None:
                last = torch.zeros(B, self.eng.D, dtype=x.dtype, device=dev)
            last[seq[fin]] = x[fin]
        self.lens += lens
        return last

    @torch.no_grad()
    def step(self, tokens, pos=None):
        """One decode step: tokens int64 [B] at positions `pos` (default: the lengths tracked on the device).
        Returns the residual rows [B, D]. (With a page pool the pages must be there: `feed` takes them as needed.)"""
        pos = self.lens.clone() if pos is None else pos
        x = self.eng.forward(self.kvs, tokens, pos, self._slots(self.rows, pos), self.bt, self.rows)
        self.lens += 1
        return x


class GraphDecoder:
    """The decode step (LM head, sampler, one forward over the batch) captured once in a CUDA graph and replayed:
    no Python or launch overhead per kernel. The step's state lives in static device tensors: the residual rows,
    the sampler rows (seed, t, tn, td) whose t advances on the device, the session's lengths."""

    def __init__(self, ses, rows, h, warmup=2):
        self.ses, self.eng = ses, ses.eng
        self.rows = rows
        self.h = h.clone()
        self.tok = torch.zeros(ses.B, dtype=torch.long, device=h.device)
        for _ in range(warmup):                     # configures every kernel and fills the caching allocator
            self._body()
        torch.cuda.synchronize()
        self.graph = torch.cuda.CUDAGraph()
        with torch.cuda.graph(self.graph):
            self._body()

    def _body(self):
        lg = self.eng.logits(self.h)
        tok = sampler.sample_rows(lg, self.rows, self.eng.ln, self.eng.FR)
        self.h.copy_(self.ses.step(tok))
        self.rows[:, 1] += 1
        self.tok.copy_(tok)

    def step(self):
        """Runs one captured step; returns the sampled tokens (a static tensor, overwritten by the next step)."""
        self.graph.replay()
        return self.tok


class GraphHostStep:
    """One decode step driven from the host, captured in a CUDA graph: the caller copies this step's token ids,
    positions and sampler rows into the static input tensors (`tok_in`, `pos_in`, `rows_in`), replays, and reads
    the sampled tokens from `tok`. Forward, LM head and sampler run inside the graph."""

    def __init__(self, ses, rows):
        self.ses, self.eng = ses, ses.eng
        dev = rows.device
        self.tok_in = torch.zeros(ses.B, dtype=torch.long, device=dev)
        self.pos_in = ses.lens.clone()
        self.rows_in = rows.clone()
        self.tok = torch.zeros(ses.B, dtype=torch.long, device=dev)
        keep = ses.lens.clone()
        for _ in range(2):
            self._body()
        torch.cuda.synchronize()
        self.graph = torch.cuda.CUDAGraph()
        with torch.cuda.graph(self.graph):
            self._body()
        ses.lens.copy_(keep)                         # warm-up and capture advanced the device-side lengths

    def _body(self):
        x = self.ses.step(self.tok_in, self.pos_in)
        lg = self.eng.logits(x)
        self.tok.copy_(sampler.sample_rows(lg, self.rows_in, self.eng.ln, self.eng.FR))

    def step(self):
        self.graph.replay()
        return self.tok


@torch.no_grad()
def generate(eng, prompts, max_new, tn=0, td=1, seeds=None, hashes=True, max_len=None, perm_seed=None, lens=None):
    """prompts int64 [B, P] (right-padded, true lengths `lens`); generated token t of sequence b uses the noise
    keyed (seeds[b], t). Returns (tokens [B, max_new] on the host, list of per-position hash lists or None)."""
    B, P = prompts.shape
    dev = eng.dev
    seeds = list(range(B)) if seeds is None else seeds
    ses = Session(eng, B, max_len or (P + max_new), perm_seed=perm_seed)
    h = ses.prefill(prompts, lens)
    rows = torch.zeros(B, 4, dtype=torch.long, device=dev)
    rows[:, 0] = torch.tensor(seeds, device=dev)
    rows[:, 2], rows[:, 3] = tn, td
    toks, shas = [], [[] for _ in range(B)]
    for t in range(max_new):
        lg = eng.logits(h)
        rows[:, 1] = t
        y = sampler.sample_rows(lg, rows, eng.ln, eng.FR)
        toks.append(y)
        if hashes:
            for b in range(B):
                shas[b].append(logits_sha(lg[b]))
        if t + 1 < max_new:
            h = ses.step(y)
    eng.check()
    return torch.stack(toks, 1).cpu(), (shas if hashes else None)
