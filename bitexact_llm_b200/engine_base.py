"""What the decode loop (`decode.Session`, `generate`) asks of an engine besides `forward`, `logits` and `check`: the
per-layer cache of a session and the tile table of a prompt portion. The defaults are those of the integer engines (a
paged limb-plane KV cache in every layer, the prefill tile kernel on longer prompts)."""

import torch


class TokenRowEngine:
    """Engines with D, V, L, FR, ln, dev and forward(caches, ids, pos, slot, bt, rmap, tiles=None)."""

    page = 16               # tokens per cache page of a session
    tiles_from = 384        # prompt portions that end before this position attend row by row
    # (the integer tile kernel pays for itself once a tile walks a few key blocks: 0.83 x the row kernel on 128-token
    # prompts, 1.7 x on 2048-token ones)

    def new_cache(self, n_seqs, n_blocks, bs):
        """The caches of a session of n_seqs sequences over n_blocks pages of bs tokens (page 0: null page), one per
        layer, as `forward` takes them."""
        return [torch.zeros(n_blocks, self.HKV, bs, 8 * self.HD, dtype=torch.int8, device=self.dev) for _ in range(self.L)]

    def tile_table(self, runs, bs):
        """Attention tiles for runs = [(table row, first token row, tokens, context length)] of a step, int32 [T, 3] on
        the host, or None when this engine has no tile kernel for its geometry."""
        from .vllm_plugin import tri_prefill
        G = self.H // self.HKV
        if self.HD != 64 or tri_prefill.BM % G or bs not in (8, 16, 32, 64, 128):
            return None
        return tri_prefill.tile_table(runs, G, tri_prefill.ROWS)

    def logits_float(self, h):
        """`logits` as float32."""
        return (self.logits(h).double() * 2.0 ** -self.FR).float()
