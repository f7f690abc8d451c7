"""The residual of a hybrid float model: one stream with layer norms, or several with hyper-connections and RMS norms.

An object holds the rows of one forward call. `open(sub, zero)` gives the normed input of the next sublayer, `target()` the
rows its output goes to and whether it is added there, `due(experts)` hands over what is still due to those rows, `close()`
returns the residual float [M, D]. `sub` is what `prepare` made of the sublayer's tensors; `final_norm` belongs to the head."""

import torch

from . import ops
from .layers import _vec


class LayerNormResidual:
    """One residual x float [M, D]; sublayers add to it, experts' outputs are folded into the next norm."""

    def __init__(self, eng, M, ids):
        self.eng, self.start, self.experts = eng, dict(ids=ids, embed=eng.embed), None
        self.x = torch.empty(M, eng.D, dtype=torch.float32, device=eng.dev)
        self.h = torch.empty(M, ops.pad8(eng.D), dtype=eng.dtype, device=eng.dev)

    @staticmethod
    def prepare(norm, hc, dev):
        return tuple(_vec(t, dev) for t in norm)

    def open(self, sub, zero=None):
        ops.norm(self.x, *sub, self.eng.spec.eps, self.h, experts=self.experts, zero=zero, **self.start)
        self.start, self.experts = {}, None
        return self.h

    def target(self):
        return self.x, True

    def due(self, experts):
        self.experts = experts

    def close(self):
        if self.experts is not None or self.start:
            ops.norm(self.x, None, None, self.eng.spec.eps, experts=self.experts, **self.start)
        return self.x

    @staticmethod
    def final_norm(x, norm, eps, h):
        ops.norm(x, *norm, eps, h)


class StreamsResidual:
    """Streams float [M, S, D]; a sublayer reads a weighted sum of them and its output y is mixed into all of them, in one
    kernel with the next sublayer's norm."""

    def __init__(self, eng, M, ids):
        self.eng, self.start, self.update, self.sub = eng, (ids, eng.embed), None, None
        self.x = torch.empty(M, eng.spec.streams, eng.D, dtype=torch.float32, device=eng.dev)
        self.y = torch.empty(M, eng.D, dtype=torch.float32, device=eng.dev)
        self.h = torch.empty(M, ops.pad8(eng.D), dtype=eng.dtype, device=eng.dev)

    @staticmethod
    def prepare(norm, hc, dev):
        return (1.0 + _vec(norm, dev),) + (tuple(_vec(hc[k], dev) for k in ("in", "out", "mix")) if hc is not None else ())

    def open(self, sub, zero=None):
        if zero is not None:
            zero.zero_()
        w, mix_in, out, mix = sub
        ops.streams(self.x, self.eng.spec.eps, self.start, self.update, mix_in, w, self.h)
        self.start, self.update = None, (self.y, out, mix)
        return self.h

    def target(self):
        return self.y, False

    def due(self, experts):
        if experts is not None:
            ops.norm(self.y, None, None, self.eng.spec.eps, experts=experts)

    def close(self):
        total = torch.empty_like(self.y)
        ops.streams(self.x, self.eng.spec.eps, self.start, self.update, total=total)
        return total

    @staticmethod
    def final_norm(x, norm, eps, h):
        ops.streams(x[:, None], eps, w=norm[0], h=h)
