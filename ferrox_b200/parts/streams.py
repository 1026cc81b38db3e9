"""A residual of several streams (hyper-connections): the norm that reads it and the block that writes it.

A token carries a small matrix R whose rows are its streams.  The mixer (1) and the feed-forward (2) of a layer, each with
constants of its own,

    y_q = f_q(norm_q(in_q^T R));   R <- mix_q^T R + out_q y_q^T

The constants are weights and do not depend on the token, so the layer's two updates are one,

    R <- (mix_1 mix_2)^T R + (mix_2^T out_1) y_1^T + out_2 y_2^T

and what the feed-forward reads can be had from the layer's old R: (mix_1 in_2)^T R + (in_2 . out_1) y_1^T,

so that a layer passes over the streams twice (once reading, once reading and writing) instead of reading and writing them
for every sublayer.  Both passes are one kernel (``ops.stream_step``), which also adds a token's expert rows up, applies
the weights of a mixer made of mixers and norms what the next sublayer reads.  The products of constants are worked out
in 64 bits when the weights are loaded and rounded once to 32.
"""
from __future__ import annotations

import torch

from ..kernels import ops
from ..weights.loader import TensorDecl
from .base import Block, Norm, build_part, register_part


def _floats(t: torch.Tensor) -> list:
    return t.to(torch.float32).tolist()


class StreamNorm(Norm):
    """norm(in^T R) of rows [T, streams * size]; ``in_name`` None: the plain sum."""

    graph_safe = True

    def __init__(self, spec):
        super().__init__(spec)
        if not 1 <= spec.streams <= ops.MAX_STREAMS:
            raise ValueError(f"streams={spec.streams}: between 1 and {ops.MAX_STREAMS}")
        self.norm = build_part(spec.norm)

    def tensor_decls(self):
        d = self.norm.tensor_decls()
        if self.spec.in_name:
            d.append(TensorDecl(self.spec.in_name, (self.spec.streams,), mean=1.0 / self.spec.streams))
        return d

    def load(self, src, rt):
        super().load(src, rt)
        self.norm.load(src, rt)
        if self.norm.as_rms() is None:
            raise ValueError("streams are read through an RMS norm")
        s = self.spec.streams
        self.reads = (src.get(self.spec.in_name).to("cpu", torch.float64) if self.spec.in_name
                      else torch.ones(s, dtype=torch.float64))

    def reading(self, n_rows, weights=None):
        """What ``ops.stream_step`` takes as ``read``: the weights of the streams (this norm's own unless given), the
        norm's, and a new output of ``n_rows`` rows."""
        w, eps = self.norm.as_rms()
        return _floats(self.reads if weights is None else weights), w, eps, self.rt.empty(n_rows, self.spec.norm.size)

    def forward(self, h, rows=None):
        n = h.shape[0] if rows is None else rows.numel()
        return ops.stream_step(h, self.spec.streams, read=self.reading(n), rows=rows)


class HyperBlock(Block):
    passes_norm = True

    def __init__(self, spec):
        super().__init__(spec)
        self.norm1 = build_part(spec.norm1)
        self.mixer = build_part(spec.mixer)
        self.ffn = build_part(spec.ffn) if spec.ffn is not None else None
        self.norm2 = build_part(spec.norm2) if self.ffn is not None else None
        self.n_sub = 1 if self.ffn is None else 2
        if len(spec.connections) != self.n_sub:
            raise ValueError("hyper_connections: one pair of tensors a sublayer")

    def _parts(self):
        return [p for p in (self.norm1, self.mixer, self.norm2, self.ffn) if p is not None]

    @property
    def graph_safe(self):
        return all(p.graph_safe for p in self._parts())

    def tensor_decls(self):
        s = self.spec.streams
        d = [x for p in self._parts() for x in p.tensor_decls()]
        for mix, out in self.spec.connections:
            d += [TensorDecl(mix, (s, s), init="identity"), TensorDecl(out, (s,), mean=1.0)]
        return d + [TensorDecl(n, tuple(shape), optional=True) for n, shape in self.spec.unused_tensors]

    def load(self, src, rt):
        super().load(src, rt)
        for p in self._parts():
            p.load(src, rt)
        get = lambda name: src.get(name).to("cpu", torch.float64)
        (m1, o1) = (get(n) for n in self.spec.connections[0])
        if self.ffn is None:
            self.mix, self.out1 = _floats(m1), _floats(o1)
            return
        (m2, o2) = (get(n) for n in self.spec.connections[1])
        in2 = self.norm2.reads
        self.mid_reads = m1 @ in2                          # what the feed-forward reads of the layer's old streams
        self.mid_result = _floats((in2 @ o1).reshape(1))   # and of the mixer's result
        self.mix, self.out1, self.out2 = _floats(m1 @ m2), _floats(o1 @ m2), _floats(o2)

    def reset_after_fault(self):
        for p in self._parts():
            p.reset_after_fault()

    def _mixer_results(self, x, batch, cache):
        """[(32-bit rows, their weight)]: more than one where the mixer is made of mixers."""
        if hasattr(self.mixer, "forward_parts"):
            outs = self.mixer.forward_parts(x, batch, cache)
            if len(outs) <= 2:
                return outs
        y = self.rt.empty(x.shape[0], x.shape[1], dtype=torch.float32)
        if hasattr(self.mixer, "forward_parts"):      # more parts than the kernel takes: added up first
            y.zero_()
            for part, scale in outs:
                ops.scaled_add_norm(y, part, scale, stream=batch.stream)
        else:
            self.mixer.forward_into(x, y, batch, cache, accumulate=False)
        return [(y, 1.0)]

    def forward(self, h, batch, cache, x=None, then_norm=None):
        S, T, st = self.spec.streams, h.shape[0], batch.stream
        if x is None:
            with ops.trace_scope("norm"):
                x = self.norm1.forward(h)
        with ops.trace_scope("mixer"):
            outs = self._mixer_results(x, batch, cache)
        weigh = lambda c: [(y, [scale * v for v in c]) for y, scale in outs]
        experts = None
        terms = weigh(self.out1)
        if self.ffn is not None:
            with ops.trace_scope("norm"):
                x2 = ops.stream_step(h, S, terms=weigh(self.mid_result), read=self.norm2.reading(T, self.mid_reads), stream=st)
            with ops.trace_scope("feed-forward"):
                if self.ffn.gives_rows:
                    experts = (self.ffn.expert_rows(x2, batch), self.out2)
                else:
                    y2 = self.rt.empty(T, x2.shape[1], dtype=torch.float32)
                    self.ffn.forward_into(x2, y2, batch, accumulate=False)
                    terms = terms + [(y2, self.out2)]
        with ops.trace_scope("norm"):
            read = then_norm.reading(T) if isinstance(then_norm, StreamNorm) else None
            return ops.stream_step(h, S, terms=terms, experts=experts, mix=self.mix, read=read, stream=st)


register_part("stream_norm", StreamNorm, replace=True)
register_part("hyper_connections", HyperBlock, replace=True)
