"""A layer over several residual streams (hyper-connections).

x is float32 [rows, streams x hidden], a row's streams side by side. A sublayer reads u = sum_s in[s] x_s
through its norm; its result y, times a weight a channel where the layer has one, goes back into all streams at once:
x_t <- sum_s mix[s, t] x_s + out[t] y. Writing a sublayer's result and reading the next one's input (this
layer's feed-forward or the next layer's mixer) is one kernel.
"""
from __future__ import annotations

from .. import kernels as K
from .base import Part
from .registry import build_part


class StreamRead:
    """What a sublayer reads: norm(sum_s in[s] x_s). Takes a norm's place between two layers (`Block.first_norm`)."""

    def __init__(self, ctx, norm, count: int):
        self.ctx, self.norm, self.count = ctx, norm, count
        if not hasattr(norm, "wide_key"):
            raise ValueError("streams block: the norms must be RMS or layer norms")

    def load(self, w_in):
        self.key = (w_in, *self.norm.wide_key())

    def forward(self, x):
        return K.stream_step(x, self.count, None, self.key, self.ctx.dtype)


class StreamBlock(Part):
    @staticmethod
    def _sublayers(spec):
        """(norm's role, the streams' tensors, the branch weight's name or None) of every sublayer."""
        scales = spec.scales or (None, None)
        out = [("pre_mixer", spec.streams[0], scales[0])]
        if spec.ffn is not None:
            out.append(("pre_ffn", spec.streams[1], scales[1]))
        return out

    @classmethod
    def expected_tensors(cls, spec):
        from .registry import part_class

        out = {}
        out.update(part_class("mixer", spec.mixer.kind).expected_tensors(spec.mixer))
        if spec.ffn is not None:
            out.update(part_class("feed_forward", spec.ffn.kind).expected_tensors(spec.ffn))
        for role, st, scale in cls._sublayers(spec):
            n = spec.norms[role]
            out.update(part_class("norm", n.kind).expected_tensors(n))
            out[st.read], out[st.write], out[st.mix] = (st.count,), (st.count,), (st.count, st.count)
            if scale is not None:
                out[scale] = (n.width,)
        return out

    def __init__(self, spec, ctx):
        super().__init__(spec, ctx)
        if spec.streams is None or spec.streams[0] is None or (spec.ffn is not None and spec.streams[1] is None):
            raise ValueError("streams block: a sublayer does not say how it reads and writes the streams")
        self.sublayers = self._sublayers(spec)
        self.count = spec.streams[0].count
        if any(st.count != self.count or st.count < 1 for _, st, _ in self.sublayers):
            raise ValueError(f"streams block: sublayers of {[st.count for _, st, _ in self.sublayers]} streams")
        self.mixer = build_part("mixer", spec.mixer, ctx)
        self.ffn = build_part("feed_forward", spec.ffn, ctx) if spec.ffn is not None else None
        self.norms = [build_part("norm", spec.norms[role], ctx) for role, _, _ in self.sublayers]
        self.reads = [StreamRead(ctx, n, self.count) for n in self.norms]

    @property
    def graph_safe(self) -> bool:
        parts = [self.mixer, *self.norms] + ([self.ffn] if self.ffn is not None else [])
        return all(p.graph_safe for p in parts)

    def cache_needs(self):
        return self.mixer.cache_needs()

    def first_norm(self):
        return self.reads[0]

    def load(self, tensors):
        self.mixer.load(tensors)
        if self.ffn is not None:
            self.ffn.load(tensors)
        f32 = lambda name: tensors[name].to(self.ctx.device).float().contiguous()
        self.writes = []
        for norm, read, (_, st, scale) in zip(self.norms, self.reads, self.sublayers):
            norm.load(tensors)
            read.load(f32(st.read))
            self.writes.append((f32(scale) if scale is not None else None, f32(st.mix), f32(st.write)))

    def _add(self, x, i: int, branch, following):
        """Writes sublayer i's result into the streams; returns what `following` reads, if it reads streams."""
        fused = isinstance(following, StreamRead)
        return K.stream_step(x, self.count, (branch, *self.writes[i]), following.key if fused else None, self.ctx.dtype)

    def forward(self, x, h, batch, cache, next_norm):
        if h is None:
            h = self.reads[0].forward(x)
        a = self.mixer.forward(h, batch, cache)
        if self.ffn is None:
            return x, self._add(x, 0, a, next_norm)
        h = self._add(x, 0, a, self.reads[1])
        return x, self._add(x, 1, self.ffn.forward(h), next_norm)
