"""Two mixers side by side that read the same input: left_scale * left(h) + right_scale * right(h).

Each side keeps what it keeps under its own name in the layer's cache (`CacheNeeds.named`), and sees
the cache through that name (`LayerCache.scoped`); at most one side asks for pages. Where both sides can
take their inputs from a product made for both (`input_names`, `forward_stacked`), the layer is one stacked
product for all roles of both sides, the sides' own steps, which leave their scaled results side by side in
one row, and one output product over both. Elsewhere each side runs its own products and the weighted sum is
one kernel in 32-bit; a side whose output product has a bias that it can leave to its caller
(`forward_unbiased` and `out_bias`) has it added there. Where each side's result is normed before the sum
(`left_norm`, `right_norm`) the sides have an output product each, and what they give is a `kernels.NormedSum`: the
kernel that adds it to the residual streams norms both on the way in.
"""
from __future__ import annotations

import torch

from .. import kernels as K
from .base import Part, linear, matrix_for, pad_columns, stack_rows
from .registry import build_part, part_class


class ParallelMixer(Part):
    @staticmethod
    def expected_tensors(spec):
        out = {}
        for side in (spec.left, spec.right):
            out.update(part_class("mixer", side.kind).expected_tensors(side))
        for n in (spec.left_norm, spec.right_norm):
            if n is not None:
                out[n.weight] = (n.width,)
        return out

    def __init__(self, spec, ctx):
        super().__init__(spec, ctx)
        self.left = build_part("mixer", spec.left, ctx)
        self.right = build_part("mixer", spec.right, ctx)
        names = [side.input_names() if hasattr(side, "input_names") else None for side in (self.left, self.right)]
        self.names = names if all(n is not None for n in names) else None      # one product for both sides
        self.normed = spec.left_norm is not None
        norms = [n for n in (spec.left_norm, spec.right_norm) if n is not None]
        if len(norms) == 1 or any(n.kind != "rms" or n.width != spec.left.hidden or n.eps != norms[0].eps for n in norms):
            raise ValueError("parallel: the sides' results are normed both or not at all, by RMS norms over the model's width with one eps")
        self.cache_needs()                      # refuses two sides that both want pages

    @property
    def graph_safe(self) -> bool:
        return self.left.graph_safe and self.right.graph_safe

    def load_shared(self, tensors):
        expected = self.expected_tensors(self.spec)
        self.w_in = stack_rows(self.ctx, tensors, self.names[0] + self.names[1], "parallel")
        self.right_base = sum(expected[n][0] for n in self.names[0])
        out = [matrix_for(self.ctx, tensors[side.weights["o"]]) for side in (self.spec.left, self.spec.right)]
        if self.normed:
            self.w_left, self.w_right = (pad_columns(self.ctx, w) for w in out)
        else:
            self.w_o = pad_columns(self.ctx, torch.cat(out, dim=1).contiguous())
        self.left.load_shared(tensors)
        self.right.load_shared(tensors)

    def load(self, tensors):
        if self.normed:
            weights = ((tensors[n.weight].to(self.ctx.device).float() + n.offset) * float(scale)
                       for n, scale in ((self.spec.left_norm, self.spec.left_scale), (self.spec.right_norm, self.spec.right_scale)))
            self.norm_left, self.norm_right = (w.contiguous() for w in weights)
        if self.names is not None:
            return self.load_shared(tensors)
        self.left.load(tensors)
        self.right.load(tensors)
        s, dev = self.spec, self.ctx.device
        width = s.left.hidden
        self.va = torch.full((width,), float(s.left_scale), dtype=torch.float32, device=dev)
        self.vb = torch.full((width,), float(s.right_scale), dtype=torch.float32, device=dev)
        self.vc = None
        for side, scale in ((self.left, s.left_scale), (self.right, s.right_scale)):
            bias = getattr(side, "out_bias", None) if hasattr(side, "forward_unbiased") else None
            if bias is not None:
                self.vc = bias.float() * float(scale) + (self.vc if self.vc is not None else 0.0)
        if self.vc is not None:
            self.vc = self.vc.contiguous()

    def cache_needs(self):
        return self.left.cache_needs().named("left").merged(self.right.cache_needs().named("right"))

    def forward_shared(self, h, batch, cache):
        s, split = self.spec, self.left.inner_width
        stacked = linear(self.ctx, h, self.w_in, out_dtype=torch.float32, keep_split=True)
        if self.normed:
            left = self.left.forward_stacked(stacked, 0, batch, cache.scoped("left"))
            right = self.right.forward_stacked(stacked, self.right_base, batch, cache.scoped("right"))
            return self.normed_sum(linear(self.ctx, left, self.w_left, out_dtype=torch.float32, keep_split=True),
                                   linear(self.ctx, right, self.w_right, out_dtype=torch.float32, keep_split=True))
        both = K.new((h.shape[0], self.w_o.shape[1]), self.ctx.dtype, h.device)
        self.left.forward_stacked(stacked, 0, batch, cache.scoped("left"), out=both, column=0, pad_to=split, scale=s.left_scale)
        self.right.forward_stacked(stacked, self.right_base, batch, cache.scoped("right"), out=both, column=split,
                                   pad_to=self.w_o.shape[1] - split, scale=s.right_scale)
        return linear(self.ctx, both, self.w_o, keep_split=True)

    def normed_sum(self, left, right):
        return K.NormedSum(left, self.norm_left, right, self.norm_right, self.spec.left_norm.eps)

    def forward(self, h, batch, cache):
        if self.names is not None:
            return self.forward_shared(h, batch, cache)
        if self.normed:
            return self.normed_sum(*(K.finish(side.forward(h, batch, cache.scoped(name)), torch.float32)
                                     for side, name in ((self.left, "left"), (self.right, "right"))))
        run = lambda side, name: (side.forward_unbiased if hasattr(side, "forward_unbiased") else side.forward)(h, batch, cache.scoped(name))
        return K.weighted_sum2(run(self.left, "left"), self.va, run(self.right, "right"), self.vb, self.vc)
