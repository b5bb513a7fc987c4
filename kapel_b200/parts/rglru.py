"""A real-gated linear recurrent unit between two branches (Griffin's recurrent block) as a mixer with a
state of its own.

One stacked product gives y | x in 32-bit. A kernel convolves x per channel over the last rows (the rows
before this step come from the request's slot), one makes both gates (a square matrix a part of the
channels, in true 32-bit) and from them what every row does to the state, and one walks each request's rows,
times gelu of the other branch; then the output product. A prompt portion's rows are walked as runs side by
side, a few rows one after the other: the same steps, composed in another order.
"""
from __future__ import annotations

import torch

from .. import kernels as K
from ..cache import CacheNeeds, StateSpec
from .base import Part, linear, matrix_for, matrix_named, pad_columns, product_width, stack_rows


class RGLRU(Part):
    graph_safe = True

    @staticmethod
    def expected_tensors(spec):
        w, n, part = spec.weights, spec.width, spec.width // spec.blocks
        return {w["y"]: (n, spec.hidden), w["y_bias"]: (n,), w["x"]: (n, spec.hidden), w["x_bias"]: (n,),
                w["conv"]: (n, spec.conv), w["conv_bias"]: (n,),
                w["ra"]: (spec.blocks, part, part), w["ra_bias"]: (spec.blocks, part),
                w["ri"]: (spec.blocks, part, part), w["ri_bias"]: (spec.blocks, part),
                w["lam"]: (n,), w["o"]: (spec.hidden, n)}

    def __init__(self, spec, ctx):
        super().__init__(spec, ctx)
        if spec.width % spec.blocks:
            raise ValueError(f"rglru: {spec.width} channels in {spec.blocks} parts")
        if not 1 <= spec.conv <= 16:
            raise ValueError(f"rglru: a convolution over {spec.conv} rows (1 to 16)")

    def load(self, tensors):
        w, dev = self.spec.weights, self.ctx.device
        self.w_in = stack_rows(self.ctx, tensors, [w["y"], w["x"]], "rglru")
        self.w_o = pad_columns(self.ctx, matrix_named(self.ctx, tensors, w["o"]))      # the scan's kernel writes rows this wide
        f32 = lambda name: tensors[name].to(dev).float().reshape(-1).contiguous()
        self.y_bias, self.x_bias, self.conv_bias, self.ra_bias, self.ri_bias, self.lam = (
            f32(w[r]) for r in ("y_bias", "x_bias", "conv_bias", "ra_bias", "ri_bias", "lam"))
        self.conv = tensors[w["conv"]].to(dev).float().contiguous()
        self.ra, self.ri = (matrix_for(self.ctx, tensors[w[r]]) for r in ("ra", "ri"))

    def cache_needs(self) -> CacheNeeds:
        s = self.spec
        return CacheNeeds(state=StateSpec((s.width,)), states=(("conv", StateSpec((K.conv_history_floats(s.width, s.conv),))),))

    def forward(self, h, batch, cache):
        s = self.spec
        stacked = linear(self.ctx, h, self.w_in, out_dtype=torch.float32, keep_split=True)
        ranges = batch.entry_ranges()
        u = K.conv_rows(stacked, s.width, s.width, self.x_bias, self.conv, self.conv_bias, cache.state_of("conv"), batch.row_entry, ranges,
                        batch.slots, batch.entries, s.conv)
        ab = K.lru_gates(u, self.ra, self.ri, self.ra_bias, self.ri_bias, self.lam, s.rate)
        y = K.lru_scan(ab, stacked, 0, self.y_bias, cache.state(), ranges, batch.slots, batch.entries, batch.longest_portion(), self.ctx.dtype,
                       pad_to=product_width(self.ctx, s.width))
        return linear(self.ctx, y, self.w_o, keep_split=True)
