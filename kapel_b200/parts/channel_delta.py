"""The gated delta rule with a decay a head and key channel, as a mixer with a state of its own.

One stacked product gives q | k | v | b | a1 | g1 in 32-bit (b: a column a head; a1 and g1: the first
factors of the decay's and the output gate's low-rank projections). The scan's kernels convolve q, k and v
over the last rows per channel (the rows before this step come from the request's slot), apply silu, make q
and k unit vectors, finish the decay (a2, softplus, the exponentials) and the step size, and walk each
request's rows in order from the memory its slot holds. The output gate's second factor is a small product
of its own. Then each head's read-out is divided by its root mean square, times a weight shared by the heads,
times sigmoid of the gate, and the output product follows. Prompt portions and single tokens take the same
kernels.
"""
from __future__ import annotations

import torch

from .. import kernels as K
from ..cache import CacheNeeds, StateSpec
from .base import Part, linear, matrix_named, pad_columns, product_width, stack_rows


class ChannelDelta(Part):
    graph_safe = True

    @staticmethod
    def expected_tensors(spec):
        w = spec.weights
        kd, n, he = spec.num_kv_heads * spec.head_dim, spec.num_heads * spec.head_dim, spec.num_heads * spec.v_head_dim
        return {
            w["q"]: (kd, spec.hidden), w["k"]: (kd, spec.hidden), w["v"]: (he, spec.hidden),
            w["q_conv"]: (kd, spec.conv), w["k_conv"]: (kd, spec.conv), w["v_conv"]: (he, spec.conv),
            w["b"]: (spec.num_heads, spec.hidden), w["A_log"]: (spec.num_heads,), w["norm"]: (spec.v_head_dim,),
            w["a1"]: (spec.decay_rank, spec.hidden), w["a2"]: (n, spec.decay_rank), w["dt_bias"]: (n,),
            w["g1"]: (spec.gate_rank, spec.hidden), w["g2"]: (he, spec.gate_rank), w["o"]: (spec.hidden, he),
        }

    def __init__(self, spec, ctx):
        super().__init__(spec, ctx)
        if spec.num_heads % spec.num_kv_heads:
            raise ValueError(f"channel_delta: {spec.num_heads} heads over {spec.num_kv_heads} key heads")
        if spec.head_dim > 256:
            raise ValueError(f"channel_delta: a key size of {spec.head_dim} is more than the scan kernel's 256")
        if not 1 <= spec.conv <= 16:
            raise ValueError(f"channel_delta: a convolution over {spec.conv} rows (1 to 16)")
        self.channels = 2 * spec.num_kv_heads * spec.head_dim + spec.num_heads * spec.v_head_dim

    def load(self, tensors):
        s, w, dev = self.spec, self.spec.weights, self.ctx.device
        self.w_in = stack_rows(self.ctx, tensors, [w[r] for r in ("q", "k", "v", "b", "a1", "g1")], "channel_delta")
        self.w_o = pad_columns(self.ctx, matrix_named(self.ctx, tensors, w["o"]))      # the gate kernel writes rows this wide
        self.w_gate = pad_columns(self.ctx, matrix_named(self.ctx, tensors, w["g2"]))
        f32 = lambda n: tensors[n].to(dev).float().contiguous()
        self.conv = torch.cat([f32(w["q_conv"]), f32(w["k_conv"]), f32(w["v_conv"])], dim=0).contiguous()
        self.a_log, self.dt_bias = f32(w["A_log"]), f32(w["dt_bias"])
        self.a2 = f32(w["a2"]).t().contiguous()                                         # turned: [rank, heads d]
        n = tensors[w["norm"]].to(dev)
        n = n.float() if self.ctx.is_f32 else n
        self.norm_weight = n.repeat(s.num_heads).contiguous()                           # one weight for all heads

    def cache_needs(self) -> CacheNeeds:
        s = self.spec
        return CacheNeeds(state=StateSpec((s.num_heads * s.head_dim * s.v_head_dim,)),
                          states=(("conv", StateSpec((K.conv_history_floats(self.channels, s.conv),))),))

    def forward(self, h, batch, cache):
        s = self.spec
        he = s.num_heads * s.v_head_dim
        b_off, a1_off = self.channels, self.channels + s.num_heads
        stacked = linear(self.ctx, h, self.w_in, out_dtype=torch.float32, keep_split=True)
        o = K.cdelta_scan(stacked, 0, b_off, a1_off, self.a2, self.dt_bias, self.a_log, self.conv, cache.state_of("conv"), cache.state(),
                          batch.row_entry, batch.entry_ranges(), batch.slots, batch.entries, s.num_heads, s.num_kv_heads, s.head_dim,
                          s.v_head_dim, s.conv, s.head_dim ** -0.5, s.unit_eps)
        low = K.take_cols(stacked, a1_off + s.decay_rank, s.gate_rank, self.w_gate.dtype, self.w_gate.shape[1])
        gate = linear(self.ctx, low, self.w_gate, out_dtype=torch.float32, keep_split=True)
        y = K.head_gate(o, gate, 0, self.norm_weight, True, s.eps, self.ctx.dtype, pad_to=product_width(self.ctx, he))
        return linear(self.ctx, y, self.w_o, keep_split=True)
