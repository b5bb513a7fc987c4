"""Linear attention with a fixed decay a head (retention) as a mixer with a state of its own.

One stacked product gives q | k | v | g in 32-bit. The scan's kernels apply the activation, turn q and k, scale k
and walk each request's rows in order from the memory its slot holds: S <- decay S + k v^T, o = S^T q. Then each head's
read-out (or all heads' together, times a weight) is divided by its root mean square, times silu or sigmoid of g, and the
output product follows. Prompt portions
and single tokens take the same kernels. A caller that runs two mixers over one product may take the steps
between the products alone (`input_names`, `forward_stacked`).
"""
from __future__ import annotations

import torch

from .. import kernels as K
from ..cache import CacheNeeds, StateSpec
from .base import Part, linear, matrix_named, pad_columns, product_width, stack_rows
from .registry import build_part


class Retention(Part):
    graph_safe = True

    @staticmethod
    def expected_tensors(spec):
        w, nq, nv = spec.weights, spec.num_heads * spec.head_dim, spec.num_heads * spec.v_head_dim
        out = {w["q"]: (nq, spec.hidden), w["k"]: (nq, spec.hidden), w["v"]: (nv, spec.hidden), w["g"]: (nv, spec.hidden),
               w["o"]: (spec.hidden, nv)}
        if spec.whole_norm:
            out[w["norm"]] = (nv,)
        return out

    def __init__(self, spec, ctx):
        super().__init__(spec, ctx)
        if spec.head_dim > 256:
            raise ValueError(f"retention: a key size of {spec.head_dim} is more than the scan kernel's 256")
        if len(spec.decay) != spec.num_heads:
            raise ValueError(f"retention: {len(spec.decay)} decays for {spec.num_heads} heads")
        if spec.activation not in K.RETENTION_ACTS or spec.gate not in ("silu", "sigmoid"):
            raise ValueError(f"retention: activation {spec.activation!r}, gate {spec.gate!r} are not built")
        self.position = build_part("position", spec.position, ctx)
        if getattr(self.position, "neighbours", False):
            raise ValueError("retention: the rotation of neighbouring components is not built")

    def input_names(self):
        """The weights whose rows make up the stacked product, in order."""
        return [self.spec.weights[r] for r in ("q", "k", "v", "g")]

    def load_shared(self, tensors):
        """`load` without the two products' weights, for a caller that multiplies by them (`forward_stacked`)."""
        self.decay = torch.tensor(self.spec.decay, dtype=torch.float32, device=self.ctx.device)
        self.norm_weight = tensors[self.spec.weights["norm"]].to(self.ctx.device).float().contiguous() if self.spec.whole_norm else None

    def load(self, tensors):
        self.w_in = stack_rows(self.ctx, tensors, self.input_names(), "retention")
        self.w_o = pad_columns(self.ctx, matrix_named(self.ctx, tensors, self.spec.weights["o"]))      # the gate kernel writes rows this wide
        self.load_shared(tensors)

    def cache_needs(self) -> CacheNeeds:
        s = self.spec
        return CacheNeeds(state=StateSpec((s.num_heads * s.head_dim * s.v_head_dim,)))

    @property
    def inner_width(self) -> int:
        return self.spec.num_heads * self.spec.v_head_dim

    def forward_stacked(self, stacked, base: int, batch, cache, out=None, column: int = 0, pad_to=None, scale: float = 1.0):
        """The output product's input [rows, heads x value size] from the columns `base`.. of a stacked product; with
        `out`, times `scale` and written to its columns from `column` on, zeros up to `column` + `pad_to`."""
        s = self.spec
        nq, nv = s.num_heads * s.head_dim, self.inner_width
        rotary = self.position.rotary_dim
        o = K.retention_scan(stacked, base, base + nq, base + 2 * nq, self.decay, self.position.tables(batch) if rotary else None, rotary,
                             s.head_dim ** -0.5 if s.key_scale is None else s.key_scale, cache.state(), batch.entry_ranges(), batch.slots,
                             batch.entries, batch.longest_portion(), s.num_heads, s.head_dim, s.v_head_dim, act=s.activation)
        if s.whole_norm:                                     # the heads' read-outs are one vector to the norm
            o = o.view(o.shape[0], 1, nv)
        return K.head_gate(o, stacked, base + 2 * nq + nv, self.norm_weight, True, s.eps, self.ctx.dtype, gate_act=s.gate, scale=scale, out=out, column=column,
                           pad_to=product_width(self.ctx, nv) if pad_to is None else pad_to)

    def forward(self, h, batch, cache):
        stacked = linear(self.ctx, h, self.w_in, out_dtype=torch.float32, keep_split=True)
        return linear(self.ctx, self.forward_stacked(stacked, 0, batch, cache), self.w_o, keep_split=True)
