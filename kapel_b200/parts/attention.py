"""Grouped-query attention over the paged cache.

q, k, v come from one stacked product (Kapel stacks them at load: crates/kapel-models/src/model.rs:415-480,
1506-1517); one kernel rotates q and k and appends k and v to the cache at the rows' lines
(Kapel: rope_any twice and write_rows_any twice, model.rs:1561-1579); attention reads the pages
through the block table with scale, soft cap and window as arguments (model.rs:1580-1590);
then the output product (model.rs:1633-1637).

A spec may ask for more than that: a norm over the whole query and key projections, values of
another size than keys, first keys that stay visible below the window, a sigmoid gate on the
heads' outputs, a sink (learned, or 1 in the denominator) beside norms over the projection, keys and values that
are another layer's. Such a layer runs the general path: one stacked product q|k|v|g in 32-bit (q|g where
the keys are another layer's), one kernel that norms q and k, turns them (either pairing) and appends k and v to the
cache, the tensor-core kernels where keys and values have one size and no first keys are kept (else the row-wise
kernel), the gate, the output product.

A spec with an RMS norm over every head's query and key (`q_head_norm`, `k_head_norm`: one weight
of the head's size for all heads), a sink in the softmax's denominator or one gate a head runs the third
path: the stacked product in 32-bit, one kernel that norms each head, rotates it and appends keys and
values (of their own size) to the cache, then the tensor-core kernels where keys and values have one size
and the row-wise kernel elsewhere, the gate, the output product. A caller that runs two mixers over one
product may take this path in two steps (`input_names`, `forward_stacked`).

A spec with biases, pooled blocks below the window, a number a head on the scores, mixed heads'
weights or values mixed with another layer's runs the fourth path (`forward_pooled`): the stacked
product in 32-bit; one kernel for biases, the norms over the whole projections, the rotation (either
pairing), the value mix and the append; one that leaves the means of every block the step completes
in the request's slot of the layer's state table; then the attention kernel over window and blocks.

A spec with short convolutions on queries and keys whose values are its keys runs the fifth path
(`forward_convolved`): the stacked product q|k in 32-bit; one kernel that adds the biases, convolves every
channel over the last rows (the rows before the step from the request's state) and appends the keys, which
are also the values (one table); the row-wise attention kernel with the block mask and 1 in the
denominator; the output product, whose bias the caller may add (`forward_unbiased`, `out_bias`).
"""
from __future__ import annotations

import torch

from .. import kernels as K
from ..cache import CacheNeeds, PagedKV, StateSpec
from .base import Part, linear, matrix_named, pad_columns, product_width, require_product_widths, stack_rows
from .registry import build_part


class Attention(Part):
    graph_safe = True

    @staticmethod
    def expected_tensors(spec):
        dv = spec.v_head_dim or spec.head_dim
        qd, kvd = spec.num_heads * spec.head_dim, spec.num_kv_heads * spec.head_dim
        w = spec.weights
        if spec.values_are_keys:
            out = {w["q"]: (qd, spec.hidden), w["k"]: (kvd, spec.hidden), w["o"]: (spec.hidden, qd)}
            if spec.conv:
                out[w["q_conv"]], out[w["k_conv"]] = (qd, spec.conv), (kvd, spec.conv)
            if spec.qk_bias:
                out[w["q_bias"]], out[w["k_bias"]] = (qd,), (kvd,)
            if spec.out_bias:
                out[w["o_bias"]] = (spec.hidden,)
            return out
        out = {w["q"]: (qd, spec.hidden), w["o"]: (spec.hidden, spec.num_heads * dv)}
        if not spec.borrows_kv:
            out[w["k"]], out[w["v"]] = (kvd, spec.hidden), (spec.num_kv_heads * dv, spec.hidden)
        if spec.gated:
            out[w["g"]] = (spec.num_heads if spec.gate_by_head else spec.num_heads * dv, spec.hidden)
        if spec.sink:
            out[w["sink"]] = (spec.num_heads,)
        for n in (spec.q_norm, spec.k_norm, spec.q_head_norm, spec.k_head_norm):
            if n is not None:
                out[n.weight] = (n.width,)
        if spec.bias:
            out[w["q_bias"]], out[w["k_bias"]], out[w["v_bias"]] = (qd,), (kvd,), (spec.num_kv_heads * dv,)
        if spec.head_temp:
            out[w["temp"]] = (spec.num_heads,)
        if spec.talk:
            out[w["talk"]] = (spec.num_heads, spec.num_heads)
        if spec.value_mix == "mix":
            out[w["vmix"]] = ()
        return out

    def __init__(self, spec, ctx):
        super().__init__(spec, ctx)
        if spec.num_heads % spec.num_kv_heads:
            raise ValueError(f"attention: {spec.num_heads} heads over {spec.num_kv_heads} kv heads")
        self.v_dim = spec.v_head_dim or spec.head_dim
        self.by_head = bool(spec.q_head_norm or spec.k_head_norm or spec.gate_by_head
                            or (spec.sink and not (spec.q_norm or spec.k_norm or spec.borrows_kv)))
        if spec.gate_by_head and not spec.gated:
            raise ValueError("attention: one gate a head for a layer without a gate")
        self.convolved = bool(spec.conv or spec.values_are_keys or spec.block_mask or spec.qk_bias or spec.out_bias)
        self.out_bias = None
        if self.convolved:
            if not (spec.values_are_keys and 1 <= spec.conv <= 16):
                raise ValueError("attention: a block mask or biases on q, k and o are built for the path with "
                                 f"convolutions (1 to 16 rows, got {spec.conv}) whose values are its keys")
            if (self.by_head or spec.borrows_kv or spec.gated or spec.q_norm or spec.k_norm or spec.keep_first or spec.softcap or spec.window or spec.bias
                    or spec.pool or spec.head_temp or spec.talk or spec.value_mix or spec.v_head_dim not in (None, spec.head_dim)):
                raise ValueError("attention: convolutions together with norms, a sink, a gate, a window, a soft cap, pooled blocks, mixed heads or "
                                 "values of their own are not built")
            if spec.block_mask < 0:
                raise ValueError(f"attention: blocks of {spec.block_mask} positions")
        self.pooled = bool(spec.bias or spec.pool or spec.head_temp or spec.talk or spec.value_mix)
        if self.pooled:
            if self.by_head or spec.sink or spec.unit_sink or spec.borrows_kv or spec.gated or spec.keep_first or spec.softcap:
                raise ValueError("attention: biases, pooled blocks, head temperatures, mixed heads or mixed values together with norms "
                                 "over each head, a sink, a gate, kept first keys or a soft cap are not built")
            if spec.pool and (not spec.window or spec.pool_blocks <= 0):
                raise ValueError(f"attention: blocks of {spec.pool} need a window (got {spec.window}) and a count of blocks (got {spec.pool_blocks})")
            if spec.value_mix not in (None, "source", "mix"):
                raise ValueError(f"attention: value_mix {spec.value_mix!r} is not known (\"source\", \"mix\")")
        self.general = bool(spec.gated or spec.q_norm or spec.k_norm or spec.keep_first or self.v_dim != spec.head_dim or spec.borrows_kv
                            or spec.unit_sink) and not self.by_head and not self.pooled and not self.convolved
        if self.by_head and (spec.q_norm or spec.k_norm or spec.keep_first or spec.borrows_kv):
            raise ValueError("attention: norms over each head or one gate a head together with norms over the whole projection, another layer's "
                             "keys or kept first keys are not built")
        if spec.sink and spec.unit_sink:
            raise ValueError("attention: a learned sink and 1 in the denominator exclude one another")
        if (spec.sink or spec.unit_sink) and spec.keep_first:
            raise ValueError("attention: a sink together with kept first keys is not built")
        if spec.borrows_kv and spec.k_norm:
            raise ValueError("attention: a layer that takes another layer's keys has no norm of its own on them")
        for n in (spec.q_head_norm, spec.k_head_norm):
            if n is not None and (n.kind != "rms" or n.width != spec.head_dim):
                raise ValueError(f"attention: a norm over each head must be an RMS norm of width {spec.head_dim}")
        if not self.general and not self.by_head and not self.pooled and not self.convolved and spec.head_dim % 16:
            raise ValueError(f"attention: head_dim {spec.head_dim} must be a multiple of 16 for the kernels")
        if spec.keep_first < 0 or (spec.keep_first and not spec.window):
            raise ValueError(f"attention: {spec.keep_first} first keys kept with window {spec.window}")
        for n, width in ((spec.q_norm, spec.num_heads * spec.head_dim), (spec.k_norm, spec.num_kv_heads * spec.head_dim)):
            if n is not None and (n.kind != "rms" or n.width != width):
                raise ValueError(f"attention: a norm over the whole projection must be an RMS norm of width {width}")
        if not self.general and not self.by_head and not self.pooled and not self.convolved:
            require_product_widths(ctx, "attention", hidden_size=spec.hidden,
                                   **{"num_attention_heads x value size": spec.num_heads * self.v_dim})
        self.position = build_part("position", spec.position, ctx)
        if self.convolved and self.position.rotary_dim:
            raise ValueError("attention: a rotation together with convolutions is not built")
        if not self.pooled and not self.general and getattr(self.position, "neighbours", False):
            raise ValueError("attention: the rotation of neighbouring components is built for the paths with biases, pooled blocks, mixed heads, "
                             "norms over the projection or another layer's keys only")

    def load_convolved(self, tensors):
        s, w, dev = self.spec, self.spec.weights, self.ctx.device
        self.w_qkv = stack_rows(self.ctx, tensors, [w["q"], w["k"]], "attention")
        self.w_o = pad_columns(self.ctx, matrix_named(self.ctx, tensors, w["o"]))
        f32 = lambda n: tensors[n].to(dev).float().contiguous()
        self.conv = torch.cat([f32(w["q_conv"]), f32(w["k_conv"])], dim=0).contiguous()
        self.qk_bias = torch.cat([f32(w["q_bias"]), f32(w["k_bias"])]).contiguous() if s.qk_bias else None
        self.out_bias = f32(w["o_bias"]) if s.out_bias else None
        self.ones = torch.ones((s.hidden,), dtype=torch.float32, device=dev) if s.out_bias else None
        self.sinks = torch.zeros((s.num_heads,), dtype=torch.float32, device=dev) if s.unit_sink else None      # e^0 = 1 in the denominator

    def input_names(self):
        """The weights whose rows make up the stacked product, in order; None where the layer cannot share one."""
        w = self.spec.weights
        return [w["q"], w["k"], w["v"]] + ([w["g"]] if self.spec.gated else []) if self.by_head else None

    def load_shared(self, tensors):
        """`load` without the two products' weights, for a caller that multiplies by them (`forward_stacked`)."""
        self.load_sinks(tensors)
        self.load_norms(tensors)

    def load_sinks(self, tensors):
        s = self.spec
        self.sinks = tensors[s.weights["sink"]].to(self.ctx.device).float().contiguous() if s.sink else None
        if s.unit_sink:
            self.sinks = torch.zeros((s.num_heads,), dtype=torch.float32, device=self.ctx.device)       # e^0 = 1 in the denominator

    def load(self, tensors):
        if self.convolved:
            return self.load_convolved(tensors)
        w = self.spec.weights
        names = [w["q"]] + ([] if self.spec.borrows_kv else [w["k"], w["v"]]) + ([w["g"]] if self.spec.gated else [])
        self.w_qkv = stack_rows(self.ctx, tensors, names, "attention")
        self.w_o = matrix_named(self.ctx, tensors, w["o"])
        if self.by_head:
            self.w_o = pad_columns(self.ctx, self.w_o)
            return self.load_shared(tensors)
        if self.general or self.pooled:
            self.w_o = pad_columns(self.ctx, self.w_o)
        if self.general:
            self.load_sinks(tensors)
        if self.pooled:
            dev = self.ctx.device
            small = lambda name: (tensors[name].to(dev).float() if self.ctx.is_f32 else tensors[name].to(dev)).contiguous()
            self.biases = tuple(small(w[r]) for r in ("q_bias", "k_bias", "v_bias")) if self.spec.bias else None
            self.temp = tensors[w["temp"]].to(dev).float().contiguous() if self.spec.head_temp else None
            self.talk = tensors[w["talk"]].to(dev).float().contiguous() if self.spec.talk else None
            self.v_weight = small(w["vmix"]).reshape(1) if self.spec.value_mix == "mix" else None
        self.load_norms(tensors)

    def load_norms(self, tensors):
        self.proj_norms = []
        for n in (self.spec.q_head_norm, self.spec.k_head_norm) if self.by_head else (self.spec.q_norm, self.spec.k_norm):
            if n is None:
                self.proj_norms.append(None)
                continue
            t = tensors[n.weight]
            t = t.to(self.ctx.device) if t.device != self.ctx.device else t
            self.proj_norms.append((t.float() if self.ctx.is_f32 else t.contiguous(), n.eps, n.offset))

    def cache_needs(self) -> CacheNeeds:
        s = self.spec
        if self.convolved:
            # one table: a key is also the value. A block mask gives no pages back (a block's pages stay until the request ends).
            states = (("conv", StateSpec((K.conv_state_floats(s.num_heads, s.num_kv_heads, s.head_dim, s.conv),))),)
            return CacheNeeds(paged=PagedKV(s.num_kv_heads, s.head_dim, None, 0, None, shared_values=True), states=states)
        if self.pooled and s.pool:
            # The pages keep the window's tokens, and a block's tokens until its last one has come (the
            # means are taken from the pages then); the means of a request's blocks are its state.
            kept = max(s.window, s.pool)
            return CacheNeeds(paged=PagedKV(s.num_kv_heads, s.head_dim, kept, 0, self.v_dim if self.v_dim != s.head_dim else None),
                              state=StateSpec((s.pool_blocks, s.num_kv_heads, s.head_dim + self.v_dim)))
        return CacheNeeds(paged=PagedKV(s.num_kv_heads, s.head_dim, s.window, s.keep_first if s.window else 0,
                                        self.v_dim if self.v_dim != s.head_dim else None))

    def forward_pooled(self, h, batch, cache):
        s, dv = self.spec, self.v_dim
        nq, nk = s.num_heads * s.head_dim, s.num_kv_heads * s.head_dim
        stacked = linear(self.ctx, h, self.w_qkv, out_dtype=torch.float32, keep_split=True)
        k_table, v_table = cache.tables()
        group = batch.groups[cache.group]
        rotary = self.position.rotary_dim
        v_other = None
        if s.value_mix == "mix":
            v_other = batch.memo.get(("value_mix", s.value_mix_key))
            if v_other is None:
                raise ValueError(f"attention: values are mixed with those of {s.value_mix_key!r}, which no earlier layer of the step has kept")
        q, kept = K.proj_rope_append(
            stacked, 0, nq, nq + nk, self.biases, self.proj_norms[0], self.proj_norms[1],
            self.position.tables(batch) if rotary else None, rotary, getattr(self.position, "neighbours", False),
            v_other, self.v_weight if v_other is not None else None, s.value_mix == "source", group.lines, k_table, v_table,
            s.num_heads, s.num_kv_heads, s.head_dim, dv, cache.owns, self.ctx.dtype)
        if kept is not None:
            batch.memo[("value_mix", s.value_mix_key)] = kept
        pooled = None
        if s.pool:
            pooled = cache.state()
            if cache.owns:
                K.pool_blocks(k_table, v_table, group.block_table, batch.row_entry, batch.positions, group.lines, batch.slots, pooled, s.pool)
        splits, split_keys = batch.pooled_slices(s.window, s.pool) if hasattr(batch, "pooled_slices") else (1, 0)
        tiles = batch.pooled_tiles() if hasattr(batch, "pooled_tiles") else None
        y = K.pooled_attention(q, k_table, v_table, pooled, group.block_table, batch.row_entry, batch.row_count, batch.slots,
                               self.talk, self.temp, self.ctx.page_size, s.window, s.pool, s.scale, splits, split_keys, tiles,
                               batch.longest_count() if tiles is not None else None)
        width = product_width(self.ctx, s.num_heads * dv)
        y = y.view(y.shape[0], s.num_heads * dv)
        if width != y.shape[1]:
            y = K.pad_cols(y, width)
        return linear(self.ctx, y, self.w_o, keep_split=True)

    def forward_unbiased(self, h, batch, cache):
        """`forward` without the output product's bias (`out_bias`), for a caller that adds it in a kernel of its own."""
        if not self.convolved:
            return self.forward(h, batch, cache)
        s = self.spec
        nq = s.num_heads * s.head_dim
        stacked = linear(self.ctx, h, self.w_qkv, out_dtype=torch.float32, keep_split=True)
        k_table, _ = cache.tables()
        group = batch.groups[cache.group]
        q = K.conv_append(stacked, 0, nq, self.qk_bias, self.conv, cache.state_of("conv"), batch.row_entry, batch.entry_ranges(),
                          batch.slots, batch.entries, group.lines, k_table, s.num_heads, s.num_kv_heads, s.head_dim, s.conv, cache.owns,
                          self.ctx.dtype)
        q = q.view(-1, s.num_heads, s.head_dim)
        heads_per_kv = s.num_heads // s.num_kv_heads
        y = None
        if s.head_dim % 16 == 0 and K.attention_mma_takes(q.dtype, s.head_dim, heads_per_kv):
            # prompt portions go to the tensor-core kernel, which knows the block mask and the sink (in one slot: a row
            # reads at most a block of keys); a pass of single tokens stays with the row-wise kernel below
            decode, tiles, _, _, _ = batch.attention_tiles(heads_per_kv, s.num_kv_heads, None, s.head_dim, "mma", keep_first=0)
            if not decode:
                y = K.paged_attention_mma(q, k_table, k_table, group.block_table, batch.row_count, tiles, self.ctx.page_size, None,
                                          s.scale, None, 0, 0, 1, False, block=s.block_mask, sinks=self.sinks)
        if y is None:
            y = K.paged_attention_rows(q, k_table, k_table, group.block_table, batch.row_entry, batch.row_count, self.ctx.page_size,
                                       None, s.scale, None, batch.attention_slots(s.block_mask or None), sinks=self.sinks,
                                       block=s.block_mask)
        y = y.view(y.shape[0], nq)
        width = product_width(self.ctx, nq)
        if width != nq:
            y = K.pad_cols(y, width)
        return linear(self.ctx, y, self.w_o, keep_split=True)

    def forward_general(self, h, batch, cache):
        s, dv = self.spec, self.v_dim
        own = 0 if s.borrows_kv else s.num_kv_heads         # kv heads whose projections are in the product
        nq, nk = s.num_heads * s.head_dim, own * s.head_dim
        stacked = linear(self.ctx, h, self.w_qkv, out_dtype=torch.float32, keep_split=True)
        k_table, v_table = cache.tables()
        group = batch.groups[cache.group]
        rotary = self.position.rotary_dim
        if rotary or s.borrows_kv:
            q, _ = K.proj_rope_append(
                stacked, 0, nq, nq + nk, None, self.proj_norms[0], self.proj_norms[1], self.position.tables(batch) if rotary else None, rotary,
                getattr(self.position, "neighbours", False), None, None, False, group.lines, k_table, v_table, s.num_heads, own, s.head_dim, dv,
                cache.owns and own > 0, self.ctx.dtype)
        else:
            q = K.proj_norm_append(stacked, 0, nq, nq + nk, self.proj_norms[0], self.proj_norms[1], group.lines, k_table, v_table,
                                   s.num_heads, s.num_kv_heads, s.head_dim, dv, cache.owns, self.ctx.dtype)
        heads_per_kv = s.num_heads // s.num_kv_heads
        keep = s.keep_first if s.window else 0
        y = None
        if dv == s.head_dim and K.attention_mma_takes(q.dtype, s.head_dim, heads_per_kv):
            # with kept first keys only prompt portions go to the tensor-core kernel; a pass of single tokens stays with
            # the row-wise kernel below
            prompt = "mma" if keep or self.sinks is not None else K.attention_prompt_kernel(s.num_heads, s.num_kv_heads, s.head_dim,
                                                                                            self.ctx.page_size, s.softcap)
            decode, tiles, split, slots, relative = batch.attention_tiles(heads_per_kv, s.num_kv_heads, s.window, s.head_dim, prompt, keep_first=keep)
            if not (decode and keep):
                y = K.paged_attention_mma(q, k_table, v_table, group.block_table, batch.row_count, tiles, self.ctx.page_size,
                                          s.window, s.scale, s.softcap, decode, split, slots, relative, pairs=getattr(batch, "pairs", None),
                                          keep_first=keep, sinks=self.sinks)
        if y is None:
            y = K.paged_attention_rows(
                q, k_table, v_table, group.block_table, batch.row_entry, batch.row_count, self.ctx.page_size, s.window, s.scale,
                s.softcap, batch.attention_slots(s.window, s.keep_first), s.keep_first, sinks=self.sinks)
        width = product_width(self.ctx, s.num_heads * dv)
        if s.gated:
            y = K.head_gate(y, stacked, nq + nk + own * dv, None, False, 0.0, self.ctx.dtype, pad_to=width)
            return linear(self.ctx, y, self.w_o, keep_split=True)
        y = y.view(y.shape[0], s.num_heads * dv)
        return linear(self.ctx, K.pad_cols(y, width) if width != y.shape[1] else y, self.w_o, keep_split=True)

    def forward_by_head(self, h, batch, cache):
        stacked = linear(self.ctx, h, self.w_qkv, out_dtype=torch.float32, keep_split=True)
        return linear(self.ctx, self.forward_stacked(stacked, 0, batch, cache), self.w_o, keep_split=True)

    @property
    def inner_width(self) -> int:
        return self.spec.num_heads * self.v_dim

    def forward_stacked(self, stacked, base: int, batch, cache, out=None, column: int = 0, pad_to=None, scale: float = 1.0):
        """The output product's input [rows, heads x value size] (padded to the product's width), from the columns
        `base`.. of a stacked product; with `out`, times `scale` and written to its columns from `column` on, zeros
        up to `column` + `pad_to`."""
        s, dv = self.spec, self.v_dim
        nq, nk = s.num_heads * s.head_dim, s.num_kv_heads * s.head_dim
        k_table, v_table = cache.tables()
        group = batch.groups[cache.group]
        rotary = self.position.rotary_dim
        q = K.head_norm_rope_append(stacked, base, base + nq, base + nq + nk, self.proj_norms[0], self.proj_norms[1],
                                    self.position.tables(batch) if rotary else None, rotary, group.lines, k_table, v_table,
                                    s.num_heads, s.num_kv_heads, s.head_dim, dv, cache.owns, self.ctx.dtype)
        heads_per_kv = s.num_heads // s.num_kv_heads
        if dv == s.head_dim and s.head_dim % 16 == 0 and K.attention_mma_takes(q.dtype, s.head_dim, heads_per_kv):
            prompt = "mma" if self.sinks is not None else K.attention_prompt_kernel(s.num_heads, s.num_kv_heads, s.head_dim, self.ctx.page_size, s.softcap)
            decode, tiles, split, slots, relative = batch.attention_tiles(heads_per_kv, s.num_kv_heads, s.window, s.head_dim, prompt)
            y = K.paged_attention_mma(q, k_table, v_table, group.block_table, batch.row_count, tiles, self.ctx.page_size, s.window,
                                      s.scale, s.softcap, decode, split, slots, relative, pairs=getattr(batch, "pairs", None), sinks=self.sinks)
        else:
            y = K.paged_attention_rows(q, k_table, v_table, group.block_table, batch.row_entry, batch.row_count, self.ctx.page_size,
                                       s.window, s.scale, s.softcap, batch.attention_slots(s.window), sinks=self.sinks)
        width = product_width(self.ctx, s.num_heads * dv) if pad_to is None else pad_to
        if s.gated or out is not None:
            return K.head_gate(y, stacked, base + nq + nk + s.num_kv_heads * dv if s.gated else 0, None, False, 0.0, self.ctx.dtype, pad_to=width,
                               gate_act="sigmoid" if s.gated else "none", by_head=s.gate_by_head, scale=scale, out=out, column=column)
        y = y.view(y.shape[0], s.num_heads * dv)
        return K.pad_cols(y, width) if width != y.shape[1] else y

    def forward(self, h, batch, cache):
        s = self.spec
        if self.convolved:
            y = self.forward_unbiased(h, batch, cache)
            return K.weighted_sum2(y, self.ones, None, None, self.out_bias) if self.out_bias is not None else y
        if self.pooled:
            return self.forward_pooled(h, batch, cache)
        if self.by_head:
            return self.forward_by_head(h, batch, cache)
        if self.general:
            return self.forward_general(h, batch, cache)
        qkv = linear(self.ctx, h, self.w_qkv, keep_split=True)
        k_table, v_table = cache.tables()
        group = batch.groups[cache.group]
        heads_per_kv = s.num_heads // s.num_kv_heads
        if K.attention_decode_fused_takes(qkv, s.num_heads, s.num_kv_heads, s.head_dim, self.position.rotary_dim,
                                          self.ctx.page_size, self.ctx.dtype):
            decode, tiles, split, slots, relative = batch.attention_tiles(
                heads_per_kv, s.num_kv_heads, s.window, s.head_dim,
                K.attention_prompt_kernel(s.num_heads, s.num_kv_heads, s.head_dim, self.ctx.page_size, s.softcap))
            if decode and relative:         # every request brings one token: rotation, the cache's new line and attention in one kernel
                y = K.paged_attention_decode_fused(
                    qkv, self.position.tables(batch), group.lines, k_table, v_table, group.block_table, batch.row_count,
                    s.num_heads, s.num_kv_heads, s.head_dim, cache.owns, self.ctx.page_size, s.window, s.scale, s.softcap,
                    split, slots)
                return linear(self.ctx, y.view(y.shape[0], s.num_heads * s.head_dim), self.w_o, keep_split=True)
        q = K.rope_append(
            qkv, self.position.tables(batch), group.lines, k_table, v_table,
            s.num_heads, s.num_kv_heads, s.head_dim, self.position.rotary_dim, write_kv=cache.owns,
            out_dtype=self.ctx.dtype,
        )
        if K.attention_mma_takes(q.dtype, s.head_dim, heads_per_kv):
            decode, tiles, split, slots, relative = batch.attention_tiles(
                heads_per_kv, s.num_kv_heads, s.window, s.head_dim,
                K.attention_prompt_kernel(s.num_heads, s.num_kv_heads, s.head_dim, self.ctx.page_size, s.softcap))
            y = K.paged_attention_mma(
                q, k_table, v_table, group.block_table, batch.row_count, tiles,
                self.ctx.page_size, s.window, s.scale, s.softcap, decode, split, slots, relative,
                pairs=getattr(batch, "pairs", None),
            )
        else:                   # the 32-bit path, and sizes the tensor-core kernel does not take
            y = K.paged_attention_rows(
                q, k_table, v_table, group.block_table, batch.row_entry, batch.row_count,
                self.ctx.page_size, s.window, s.scale, s.softcap, batch.attention_slots(s.window),
            )
        return linear(self.ctx, y.view(y.shape[0], s.num_heads * s.head_dim), self.w_o, keep_split=True)
