"""RMS norm with an offset on its weight: y = x / sqrt(mean(x^2) + eps) * (offset + w)
(crates/kapel-ops/src/norm.rs:123-135; Gemma 2's offset is 1, crates/kapel-models/src/config.rs:284)."""
from __future__ import annotations

from .. import kernels as K
from .base import Part


class RMSNorm(Part):
    graph_safe = True
    center = False                      # whether the row's mean is taken off first

    def __init__(self, spec, ctx):
        super().__init__(spec, ctx)
        self.offset = spec.offset
        self.bias = None
        if self.spec.bias is not None and not self.center:
            raise ValueError("norm: a bias is built for layer norms only")

    @staticmethod
    def expected_tensors(spec):
        return {spec.weight: (spec.width,)}

    def load(self, tensors):
        w = tensors[self.spec.weight]
        if w.device != self.ctx.device:
            w = w.to(self.ctx.device)
        self.weight = w.float() if self.ctx.is_f32 else w.contiguous()

    def forward(self, x, out_dtype=None):
        return K.rmsnorm(x, self.weight, self.spec.eps, self.offset, out_dtype or self.ctx.dtype)

    def fuse_key(self):
        """(weight, eps, offset): what the fused add-and-norm kernel needs to apply this norm."""
        return (self.weight, self.spec.eps, self.offset)

    def scale_output(self, scale: float) -> None:
        """The norm's output times `scale` from now on: the weight (and the bias) are multiplied once, in 32-bit."""
        if scale != 1.0:
            self.weight = ((self.weight.float() + self.offset) * scale).contiguous()
            self.offset = 0.0
            if self.bias is not None:
                self.bias = (self.bias.float() * scale).contiguous()

    def wide_key(self):
        """(weight, bias or None, eps, offset, center) with float32 vectors, for a kernel that reads several streams."""
        return (self.weight.float().contiguous(), self.bias.float().contiguous() if self.bias is not None else None, self.spec.eps, self.offset,
                self.center)


class LayerNorm(RMSNorm):
    """y = (x - mean) / sqrt(mean((x - mean)^2) + eps) * (offset + w), plus a bias where the spec names one, in
    32-bit. Without a bias the fused sum-and-norm kernel takes it by a flag beside the RMS norm's triple."""

    center = True

    @staticmethod
    def expected_tensors(spec):
        return {n: (spec.width,) for n in (spec.weight, spec.bias) if n is not None}

    def load(self, tensors):
        super().load(tensors)
        if self.spec.bias is not None:
            self.bias = tensors[self.spec.bias].to(self.ctx.device).to(self.weight.dtype).contiguous()

    def forward(self, x, out_dtype=None):
        return K.layernorm(x, self.weight, self.spec.eps, self.offset, out_dtype or self.ctx.dtype, bias=self.bias)

    def fuse_key(self):
        """(weight, eps, offset, True): the last says that the row's mean is taken off first. None with a bias."""
        return (self.weight, self.spec.eps, self.offset, True) if self.bias is None else None


def add_branch(ctx, residual, branch, post_norm, next_norm, copy_out: bool = False):
    """residual += post_norm(branch) (post_norm None: plain sum); returns next_norm(residual),
    or None without a next norm (with `copy_out`: the new residual in the activation dtype, for a
    block whose branches read the residual itself). One kernel when the norms are RMS norms with
    weights of one dtype; a norm of another kind runs through its own `forward` around the fused sum."""
    post_key = post_norm.fuse_key() if hasattr(post_norm, "fuse_key") else None
    next_key = next_norm.fuse_key() if hasattr(next_norm, "fuse_key") else None
    if post_norm is not None and post_key is None:
        branch = post_norm.forward(K.finish(branch, ctx.dtype))
    if next_key is not None and (post_key is None or post_key[0].dtype == next_key[0].dtype):
        return K.add_rmsnorm(residual, branch, post_key, next_key, ctx.dtype)
    copied = K.add_rmsnorm(residual, branch, post_key, None, ctx.dtype, copy_out=copy_out and next_norm is None)
    return next_norm.forward(residual) if next_norm is not None else copied
