"""A layer whose norms come AFTER the residual sum (`PostNormBlockSpec`):

    x <- norm1(alpha x + mixer(x));   x <- norm2(alpha x + ffn(x))

on the fp32 stream; the sublayers read the stream itself. Between two sublayers ONE pass over the
stream takes up the output of the one, norms the sum and leaves the new stream in the type the
next one reads (`RMSNorm.join`); where the sublayer is two mixers side by side with norms of
their own, that pass norms and sums their outputs too. What the layer's last sublayer produced
leaves the block as `pending`, as with the other blocks.
"""

from __future__ import annotations

from .base import register_part
from .output_norm import OutputNormBlock
from .sandwich import _run


class PostNormUpdate:
    """A sublayer's output (`ys`: one tensor, or one a branch with the branches' `norms`) that the
    stream still has to take up: x <- norm(alpha x + scale * sum of the (normed) ys)."""

    __slots__ = ("ys", "norms", "scale", "norm", "alpha")

    def __init__(self, ys, norm, alpha, norms=None, scale=1.0):
        self.ys, self.norm, self.alpha = ys, norm, alpha
        self.norms, self.scale = norms, scale

    def take_up(self, x, out_dtype=None):
        """In place on x; returns the new stream in `out_dtype` (None: nothing)."""
        return self.norm.join(x, self.ys[0], self.alpha, out_dtype,
                              other=self.ys[1] if len(self.ys) > 1 else None, norms=self.norms,
                              scale=self.scale)

    def apply(self, x) -> None:
        self.take_up(x)


class PostNormBlock(OutputNormBlock):
    def __init__(self, spec, prefix, mode):
        super().__init__(spec, prefix, mode)
        self.kernel_libraries += ("norm",)              # (the model's last norm)
        for norm in (self.mixer_after, self.ffn_after):
            if norm is not None and (not hasattr(norm, "join") or norm.offset):
                raise ValueError(f"{type(norm).__name__} cannot norm the residual sum")

    def _update(self, part, norm, h, step, *cache):
        alpha = self.spec.alpha
        norms = getattr(part, "norms", None)
        if norms is not None and len(norms) == 2 and not any(n.offset for n in norms) \
                and norms[0].spec == norms[1].spec:
            return PostNormUpdate(part.produce_branches(h, step, *cache), norm, alpha, norms,
                                  part.spec.scale)
        return PostNormUpdate((_run(part, h, step, *cache),), norm, alpha)


register_part("post_norm_block", PostNormBlock)
