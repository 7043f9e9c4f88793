"""A layer whose two sublayers read the output of one norm and are added together
(`ParallelBlockSpec`):

    h = norm(x);   x += mixer(h) + ffn(h)

on the fp32 residual stream. Both sublayers add into the stream themselves, the mixer first: what
the second one reads, h, was made before either. What the feed-forward hands back instead (`defer`)
leaves the block as `pending`, and the next layer's norm adds it on its way.
"""

from __future__ import annotations

from .base import Part, build_part, register_part
from .block import _normed


class ParallelBlock(Part):
    def __init__(self, spec, prefix, mode):
        super().__init__(spec, prefix, mode)
        p = spec.prefix
        self.norm = build_part(spec.norm, p + spec.norm_name, mode)
        self.mixer = build_part(spec.mixer, p + spec.mixer_name + ".", mode)
        self.ffn = None if spec.ffn is None else build_part(spec.ffn, p + spec.ffn_name + ".", mode)
        self.parts = tuple(x for x in (self.norm, self.mixer, self.ffn) if x is not None)
        self.kernel_libraries = ("norm",) + tuple(
            n for part in self.parts for n in getattr(part, "kernel_libraries", ()))
        self.graph_safe = all(getattr(part, "graph_safe", True) for part in self.parts)

    def tensor_decls(self):
        return [d for part in self.parts for d in part.tensor_decls()]

    def bind(self, arena):
        for part in self.parts:
            part.bind(arena)

    def prepare(self, device, max_positions):
        for part in self.parts:
            part.prepare(device, max_positions)

    def cache_need(self):
        return self.mixer.cache_need()

    carries_pending = True

    def forward(self, x, step, view, write_cache=True, pending=None, leave_pending=True):
        h = _normed(self.norm, x, pending)
        last = self.mixer if self.ffn is None else self.ffn
        defer = leave_pending and getattr(last, "can_defer", False)
        if self.ffn is None:
            return self.mixer.forward(h, step, view, x, write_cache, **({"defer": True} if defer else {}))
        self.mixer.forward(h, step, view, x, write_cache)
        return self.ffn.forward(h, step, x, **({"defer": True} if defer else {}))


register_part("parallel_block", ParallelBlock)
