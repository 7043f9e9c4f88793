"""The state-space dual mixer (`DualScanSpec`):

    [z | x | B | C | dt] = h Win^T
    [x | B | C] <- silu(conv([x | B | C]) + b)      a causal convolution a channel over `taps` tokens
    dt <- softplus(dt + dt_bias);   A = -exp(A_log)                        (one number a head)
    S <- exp(dt A) S + dt B x^T;   y = S^T C + D x                         (a head; S is state x vdim)
    out = Wo [ n(y * silu(z)) * w ]                 n: each of `norm_groups` parts by its own rms

The projection leaves fp32 (its accumulator, unrounded); step sizes, decays and their
exponentials, the state, the sums over it, the gate and the norm are fp32 in both modes
(`csrc/recurrent_scan.cu`). A sequence's state (the convolution's last `taps - 1` inputs and S,
stored as its transpose [heads, vdim, state]) lives in the cache as two fixed-size states. The
state moves by its change, `S += (e^(dt A) - 1) S + dt B x^T`.

In bfloat16 a long part of a prompt is walked in runs of `RUN` tokens side by side. The part is a
mixer of its own (`produce`) and a branch of a `ParallelMixer`.
"""

from __future__ import annotations

import torch

from .. import ops
from ..cache.needs import MultiNeed, StateNeed
from ..weights.decl import TensorDecl
from .base import Part, register_part

#: tokens a run when a long prompt is walked in runs side by side
RUN = 64


class DualScanMixer(Part):
    kernel_libraries = ("recurrent_scan", "gemm_f32", "gemm_tc")

    def __init__(self, spec, prefix, mode):
        super().__init__(spec, prefix, mode)
        s = spec
        if s.heads % s.groups:
            raise ValueError(f"{s.heads} heads are not a multiple of {s.groups} groups")
        if s.state > 256 or not 1 <= s.taps <= 64:
            raise ValueError("the scan kernels take up to 256 states a head and 1 to 64 taps")
        self.inner = s.heads * s.value_dim
        if self.inner % s.norm_groups:
            raise ValueError(f"{self.inner} channels are not a multiple of {s.norm_groups} norm groups")
        self.channels = self.inner + 2 * s.groups * s.state      # what passes the convolution

    # -- what a branch offers -------------------------------------------------------------

    @property
    def input_rows(self) -> int:
        return self.inner + self.channels + self.spec.heads

    def input_decls(self, group):
        return [TensorDecl(self.prefix + "in", (self.input_rows, self.spec.hidden), group=group)]

    def other_decls(self):
        s, p = self.spec, self.prefix
        return [TensorDecl(p + "conv", (self.channels, s.taps)),
                TensorDecl(p + "conv.b", (self.channels,)),
                TensorDecl(p + "dt_bias", (s.heads,), init="uniform", span=(-4.0, -1.0)),
                TensorDecl(p + "A_log", (s.heads,), init="uniform", span=(-2.0, 1.0)),
                TensorDecl(p + "D", (s.heads,), init="ones_normal"),
                TensorDecl(p + "norm", (self.inner,), init="ones_normal"),
                TensorDecl(p + "o", (s.hidden, self.inner))]

    def input_bias(self, arena):
        return None

    def bind_rest(self, arena):
        p = self.prefix
        self.conv_w, self.conv_b = arena.view(p + "conv"), arena.view(p + "conv.b")
        self.norm_w, self.w_o = arena.view(p + "norm"), arena.view(p + "o")
        self.dt_bias = arena.view(p + "dt_bias").float().contiguous()
        self.d_skip = arena.view(p + "D").float().contiguous()
        # the decay rates, worked out in float64 once
        self.a = (-torch.exp(arena.view(p + "A_log").double())).float().contiguous()

    def mix(self, proj, offset, h, step, view, write_cache=True):
        """From the fused product `proj` (fp32 [T, columns], this branch's columns from
        `offset` on) to the input of `w_o`: [T, heads * value_dim] of the activations' type."""
        s = self.spec
        conv_view, scan_view = view.parts
        at = offset + self.inner
        xbc = ops.causal_conv(proj[:, at:at + self.channels], self.channels, self.conv_w,
                              self.conv_b, conv_view.state, step, self.act_dtype,
                              keep_state=write_cache)
        dt = proj[:, at + self.channels:at + self.channels + s.heads]
        y = ops.dual_scan(xbc, 0, self.inner, self.inner + s.groups * s.state, dt, self.dt_bias,
                          self.a, self.d_skip, s.heads, s.groups, s.state, s.value_dim,
                          scan_view.state, step, keep_state=write_cache, run=self._run(step))
        return ops.norm_gate(y, self.norm_w, proj[:, offset:at], s.eps, 1.0, self.act_dtype,
                             group=self.inner // s.norm_groups, gate_silu=True, gate_first=True)

    def _run(self, step) -> int:
        """Tokens a run of a long prompt: in bfloat16 a sequence's part of the step is walked
        in runs side by side (the states carried between them in fp32). In the 32-bit mode,
        and for short parts, one walk, whose sums do not depend on how the sequence was cut."""
        if self.act_dtype == torch.float32 or getattr(step, "max_new", 0) < 4 * RUN:
            return 0
        return RUN

    # -- the part alone ---------------------------------------------------------------------

    def tensor_decls(self):
        return self.input_decls(None) + self.other_decls()

    def bind(self, arena):
        self.w_in = arena.view(self.prefix + "in")
        self.bind_rest(arena)

    def cache_need(self):
        s = self.spec
        return MultiNeed((StateNeed((s.taps - 1, self.channels), "float32"),
                          StateNeed((s.heads, s.value_dim, s.state), "float32")))

    def produce(self, h, step, view, write_cache=True):
        """The mixer's output, fp32 [T, hidden]."""
        proj = ops.linear(h, self.w_in, out_dtype=torch.float32)
        return ops.linear(self.mix(proj, 0, h, step, view, write_cache), self.w_o,
                          out_dtype=torch.float32)

    def forward(self, h, step, view, residual, write_cache=True):
        proj = ops.linear(h, self.w_in, out_dtype=torch.float32)
        ops.linear(self.mix(proj, 0, h, step, view, write_cache), self.w_o,
                   accumulate_into=residual)


register_part("dual_scan", DualScanMixer)
