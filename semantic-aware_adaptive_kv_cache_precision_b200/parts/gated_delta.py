"""The gated delta-rule mixer (`GatedDeltaSpec`):

    [q | k | v | g | a | b] = h Win^T
    q, k, v <- silu(conv(q)), silu(conv(k)), silu(conv(v))    a causal convolution a channel, `taps` tokens
    q <- q_scale * q / sqrt(sum(q^2) + unit_eps),  k <- k / sqrt(sum(k^2) + unit_eps)          (a head)
    decay = exp(-exp(A_log) softplus(a + dt_bias)),  beta = sigmoid(b)              (one number a head)
    S <- decay S;  u = beta (v - S^T k);  S <- S + k u^T;  o = S^T q      (a head; S is head_dim x vdim)
    out = Wo [ o / rms(o) * w * silu(g) ]                                            (rms a head)

The projection leaves fp32 (its accumulator, unrounded) and everything between it and the input of
the output product is fp32 in both modes (`csrc/gated_delta.cu`; norm and gate in
`csrc/recurrent_scan.cu`). A sequence's state (the convolutions' last `taps - 1` inputs and S,
stored as its transpose [heads, vdim, head_dim]) lives in the cache as two fixed-size states.

In bfloat16 the tokens of a prompt are taken four at a time (`ops.gated_delta`); in the 32-bit mode,
and for decode steps, one at a time, with sums that do not depend on how the sequence was cut. The
part is a mixer of its own (`produce`) and a branch of a `ParallelMixer`.
"""

from __future__ import annotations

import torch

from .. import ops
from ..cache.needs import MultiNeed, StateNeed
from ..weights.decl import TensorDecl
from .base import Part, register_part


class GatedDeltaMixer(Part):
    kernel_libraries = ("gated_delta", "recurrent_scan", "gemm_f32", "gemm_tc")

    def __init__(self, spec, prefix, mode):
        super().__init__(spec, prefix, mode)
        s = spec
        if s.heads % s.kv_heads:
            raise ValueError(f"{s.heads} heads are not a multiple of {s.kv_heads} kv heads")
        if s.head_dim > 512 or not 1 <= s.taps <= 64:
            raise ValueError("the delta kernels take head_dim up to 512 and 1 to 64 taps")
        self.qk_cols, self.v_cols = s.kv_heads * s.head_dim, s.heads * s.value_dim
        self.channels = 2 * self.qk_cols + self.v_cols           # what passes the convolutions

    # -- what a branch offers -------------------------------------------------------------

    def _inputs(self):
        return (("q", self.qk_cols), ("k", self.qk_cols), ("v", self.v_cols), ("g", self.v_cols),
                ("a", self.spec.heads), ("b", self.spec.heads))

    @property
    def input_rows(self) -> int:
        return self.channels + self.v_cols + 2 * self.spec.heads

    def input_decls(self, group):
        return [TensorDecl(self.prefix + n, (rows, self.spec.hidden), group=group)
                for n, rows in self._inputs()]

    def other_decls(self):
        s, p = self.spec, self.prefix
        return [TensorDecl(f"{p}{n}.conv", (rows, s.taps), init="uniform", span=(-0.7, 0.7),
                           group=p + "conv") for n, rows in self._inputs()[:3]] + [
                TensorDecl(p + "A_log", (s.heads,), init="uniform", span=(-2.0, 1.0)),
                TensorDecl(p + "dt_bias", (s.heads,), init="uniform", span=(-4.0, -1.0)),
                TensorDecl(p + "norm", (s.value_dim,), init="ones_normal"),
                TensorDecl(p + "o", (s.hidden, self.v_cols))]

    def input_bias(self, arena):
        return None

    def bind_rest(self, arena):
        s, p = self.spec, self.prefix
        self.conv_w = arena.group_view(p + "conv")
        if self.conv_w is None:
            self.conv_w = torch.cat([arena.view(f"{p}{n}.conv") for n in "qkv"])
        self.norm_w = arena.view(p + "norm").repeat(s.heads)     # (the heads share one weight)
        self.w_o = arena.view(p + "o")
        self.dt_bias = arena.view(p + "dt_bias").float().contiguous()
        # the decay rates, worked out in float64 once
        self.a = (-torch.exp(arena.view(p + "A_log").double())).float().contiguous()

    def mix(self, proj, offset, h, step, view, write_cache=True):
        """From the fused product `proj` (fp32 [T, columns], this branch's columns from `offset`
        on) to the input of `w_o`: [T, heads * value_dim] of the activations' type."""
        s = self.spec
        conv_view, state_view = view.parts
        g_off = self.channels
        a_off = g_off + self.v_cols
        mine = proj[:, offset:offset + self.input_rows]
        o = ops.gated_delta(mine, a_off, a_off + s.heads, self.conv_w, self.a, self.dt_bias,
                            conv_view.state, state_view.state, step, s.heads, s.kv_heads,
                            s.head_dim, s.value_dim, s.q_scale, s.unit_eps, keep_state=write_cache,
                            by_groups=self.act_dtype != torch.float32)
        return ops.norm_gate(o, self.norm_w, mine[:, g_off:a_off], s.eps, 1.0, self.act_dtype,
                             group=s.value_dim, gate_silu=True)

    # -- the part alone ---------------------------------------------------------------------

    def tensor_decls(self):
        return self.input_decls(self.prefix + "fused") + self.other_decls()

    def bind(self, arena):
        p = self.prefix
        self.w_in = arena.group_view(p + "fused")
        if self.w_in is None:
            self.w_in = torch.cat([arena.view(p + n) for n, _ in self._inputs()])
        self.bind_rest(arena)

    def cache_need(self):
        s = self.spec
        return MultiNeed((StateNeed((s.taps - 1, self.channels), "float32"),
                          StateNeed((s.heads, s.value_dim, s.head_dim), "float32")))

    def produce(self, h, step, view, write_cache=True):
        """The mixer's output, fp32 [T, hidden]."""
        proj = ops.linear(h, self.w_in, out_dtype=torch.float32)
        return ops.linear(self.mix(proj, 0, h, step, view, write_cache), self.w_o,
                          out_dtype=torch.float32)

    def forward(self, h, step, view, residual, write_cache=True):
        proj = ops.linear(h, self.w_in, out_dtype=torch.float32)
        ops.linear(self.mix(proj, 0, h, step, view, write_cache), self.w_o,
                   accumulate_into=residual)


register_part("gated_delta", GatedDeltaMixer)
