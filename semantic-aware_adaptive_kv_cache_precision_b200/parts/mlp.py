"""Dense gated feed-forward: `residual += down( silu(gate(h)) * up(h) )`
(`src/microinfer/model.py:392-396`, `src/core_kernels/swiglu.cu:26-38`). Gate and
up are one product over the rows [Wgate; Wup] laid back to back in device
memory; the activation is fp32 inside with one rounding at its store. The activation may
also be the clamped one (`GatedMLPSpec`)."""

from __future__ import annotations

import torch

from .. import ops
from ..weights.decl import TensorDecl
from .base import Part, register_part


class GatedMLP(Part):
    def __init__(self, spec, prefix, mode):
        super().__init__(spec, prefix, mode)
        if spec.activation not in ("silu", "clamped"):
            raise ValueError(f"activation {spec.activation!r}: 'silu' and 'clamped' are built")
        self.clamp = (spec.limit, spec.alpha, spec.plus) if spec.activation == "clamped" else None
        self.kernel_libraries = ("moe" if self.clamp else "elementwise",)
        if mode == "bfloat16":
            self.kernel_libraries += ("gemm_tc", "gemm_pair")
        if spec.bias:
            raise ValueError("a gated feed-forward with biases is not built")

    def tensor_decls(self):
        s, p = self.spec, self.prefix
        gate, up, down = self._names()
        return [TensorDecl(p + gate, (s.intermediate, s.hidden), group=p + "gate_up"),
                TensorDecl(p + up, (s.intermediate, s.hidden), group=p + "gate_up"),
                TensorDecl(p + down, (s.hidden, s.intermediate))]

    def _names(self):
        return getattr(self.spec, "names",
                       ("gate_proj.weight", "up_proj.weight", "down_proj.weight"))

    def bind(self, arena):
        p = self.prefix
        gate, up, down = self._names()
        self.w_gate_up = arena.group_view(p + "gate_up")
        if self.w_gate_up is None:
            self.w_gate_up = torch.cat([arena.view(p + gate), arena.view(p + up)])
        self.w_down = arena.view(p + down)

    def produce(self, h, step):
        """The feed-forward's output as a tensor of its own, fp32 [T, hidden]."""
        return ops.linear(ops.gated_up(h, self.w_gate_up, self.clamp), self.w_down,
                          out_dtype=torch.float32)

    can_defer = True

    def forward(self, h, step, residual, defer=False):
        act = ops.gated_up(h, self.w_gate_up, self.clamp)
        out = ops.linear(act, self.w_down, accumulate_into=residual, may_defer=defer)
        return out.delta if isinstance(out, ops.Deferred) else None


class DenseMLP(Part):
    """Dense feed-forward without a gate, `down(act(up(h)))`, with the tanh form of GELU or the
    square of relu (fp32 inside, one rounding at its store); tensors `up` and `down`."""

    kernel_libraries = ("elementwise",)

    def __init__(self, spec, prefix, mode):
        super().__init__(spec, prefix, mode)
        if spec.activation not in ("gelu_tanh", "relu_squared"):
            raise ValueError(f"activation {spec.activation!r}: 'gelu_tanh' and 'relu_squared' are "
                             "built")

    def tensor_decls(self):
        s, p = self.spec, self.prefix
        return [TensorDecl(p + "up", (s.intermediate, s.hidden)),
                TensorDecl(p + "down", (s.hidden, s.intermediate))]

    def bind(self, arena):
        self.w_up = arena.view(self.prefix + "up")
        self.w_down = arena.view(self.prefix + "down")

    def _act(self, h):
        if self.spec.activation == "relu_squared":
            return ops.dense_up(h, self.w_up)
        return ops.gelu_tanh(ops.linear(h, self.w_up, out_dtype=self.act_dtype))

    def produce(self, h, step):
        """The feed-forward's output, fp32 [T, hidden]."""
        return ops.linear(self._act(h), self.w_down, out_dtype=torch.float32)

    can_defer = True

    def forward(self, h, step, residual, defer=False):
        out = ops.linear(self._act(h), self.w_down, accumulate_into=residual, may_defer=defer)
        return out.delta if isinstance(out, ops.Deferred) else None


register_part("gated_mlp", GatedMLP)
register_part("dense_mlp", DenseMLP)
