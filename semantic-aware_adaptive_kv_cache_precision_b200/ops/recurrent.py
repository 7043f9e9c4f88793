"""The delta-rule recurrences over a step's tokens (`csrc/delta_rule.cu`: a decay and a removal rate
a channel; `csrc/gated_delta.cu`: one decay and one step a head)."""

from __future__ import annotations

import torch

from ._lib import KernelError, call, dtype_code, plain_function, ptr, require_cuda


def delta_rule(proj: torch.Tensor, offsets: tuple, w2: torch.Tensor, w0: torch.Tensor,
               a_bias: torch.Tensor, norm_w: torch.Tensor, state: torch.Tensor, step, heads: int,
               dim: int, decay_scale: float, key_eps: float, eps: float,
               out_dtype: torch.dtype, keep_state: bool = True) -> torch.Tensor:
    """`proj`: fp32 [T, P], whose columns from `offsets` = (r, k, v, g, a, l) on are the
    receptance, key, value, gate and removal-rate pre-activations (heads * dim each) and the
    decay's low-rank output (rank = w2.shape[1]). `state`: fp32 [slots, heads, dim, dim], read
    and left for each of the step's sequences. Returns the normed, gated output [T, heads *
    dim] of `out_dtype`."""
    require_cuda(proj, w2, w0, a_bias, norm_w, state)
    tokens = proj.shape[0]
    hd = heads * dim
    rank = w2.shape[1]

    def check(cond, message):
        if not cond:
            raise KernelError(message)

    check(proj.dtype == torch.float32 and proj.dim() == 2 and proj.stride(1) == 1,
          "proj: fp32 [T, P] with contiguous rows")
    check(len(offsets) == 6 and max(offsets[:5]) + hd <= proj.shape[1]
          and offsets[5] + rank <= proj.shape[1], "offsets reach beyond proj's columns")
    check(w2.shape == (hd, rank) and w2.is_contiguous(), "w2: [heads * dim, rank]")
    for t, name in ((w0, "w0"), (a_bias, "a_bias"), (norm_w, "norm_w")):
        check(t.shape == (hd,) and t.is_contiguous() and t.dtype == w2.dtype,
              f"{name}: [heads * dim] of w2's type")
    check(state.dtype == torch.float32 and state.is_contiguous()
          and tuple(state.shape[1:]) == (heads, dim, dim), "state: fp32 [slots, heads, dim, dim]")
    out = torch.empty((tokens, hd), dtype=out_dtype, device=proj.device)
    prepared = torch.empty((tokens, 3, hd), dtype=torch.float32, device=proj.device)
    raw = torch.empty((tokens, hd), dtype=torch.float32, device=proj.device)
    call("sakv_delta_rule", ptr(proj), proj.stride(0), *[int(o) for o in offsets], ptr(w2),
         ptr(w0), ptr(a_bias), ptr(norm_w), dtype_code(w2.dtype), ptr(prepared), ptr(raw), ptr(state),
         ptr(step.cu_seqlens), ptr(step.slots), ptr(out), dtype_code(out_dtype), tokens,
         step.sequences, heads, dim, rank,
         int(max(1, min(16, getattr(step, "max_new", 0) or tokens))),
         float(decay_scale), float(key_eps), float(eps), int(keep_state))
    return out


def gated_delta(proj: torch.Tensor, a_off: int, b_off: int, conv: torch.Tensor, a: torch.Tensor,
                dt_bias: torch.Tensor, conv_state: torch.Tensor, state: torch.Tensor, step,
                heads: int, kv_heads: int, dim: int, vdim: int, q_scale: float, unit_eps: float,
                keep_state: bool = True, by_groups: bool = False) -> torch.Tensor:
    """The gated delta rule over each sequence's tokens. `proj`: fp32 [T, columns] (any row stride)
    whose first columns are the pre-activations of q (kv_heads * dim), k (the same) and v (heads *
    vdim), with one column a head of the decays from `a_off` and of the betas from `b_off`. q, k, v
    pass the causal convolution `conv` ([channels, taps] over those channels) and silu, q and k
    become unit vectors a head (x / sqrt(sum(x^2) + unit_eps)), q times `q_scale`; `decay = exp(a *
    softplus(. + dt_bias))` with `a`, `dt_bias` fp32 [heads], a negative; `beta = sigmoid(.)`; then
    per head `S <- decay S; u = beta (v - S^T k); S <- S + k u^T; o = S^T q`. `conv_state`: fp32
    [slots, taps - 1, channels]; `state`: fp32 [slots, heads, vdim, dim]; both are read and (with
    `keep_state`) left. Returns o, fp32 [T, heads * vdim].

    `by_groups`: the recurrence takes four tokens at a time (their sums over the state are taken
    together). Otherwise one at a time, with sums that do not depend on how the sequence was cut."""
    require_cuda(proj, conv, a, dt_bias, conv_state, state)

    def check(cond, message):
        if not cond:
            raise KernelError(message)

    tokens, channels, taps = proj.shape[0], 2 * kv_heads * dim + heads * vdim, conv.shape[1]
    check(proj.dtype == torch.float32 and proj.dim() == 2 and proj.stride(1) == 1
          and max(channels, a_off + heads, b_off + heads) <= proj.shape[1],
          "proj: fp32 [T, columns] with contiguous rows holding q, k, v, the decays and the betas")
    check(heads % kv_heads == 0, "heads must be a multiple of kv_heads")
    check(conv.shape == (channels, taps) and conv.is_contiguous(), "conv: [channels, taps]")
    for t, name in ((a, "a"), (dt_bias, "dt_bias")):
        check(t.dtype == torch.float32 and t.shape == (heads,) and t.is_contiguous(),
              f"{name}: fp32 [heads]")
    check(conv_state.dtype == torch.float32 and conv_state.is_contiguous()
          and tuple(conv_state.shape[1:]) == (taps - 1, channels),
          "conv_state: fp32 [slots, taps - 1, channels]")
    check(state.dtype == torch.float32 and state.is_contiguous()
          and tuple(state.shape[1:]) == (heads, vdim, dim), "state: fp32 [slots, heads, vdim, dim]")
    most = int(getattr(step, "max_new", 0) or tokens)
    prepared = torch.empty((tokens, channels), dtype=torch.float32, device=proj.device)
    gates = torch.empty((tokens, heads, 2), dtype=torch.float32, device=proj.device)
    out = torch.empty((tokens, heads * vdim), dtype=torch.float32, device=proj.device)
    coef = None
    if by_groups and most > 1:
        coef = torch.empty((tokens // 4 + step.sequences, heads,
                            plain_function("sakv_delta_coefficients")()),
                           dtype=torch.float32, device=proj.device)
    call("sakv_delta_inputs", ptr(proj), proj.stride(0), int(a_off), int(b_off), ptr(conv),
         dtype_code(conv.dtype), ptr(a), ptr(dt_bias), ptr(conv_state), ptr(step.cu_seqlens),
         ptr(step.slots), ptr(prepared), ptr(gates), ptr(coef), step.sequences, most, heads,
         kv_heads, dim, vdim, taps, int(keep_state and most == 1), float(q_scale), float(unit_eps))
    call("sakv_delta_scan", ptr(prepared), ptr(gates), ptr(coef), ptr(state), ptr(step.cu_seqlens),
         ptr(step.slots), ptr(out), step.sequences, most, heads, kv_heads, dim, vdim,
         int(keep_state))
    if keep_state and most > 1 and taps > 1:
        call("sakv_conv_state", ptr(proj), proj.stride(0), ptr(conv_state), ptr(step.cu_seqlens),
             ptr(step.slots), step.sequences, channels, taps)
    return out
