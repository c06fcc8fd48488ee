"""``ssd``: a selective state-space mixer with one decay per head and token and a matrix state carried
from token to token in the request's state slot (32-bit floats, zero at admission):

    [z | x | B | C | step] = W_in h     (z, x: H heads of vdim; B, C: ``groups`` rows of ``state``; step: H)
    x, B, C <- silu(conv(x, B, C) + bias)          (a causal convolution over time per channel)
    step <- softplus(step + step_bias)
    S_t = exp(-exp(A_log_h) step) S_(t-1) + step B_t x_t^T,    y_t = S_t^T C_t + D_h x_t    (S: [state, vdim])
    y <- y * silu(z), divided by its root mean square in ``norm_groups`` equal parts, times a gain; W_o y

Head h reads B and C of group h // (H / groups).  The convolution's last taps - 1 inputs are part of
the state.  One product, the convolution kernel (which forms steps and decays too), the recurrence
kernel, the gated norm kernel and the output product; all but the products' operands is 32-bit."""
from __future__ import annotations

import torch

from dispec_b200.ops import norm32 as norm32_ops
from dispec_b200.ops import recurrence as rec_ops
from dispec_b200.ops import short_conv as conv_ops
from dispec_b200.parts.base import JoinableMixer, StateNeed, TensorSpec
from dispec_b200.registry import register_part


@register_part("mixer", "ssd")
class StateSpaceDual(JoinableMixer):
    takes_out_scale = True

    def __init__(self, hidden_size: int, num_heads: int, vdim: int, state: int, groups: int, taps: int, norm_groups: int,
                 eps: float):
        if min(hidden_size, num_heads, vdim, state, groups, taps, norm_groups) <= 0:
            raise ValueError("ssd: sizes must be positive")
        if num_heads % groups or (num_heads * vdim) % norm_groups:
            raise ValueError(f"ssd: {num_heads} heads of {vdim} do not form {groups} groups and {norm_groups} normed parts")
        self.hidden_size, self.num_heads, self.vdim, self.state, self.groups = hidden_size, num_heads, vdim, state, groups
        self.taps, self.norm_groups, self.eps = int(taps), int(norm_groups), float(eps)
        self.inner = self.out_columns = num_heads * vdim
        self.channels = self.inner + 2 * groups * state

    def tensor_specs(self):
        H, h, f32 = self.num_heads, self.hidden_size, "float32"
        return {"in.weight": TensorSpec((self.inner + self.channels + H, h)), "o.weight": TensorSpec((h, self.inner)),
                "conv.weight": TensorSpec((self.channels, self.taps), dtype=f32, init="one_plus_normal"),
                "conv.bias": TensorSpec((self.channels,), dtype=f32), "step.bias": TensorSpec((H,), dtype=f32),
                "A_log": TensorSpec((H,), dtype=f32), "D": TensorSpec((H,), dtype=f32, init="one_plus_normal"),
                "norm.weight": TensorSpec((self.inner,), dtype=f32, init="one_plus_normal")}

    def load(self, tensors):
        self.w_in, self.w_o = tensors["in.weight"], tensors["o.weight"]
        self.w_conv = tensors["conv.weight"].t().contiguous()  # [taps, channels]
        self.b_conv, self.step_bias = tensors["conv.bias"], tensors["step.bias"]
        self.a_log, self.skip = tensors["A_log"], tensors["D"]
        self.gain = (tensors["norm.weight"] * self.out_scale).contiguous()

    def state_need(self):
        matrix = StateNeed((self.num_heads, self.state, self.vdim), "float32")
        if self.taps == 1:
            return (matrix,)
        return (matrix, StateNeed((self.taps - 1, self.channels), "float32"))

    def heads(self, ctx, z, cache, state, out):
        H, dv, N, G, inner = self.num_heads, self.vdim, self.state, self.groups, self.inner
        xbc, steps = conv_ops.conv_steps(z, inner, self.w_conv, self.b_conv, state[1].buffer if self.taps > 1 else None, ctx,
                                         step_offset=inner + self.channels, step_bias=self.step_bias, a_log=self.a_log)
        y = rec_ops.linear_recurrence(xbc, inner + G * N, inner, 0, rec_ops.STEP_DECAY, H, N, dv, state[0].buffer,
                                      state[0].slots, ctx.q_start, ctx.positions, steps=steps, skip=self.skip, num_groups=G)
        norm32_ops.head_norm_gate(y, self.norm_groups, self.eps, out.dtype, gain=self.gain, gate=z[:, :inner],
                                  gate_first=True, out=out)
