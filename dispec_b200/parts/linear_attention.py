"""Linear-attention mixers whose memory is a matrix state per head and request, carried from
token to token in the request's state slot (32-bit floats, zero at admission):

    S_t = diag(a_t) S_(t-1) + b_t v_t^T,      o_t = S_t^T q_t        (S: [dim, vdim])

``retention``: a fixed decay per head, a_t = decay_h; q and k are turned by a rotary encoding
(pairs (i, i + rot/2)), k scaled by dim^(-1/2) afterwards, b_t = k_t; every head's o is divided
by its root mean square (no gain), the heads are multiplied by silu(W_g h) and projected.

``hgrn2``: the forget gate also decides what is written: f_t = lower + (1 - lower) *
sigmoid(W_f h + bias), a_t = f_t, b_t = 1 - f_t, q_t = silu(W_q h); every head's o is RMS-normed
with one gain of size vdim shared by the heads, then projected.

``lightning``: a fixed decay per head, q, k and v all pass through silu, a_t = decay_h, b_t = k_t,
no other scale; the concatenated heads are RMS-normed together with one gain over all of them,
multiplied by sigmoid(W_g h) and projected.

``gated_linear_attention``: a decay per key channel and token, a_t = sigmoid(z)^(1/tau) with
z = W_a2 (W_a1 h) + bias, q scaled by dim^(-1/2), b_t = k_t; every head's o is RMS-normed with one gain of
size vdim, multiplied by silu(W_g h) and projected.

``delta`` (with ``kv_heads`` groups of heads that share q and k): the gated delta rule, which writes what the state
does not hold yet.  q, k, v = silu(C(W h)), C a causal convolution over time per channel (``taps`` weights a
channel, zeros before the start; its last taps - 1 inputs are part of the state); q and k divided by their
length per head, x / sqrt(sum(x^2) + 1e-6), q then scaled by dim^(-1/2);

    beta = sigmoid(W_b h),  g = exp(-exp(A_log) softplus(W_a h + dt_bias))        (one each per head and token)
    S <- g S;   u = beta (v - S^T k);   S <- S + k u^T;   o = S^T q

every head's o is RMS-normed with one gain of size vdim, multiplied by silu(W_g h) and projected.

The others run one fused projection, the recurrence kernel (which forms a_t, b_t, q_t from the raw
projection rows in 32-bit), the per-head norm kernel and the output projection; ``delta`` has the
convolution kernel in front of its recurrence.
"""
from __future__ import annotations

import torch

from dispec_b200 import ops
from dispec_b200.ops import norm32 as norm32_ops
from dispec_b200.ops import recurrence as rec_ops
from dispec_b200.ops import short_conv as conv_ops
from dispec_b200.parts.base import JoinableMixer, Mixer, StateNeed, TensorSpec
from dispec_b200.registry import register_part


class _MatrixStateMixer(Mixer):
    def __init__(self, hidden_size: int, num_heads: int, dim: int, vdim: int, eps: float):
        if min(hidden_size, num_heads, dim, vdim) <= 0:
            raise ValueError("sizes of a linear-attention mixer must be positive")
        self.hidden_size, self.num_heads, self.dim, self.vdim = hidden_size, num_heads, dim, vdim
        self.eps = float(eps)
        self.w_in = self.w_o = None

    def state_need(self):
        return StateNeed((self.num_heads, self.dim, self.vdim), "float32")


@register_part("mixer", "retention")
class Retention(_MatrixStateMixer):
    def __init__(self, hidden_size: int, num_heads: int, dim: int, vdim: int, decay, eps: float,
                 position_encoding):
        super().__init__(hidden_size, num_heads, dim, vdim, eps)
        decay = [float(v) for v in decay]
        if len(decay) != num_heads:
            raise ValueError(f"retention: {len(decay)} decays for {num_heads} heads")
        self.decay_values = decay
        self.position_encoding = position_encoding
        self.decay = None

    def tensor_specs(self):
        h, H, d, dv = self.hidden_size, self.num_heads, self.dim, self.vdim
        return {"q.weight": TensorSpec((H * d, h)), "k.weight": TensorSpec((H * d, h)),
                "v.weight": TensorSpec((H * dv, h)), "g.weight": TensorSpec((H * dv, h)),
                "o.weight": TensorSpec((h, H * dv))}

    def load(self, tensors):
        self.w_in = torch.cat([tensors["q.weight"], tensors["k.weight"], tensors["v.weight"],
                               tensors["g.weight"]], dim=0).contiguous()
        self.w_o = tensors["o.weight"]
        self.decay = torch.tensor(self.decay_values, dtype=torch.float32, device=self.w_o.device)

    def forward(self, ctx, x, cache, state):
        H, d, dv = self.num_heads, self.dim, self.vdim
        proj = ops.linear(x, self.w_in, out_dtype=torch.float32)  # [T, q | k | v | g]
        rot = self.position_encoding.rotation()
        if rot is not None and rot.layout != "halves":
            raise ValueError(f"retention turns pairs (i, i + rot/2) only, not the {rot.layout!r} layout")
        o = rec_ops.linear_recurrence(
            proj, 0, H * d, 2 * H * d, rec_ops.FIXED_DECAY, H, d, dv, state.buffer, state.slots, ctx.q_start,
            ctx.positions, decay=self.decay, inv_freq=rot.inv_freq if rot is not None else None,
            rot=rot.rotary_dim if rot is not None else 0, key_scale=d ** -0.5)
        gated = norm32_ops.head_norm_gate(o, H, self.eps, x.dtype, gate=proj[:, 2 * H * d + H * dv:])
        return ops.linear(gated, self.w_o, out_dtype=torch.float32)


@register_part("mixer", "hgrn2")
class HGRN2(_MatrixStateMixer):
    def tensor_specs(self):
        h, H, d, dv = self.hidden_size, self.num_heads, self.dim, self.vdim
        return {"q.weight": TensorSpec((H * d, h)), "f.weight": TensorSpec((H * d, h)),
                "f.bias": TensorSpec((H * d,), dtype="float32", init="zeros"),
                "lower": TensorSpec((H * d,), dtype="float32", init="zeros"),
                "v.weight": TensorSpec((H * dv, h)),
                "norm.weight": TensorSpec((dv,), dtype="float32", init="one_plus_normal"),
                "o.weight": TensorSpec((h, H * dv))}

    def load(self, tensors):
        self.w_in = torch.cat([tensors["q.weight"], tensors["f.weight"], tensors["v.weight"]], dim=0).contiguous()
        self.f_bias, self.lower, self.gain = tensors["f.bias"], tensors["lower"], tensors["norm.weight"]
        self.w_o = tensors["o.weight"]

    def forward(self, ctx, x, cache, state):
        H, d, dv = self.num_heads, self.dim, self.vdim
        proj = ops.linear(x, self.w_in, out_dtype=torch.float32)  # [T, q | f | v]
        o = rec_ops.linear_recurrence(
            proj, 0, H * d, 2 * H * d, rec_ops.FORGET_GATE, H, d, dv, state.buffer, state.slots, ctx.q_start,
            ctx.positions, gate_bias=self.f_bias, lower=self.lower)
        normed = norm32_ops.head_norm_gate(o, H, self.eps, x.dtype, gain=self.gain)
        return ops.linear(normed, self.w_o, out_dtype=torch.float32)


@register_part("mixer", "lightning")
class Lightning(_MatrixStateMixer):
    def __init__(self, hidden_size: int, num_heads: int, dim: int, vdim: int, decay, eps: float):
        super().__init__(hidden_size, num_heads, dim, vdim, eps)
        decay = [float(v) for v in decay]
        if len(decay) != num_heads:
            raise ValueError(f"lightning: {len(decay)} decays for {num_heads} heads")
        self.decay_values = decay
        self.decay = self.gain = None

    def tensor_specs(self):
        h, H, d, dv = self.hidden_size, self.num_heads, self.dim, self.vdim
        return {"q.weight": TensorSpec((H * d, h)), "k.weight": TensorSpec((H * d, h)),
                "v.weight": TensorSpec((H * dv, h)), "g.weight": TensorSpec((H * dv, h)),
                "norm.weight": TensorSpec((H * dv,), dtype="float32", init="one_plus_normal"),
                "o.weight": TensorSpec((h, H * dv))}

    def load(self, tensors):
        self.w_in = torch.cat([tensors["q.weight"], tensors["k.weight"], tensors["v.weight"],
                               tensors["g.weight"]], dim=0).contiguous()
        self.w_o, self.gain = tensors["o.weight"], tensors["norm.weight"]
        self.decay = torch.tensor(self.decay_values, dtype=torch.float32, device=self.w_o.device)

    def forward(self, ctx, x, cache, state):
        H, d, dv = self.num_heads, self.dim, self.vdim
        proj = ops.linear(x, self.w_in, out_dtype=torch.float32)  # [T, q | k | v | g]
        o = rec_ops.linear_recurrence(
            proj, 0, H * d, 2 * H * d, rec_ops.FIXED_DECAY, H, d, dv, state.buffer, state.slots, ctx.q_start,
            ctx.positions, decay=self.decay, silu_inputs=True)
        gated = norm32_ops.head_norm_gate(o, 1, self.eps, x.dtype, gain=self.gain,
                                          gate=proj[:, 2 * H * d + H * dv:], gate_kind="sigmoid")
        return ops.linear(gated, self.w_o, out_dtype=torch.float32)


@register_part("mixer", "gated_linear_attention")
class GatedLinearAttention(_MatrixStateMixer):
    def __init__(self, hidden_size: int, num_heads: int, dim: int, vdim: int, rank: int, tau: float, eps: float):
        super().__init__(hidden_size, num_heads, dim, vdim, eps)
        if rank <= 0 or not float(tau) > 0.0:
            raise ValueError(f"gated_linear_attention: rank={rank} and tau={tau} must be positive")
        self.rank, self.tau = int(rank), float(tau)
        self.gate_map = self.gate_bias = self.gain = None

    def tensor_specs(self):
        h, H, d, dv, r = self.hidden_size, self.num_heads, self.dim, self.vdim, self.rank
        return {"q.weight": TensorSpec((H * d, h)), "k.weight": TensorSpec((H * d, h)), "v.weight": TensorSpec((H * dv, h)),
                "g.weight": TensorSpec((H * dv, h)), "o.weight": TensorSpec((h, H * dv)),
                "a1.weight": TensorSpec((r, h)), "a2.weight": TensorSpec((H * d, r), dtype="float32"),
                "a2.bias": TensorSpec((H * d,), dtype="float32", init="zeros"),
                "norm.weight": TensorSpec((dv,), dtype="float32", init="one_plus_normal")}

    def load(self, tensors):
        self.w_in = torch.cat([tensors[n + ".weight"] for n in ("q", "k", "v", "g", "a1")], dim=0).contiguous()
        self.gate_map = tensors["a2.weight"].t().contiguous()  # [rank, H * dim]
        self.gate_bias, self.gain, self.w_o = tensors["a2.bias"], tensors["norm.weight"], tensors["o.weight"]

    def forward(self, ctx, x, cache, state):
        H, d, dv = self.num_heads, self.dim, self.vdim
        proj = ops.linear(x, self.w_in, out_dtype=torch.float32)  # [T, q | k | v | g | a1]
        v_off, g_off = 2 * H * d, 2 * H * d + H * dv
        o = rec_ops.linear_recurrence(
            proj, 0, H * d, v_off, rec_ops.KEY_DECAY, H, d, dv, state.buffer, state.slots, ctx.q_start, ctx.positions,
            gate_map=self.gate_map, gate_bias=self.gate_bias, low_off=g_off + H * dv, q_scale=d ** -0.5,
            power=1.0 / self.tau)
        gated = norm32_ops.head_norm_gate(o, H, self.eps, x.dtype, gain=self.gain, gate=proj[:, g_off:g_off + H * dv])
        return ops.linear(gated, self.w_o, out_dtype=torch.float32)


@register_part("mixer", "delta")
class GatedDelta(JoinableMixer):
    UNIT_EPS = 1e-6  # inside the root of a head's length

    def __init__(self, hidden_size: int, num_heads: int, num_kv_heads: int, dim: int, vdim: int, taps: int, eps: float):
        if min(hidden_size, num_heads, num_kv_heads, dim, vdim, taps) <= 0 or num_heads % num_kv_heads:
            raise ValueError(f"delta: {num_heads} heads over {num_kv_heads} of {dim} and {vdim}, {taps} taps, do not describe a mixer")
        if dim > 512:
            raise ValueError(f"delta: a state of {dim} rows is more than the kernels hold (512)")
        self.hidden_size, self.num_heads, self.num_kv_heads, self.dim, self.vdim = hidden_size, num_heads, num_kv_heads, dim, vdim
        self.taps, self.eps = int(taps), float(eps)
        self.channels = 2 * num_kv_heads * dim + num_heads * vdim
        self.out_columns = num_heads * vdim
        self.w_conv = self.step_bias = self.a_log = self.gain = None

    def tensor_specs(self):
        h, H, G, d, dv, f32 = self.hidden_size, self.num_heads, self.num_kv_heads, self.dim, self.vdim, "float32"
        specs = {"g.weight": TensorSpec((H * dv, h)), "b.weight": TensorSpec((H, h)), "a.weight": TensorSpec((H, h)),
                 "o.weight": TensorSpec((h, H * dv)), "A_log": TensorSpec((H,), dtype=f32), "step.bias": TensorSpec((H,), dtype=f32),
                 "norm.weight": TensorSpec((dv,), dtype=f32, init="one_plus_normal")}
        for name, n in (("q", G * d), ("k", G * d), ("v", H * dv)):
            specs[name + ".weight"] = TensorSpec((n, h))
            specs[name + ".conv"] = TensorSpec((n, self.taps), dtype=f32, init="one_plus_normal")
        return specs

    def load(self, tensors):
        # one product: [q | k | v | gate | b | a], padded to whole groups of eight columns
        rows = [tensors[n + ".weight"] for n in ("q", "k", "v", "g", "b", "a")]
        pad = -sum(r.shape[0] for r in rows) % 8
        self.w_in = torch.cat(rows + [rows[0].new_zeros((pad, self.hidden_size))], dim=0).contiguous()
        self.w_conv = torch.cat([tensors[n + ".conv"] for n in "qkv"], dim=0).t().contiguous()  # [taps, channels]
        self.step_bias, self.a_log, self.gain, self.w_o = (tensors[n] for n in ("step.bias", "A_log", "norm.weight", "o.weight"))

    def state_need(self):
        matrix = StateNeed((self.num_heads, self.dim, self.vdim), "float32")
        return (matrix,) if self.taps == 1 else (matrix, StateNeed((self.taps - 1, self.channels), "float32"))

    def tokens_per_attention_tile(self):
        return rec_ops.DELTA_RUN  # the runs of a portion

    def heads(self, ctx, z, cache, state, out):
        H, G, d, dv, n = self.num_heads, self.num_kv_heads, self.dim, self.vdim, self.channels
        b_off = n + H * dv
        rows, steps = conv_ops.conv_heads(z, self.w_conv, state[1].buffer if self.taps > 1 else None, ctx, G, G, d, H, dv,
                                          self.UNIT_EPS, d ** -0.5, b_off, b_off + H, self.step_bias, self.a_log)
        o = rec_ops.delta_rule(ctx, rows, steps, H, G, d, dv, state[0].buffer)
        norm32_ops.head_norm_gate(o, H, self.eps, out.dtype, gain=self.gain, gate=z[:, n:b_off], out=out)
