"""Short causal convolutions over time with their last inputs in the request's state slot.  See
``csrc/short_conv.cu``."""
from __future__ import annotations

import torch

from dispec_b200.ops import library as L


def _lib():
    return L.mixer_library("short_conv")


def _check(u, weight, channels, ctx_arrays, hist):
    if not u.is_cuda:
        raise L.KernelError("short convolution: CUDA tensors only (there is no CPU path)")
    assert u.dim() == 2 and u.stride(1) == 1
    taps = 1
    if weight is not None:
        assert weight.dtype == torch.float32 and weight.is_contiguous() and weight.shape[1] == channels
        taps = weight.shape[0]
    if taps > 1:
        assert hist is not None and hist.dtype == torch.float32 and hist.is_contiguous()
        assert hist.shape[1:] == (taps - 1, channels)
    for t in ctx_arrays:
        assert t.dtype == torch.int32 and t.is_contiguous()
    return taps


def conv_steps(u: torch.Tensor, offset: int, weight: torch.Tensor, bias: torch.Tensor | None, hist: torch.Tensor | None,
               ctx, step_offset: int = 0, step_bias: torch.Tensor | None = None, a_log: torch.Tensor | None = None):
    """silu(conv + bias) of the columns ``offset`` .. + channels of ``u`` [T, columns], as float32
    [T, channels]; ``weight`` float32 [taps, channels] (last row: the current token's), ``hist`` float32
    [slots, taps - 1, channels] the last inputs of every request (None with one tap).  With
    ``step_bias`` / ``a_log`` (float32 [heads]): also float32 [T, 2, heads] of step = softplus(u[:, step_offset + h]
    + step_bias) and exp(-exp(a_log) * step).  ``ctx``: the step's arrays.  Rows with a negative
    position are skipped."""
    channels = weight.shape[1]
    taps = _check(u, weight, channels, (ctx.state_slot, ctx.q_start, ctx.seq_of_token, ctx.positions), hist)
    assert 0 <= offset and offset + channels <= u.shape[1]
    assert bias is None or (bias.dtype == torch.float32 and bias.shape == (channels,) and bias.is_contiguous())
    T = u.shape[0]
    out = torch.empty((T, channels), dtype=torch.float32, device=u.device)
    heads, steps = 0, None
    if step_bias is not None:
        heads = step_bias.shape[0]
        assert step_bias.dtype == a_log.dtype == torch.float32 and a_log.shape == (heads,)
        assert 0 <= step_offset and step_offset + heads <= u.shape[1]
        steps = torch.empty((T, 2, heads), dtype=torch.float32, device=u.device)
    L.check(_lib().dsp_conv_steps(
        L.ptr(u), L.dtype_code(u.dtype), L.i64(u.stride(0)), offset, channels, taps, L.ptr(weight), L.ptr(bias),
        L.ptr(hist), L.ptr(ctx.state_slot), L.ptr(ctx.q_start), L.ptr(ctx.seq_of_token), L.ptr(ctx.positions), L.ptr(out),
        L.i64(out.stride(0)), step_offset, heads, L.ptr(step_bias), L.ptr(a_log), L.ptr(steps), T, L.stream_handle()))
    return out, steps


def qkv_conv_rotate_store(u: torch.Tensor, weight: torch.Tensor | None, hist: torch.Tensor | None, ctx, cache,
                          inv_freq: torch.Tensor | None, rotary_dim: int, interleaved: bool, num_heads: int,
                          num_kv_heads: int, key_dim: int, value_dim: int, out_dtype: torch.dtype, head_norm: bool,
                          norm_eps: float, value_scale: float = 1.0) -> torch.Tensor:
    """From rows [q (H x Dk) | k (G x Dk) | v (G x Dv)] of a projection: every column through the
    convolution (``weight`` float32 [taps, columns], None: none; ``hist`` as in ``conv_steps``), queries and
    keys turned by position * inv_freq[i], pairs (2i, 2i + 1) with ``interleaved``, else (i, i +
    rotary_dim/2), then (``head_norm``) divided by their root mean square per head, ``norm_eps`` inside
    the root.  Keys and values (times ``value_scale``) go to the pages of ``cache``; returns the queries
    [T, H * Dk] in ``out_dtype``.  32-bit arithmetic; rows with a negative position are skipped."""
    H, G, dk, dv = num_heads, num_kv_heads, key_dim, value_dim
    channels = (H + G) * dk + G * dv
    taps = _check(u, weight, channels, (ctx.state_slot, ctx.q_start, ctx.seq_of_token, ctx.positions), hist)
    assert u.shape[1] == channels
    k_pool, v_pool, table = cache.key_pool, cache.value_pool, cache.page_table
    num_pages, g_, page_size, dk_ = k_pool.shape
    assert (g_, dk_) == (G, dk) and v_pool.shape == (num_pages, G, page_size, dv)
    assert k_pool.is_contiguous() and v_pool.is_contiguous() and k_pool.dtype == v_pool.dtype == out_dtype
    assert table.dtype == torch.int32 and table.stride(1) == 1
    if rotary_dim:
        assert inv_freq is not None and inv_freq.dtype == torch.float32 and inv_freq.shape[0] >= rotary_dim // 2
    T = u.shape[0]
    q = torch.empty((T, H * dk), dtype=out_dtype, device=u.device)
    L.check(_lib().dsp_qkv_conv_rotate_store(
        L.ptr(u), L.dtype_code(u.dtype), L.i64(u.stride(0)), taps, L.ptr(weight), L.ptr(hist), L.ptr(ctx.state_slot),
        L.ptr(ctx.q_start), L.ptr(ctx.seq_of_token), L.ptr(ctx.positions), L.ptr(table), table.stride(0), L.ptr(k_pool),
        L.ptr(v_pool), L.dtype_code(out_dtype), L.ptr(inv_freq), rotary_dim, int(bool(interleaved)), int(bool(head_norm)),
        L.f32(norm_eps), L.f32(value_scale), L.ptr(q), L.i64(q.stride(0)), T, H, G, dk, dv, page_size, num_pages,
        int(cache.write), L.stream_handle()))
    return q


def conv_heads(u: torch.Tensor, weight: torch.Tensor, hist: torch.Tensor | None, ctx, num_q: int, num_k: int, dim: int,
               num_v: int, vdim: int, eps: float, q_scale: float, beta_offset: int, decay_offset: int,
               step_bias: torch.Tensor, a_log: torch.Tensor):
    """From rows [q (num_q x dim) | k (num_k x dim) | v (num_v x vdim) | ...] of a projection: silu of every
    column's convolution (``weight`` float32 [taps, columns], ``hist`` as in ``conv_steps``), query and key heads
    divided by their length, x / sqrt(sum(x^2) + eps), queries then times ``q_scale``, as float32 rows of the same
    layout; and float32 [T, 2, num_v]: sigmoid(u[:, beta_offset + h]) and the logarithm of a decay,
    -exp(a_log) * softplus(u[:, decay_offset + h] + step_bias).  Rows with a negative position are skipped."""
    channels = (num_q + num_k) * dim + num_v * vdim
    taps = _check(u, weight, channels, (ctx.state_slot, ctx.q_start, ctx.seq_of_token, ctx.positions), hist)
    assert channels <= u.shape[1] and 0 <= beta_offset <= u.shape[1] - num_v and 0 <= decay_offset <= u.shape[1] - num_v
    for t in (step_bias, a_log):
        assert t.dtype == torch.float32 and t.shape == (num_v,) and t.is_contiguous() and t.is_cuda
    T = u.shape[0]
    out = torch.empty((T, (channels + 3) // 4 * 4), dtype=torch.float32, device=u.device)  # 16-byte rows
    steps = torch.empty((T, 2, num_v), dtype=torch.float32, device=u.device)
    L.check(_lib().dsp_conv_heads(
        L.ptr(u), L.dtype_code(u.dtype), L.i64(u.stride(0)), taps, L.ptr(weight), L.ptr(hist), L.ptr(ctx.state_slot),
        L.ptr(ctx.q_start), L.ptr(ctx.seq_of_token), L.ptr(ctx.positions), num_q, num_k, dim, num_v, vdim, L.f32(eps),
        L.f32(q_scale), L.ptr(out), L.i64(out.stride(0)), beta_offset, decay_offset, L.ptr(step_bias), L.ptr(a_log),
        L.ptr(steps), T, L.stream_handle()))
    return out[:, :channels], steps
