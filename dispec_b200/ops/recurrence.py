"""Linear attention as a recurrence over a per-request matrix state (32-bit, FMA units):
S_t = diag(a_t) S_(t-1) + b_t v_t^T,  o_t = S_t^T q_t  (``csrc/linear_recurrence.cu``), and the gated delta
rule, whose write depends on what the state already holds (``csrc/delta_rule.cu``)."""
from __future__ import annotations

import torch

from dispec_b200.ops import library as L

FIXED_DECAY, FORGET_GATE, KEY_DECAY, STEP_DECAY = 0, 1, 2, 3


def linear_recurrence(proj: torch.Tensor, q_off: int, k_off: int, v_off: int, mode: int, num_heads: int,
                      dim: int, vdim: int, state: torch.Tensor, state_slot: torch.Tensor,
                      q_start: torch.Tensor, positions: torch.Tensor, *, decay: torch.Tensor | None = None,
                      inv_freq: torch.Tensor | None = None, rot: int = 0, key_scale: float = 1.0,
                      gate_bias: torch.Tensor | None = None, lower: torch.Tensor | None = None,
                      silu_inputs: bool = False, gate_map: torch.Tensor | None = None, low_off: int = 0,
                      q_scale: float = 1.0, power: float = 1.0, steps: torch.Tensor | None = None,
                      skip: torch.Tensor | None = None, num_groups: int = 0) -> torch.Tensor:
    """``proj`` [T, columns]: the raw rows of the mixer's fused projection (query columns from
    ``q_off``, key or forget-gate columns from ``k_off``, value columns from ``v_off``, each head by
    head).  ``state`` float32 [slots, H, dim, vdim] is read and left updated for the sequences of the
    step (``q_start`` [S + 1], ``state_slot`` [S]); a sequence whose first position is negative is
    skipped.  ``silu_inputs`` (fixed decay only): the raw query, key and value columns pass through
    silu before anything else.  Returns o as float32 [T, H * vdim].

    ``KEY_DECAY``: query columns times ``q_scale``, key columns times ``key_scale``, and a decay per key
    channel sigmoid(z)^power with z = r ``gate_map`` + ``gate_bias``, r the columns of the row from
    ``low_off`` on and ``gate_map`` float32 [rank, H * dim].  ``STEP_DECAY``: ``proj`` float32; query and key
    columns (``dim`` for each of ``num_groups`` groups of heads) are shared by the heads of a group,
    ``steps`` float32 [T, 2, H] holds the factor on the value and the decay of every token and head, and
    ``skip`` float32 [H] times the value is added to o."""
    if not (proj.is_cuda and state.is_cuda):
        raise L.KernelError("linear_recurrence: CUDA tensors only (there is no CPU path)")
    assert proj.dim() == 2 and proj.stride(1) == 1
    assert state.dtype == torch.float32 and state.is_contiguous() and state.shape[1:] == (num_heads, dim, vdim)
    for t in (state_slot, q_start, positions):
        assert t.dtype == torch.int32 and t.is_contiguous()
    for t in (decay, inv_freq, gate_bias, lower, gate_map, steps, skip):
        assert t is None or (t.dtype == torch.float32 and t.is_contiguous() and t.is_cuda)
    S = state_slot.shape[0]
    assert q_start.shape[0] == S + 1
    T = proj.shape[0]
    rank, heads_per_group = 0, 1
    if mode == KEY_DECAY:
        rank = gate_map.shape[0]
        assert gate_map.shape == (rank, num_heads * dim) and gate_bias.shape == (num_heads * dim,)
        assert 0 <= low_off and low_off + rank <= proj.shape[1]
    if mode == STEP_DECAY:
        assert num_groups > 0 and num_heads % num_groups == 0 and proj.dtype == torch.float32
        assert steps.shape == (T, 2, num_heads) and skip.shape == (num_heads,)
        heads_per_group = num_heads // num_groups
    out = torch.empty((T, num_heads * vdim), dtype=torch.float32, device=proj.device)
    lib = L.mixer_library("linear_recurrence")
    # portions of prompts: a first, parallel kernel writes q_t, b_t (a_t) of every token as floats and
    # the sequential kernel streams them; steps of (nearly) single tokens transform while staging
    scratch = None
    if T > 2 * S and mode != STEP_DECAY:
        planes = 2 if mode == FIXED_DECAY else 3
        scratch = torch.empty((T, planes, num_heads * dim), dtype=torch.float32, device=proj.device)
    L.check(lib.dsp_linear_recurrence(
        L.ptr(proj), L.dtype_code(proj.dtype), L.i64(proj.stride(0)), q_off, k_off, v_off, mode, num_heads, dim,
        vdim, L.ptr(decay), L.ptr(inv_freq), rot, L.f32(key_scale), int(silu_inputs), L.ptr(gate_bias), L.ptr(lower),
        L.ptr(gate_map), low_off, rank, L.f32(q_scale), L.f32(power), L.ptr(steps), L.ptr(skip), heads_per_group, L.ptr(state),
        L.ptr(state_slot), L.ptr(q_start), L.ptr(positions), L.ptr(out), L.i64(out.stride(0)), S, T,
        L.ptr(scratch), L.stream_handle()))
    return out


DELTA_RUN = 8  # tokens of a portion that the delta rule takes together: the step lists its runs like attention tiles
_DELTA_COEF = 20
_DELTA_MAX_WALK = 256  # state rows up to which portions are taken in runs


def delta_rule(ctx, rows: torch.Tensor, steps: torch.Tensor, num_heads: int, num_groups: int, dim: int, vdim: int,
               state: torch.Tensor) -> torch.Tensor:
    """S <- g S; u = beta (v - S^T k); S <- S + k u^T; o = S^T q for every token of the step, in order.

    ``rows`` float32 [T, columns]: q and k (``num_groups`` x ``dim`` each) and v (``num_heads`` x ``vdim``) side by
    side; head h uses q and k of group h // (num_heads / num_groups).  ``steps`` float32 [T, 2, H]: beta and ln g.
    ``state`` float32 [slots, H, dim, vdim] is read and left updated for the step's requests (``ctx``: the
    step's arrays, with its list of runs of ``DELTA_RUN`` tokens); a request whose first position is
    negative is skipped.  Returns o as float32 [T, H * vdim]."""
    if not (rows.is_cuda and state.is_cuda):
        raise L.KernelError("delta_rule: CUDA tensors only (there is no CPU path)")
    H, G, T, S = num_heads, num_groups, rows.shape[0], ctx.state_slot.shape[0]
    assert rows.dtype == torch.float32 and rows.dim() == 2 and rows.stride(1) == 1
    assert rows.shape[1] == 2 * G * dim + H * vdim and H % G == 0
    assert steps.dtype == torch.float32 and steps.shape == (T, 2, H) and steps.is_contiguous()
    assert state.dtype == torch.float32 and state.is_contiguous() and state.shape[1:] == (H, dim, vdim)
    for t in (ctx.state_slot, ctx.q_start, ctx.positions):
        assert t.dtype == torch.int32 and t.is_contiguous()
    out = torch.empty((T, H * vdim), dtype=torch.float32, device=rows.device)
    run_seq, run_tok0, num_runs = ctx.attention_tiles[DELTA_RUN]
    coef = None
    if T > ctx.num_decode_seqs and dim <= _DELTA_MAX_WALK:
        coef = torch.empty((T, H, _DELTA_COEF), dtype=torch.float32, device=rows.device)
    L.check(L.mixer_library("delta_rule").dsp_delta_rule(
        L.ptr(rows), L.i64(rows.stride(0)), 0, G * dim, 2 * G * dim, L.ptr(steps), H, G, dim, vdim, L.ptr(state),
        L.ptr(ctx.state_slot), L.ptr(ctx.q_start), L.ptr(ctx.positions), L.ptr(run_seq), L.ptr(run_tok0), num_runs,
        L.ptr(out), L.i64(out.stride(0)), S, ctx.num_decode_seqs, L.ptr(coef), L.stream_handle()),
        launches=(1 if ctx.num_decode_seqs or coef is None else 0) + (2 if coef is not None else 0))
    return out
