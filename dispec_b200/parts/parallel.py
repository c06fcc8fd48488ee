"""``parallel``: two mixers side by side on the same input,

    y = left_scale * left(h) + right_scale * right(h).

Both are joinable mixers (``JoinableMixer``): their input matrices are stacked into one product, each runs
its own middle part on its columns, and their output matrices are joined along the input dimension,
so that the sum is part of the output product.  The factors are applied by the mixers themselves, in
32-bit, on the rows in front of that product.  At most one of the two keeps tokens in the paged cache."""
from __future__ import annotations

import torch

from dispec_b200 import ops
from dispec_b200.parts.base import JoinableMixer, Mixer
from dispec_b200.registry import register_part


def _needs(mixer) -> tuple:
    need = mixer.state_need()
    return need if isinstance(need, tuple) else ((need,) if need is not None else ())


@register_part("mixer", "parallel")
class ParallelMixer(Mixer):
    def __init__(self, left, right, left_scale: float = 1.0, right_scale: float = 1.0):
        for m in (left, right):
            if not isinstance(m, JoinableMixer):
                raise ValueError(f"parallel: {type(m).__name__} cannot be joined with another mixer")
        if left.cache_need() is not None and right.cache_need() is not None:
            raise ValueError("parallel: only one of the two mixers can keep tokens in the paged cache")
        for m, factor in ((left, left_scale), (right, right_scale)):
            if float(factor) != 1.0 and not m.takes_out_scale:
                raise ValueError(f"parallel: {type(m).__name__} takes no factor on its result")
        self.mixers = (left, right)
        left.out_scale, right.out_scale = float(left_scale), float(right_scale)
        self.w_in = self.b_in = self.w_o = self.b_o = None

    def prepare(self, device):
        """Joins the two mixers' matrices (they are loaded by now) and lets go of the single ones."""
        left, right = self.mixers
        if any(m.b_in is not None for m in self.mixers):
            self.b_in = torch.cat([m.b_in if m.b_in is not None else
                                   torch.zeros(m.w_in.shape[0], dtype=m.w_in.dtype, device=m.w_in.device) for m in self.mixers])
        self.columns = (left.w_in.shape[0], right.w_in.shape[0])
        self.w_in = torch.cat([left.w_in, right.w_in], dim=0).contiguous()
        self.w_o = torch.cat([left.w_o, right.w_o], dim=1).contiguous()
        biases = [m.b_o for m in self.mixers if m.b_o is not None]
        if len(biases) == 2:
            raise ValueError("parallel: only one of the two mixers can have an output bias")
        self.b_o = biases[0] if biases else None
        for m in self.mixers:
            m.w_in = m.b_in = m.w_o = m.b_o = None

    def cache_need(self):
        return self.mixers[0].cache_need() or self.mixers[1].cache_need()

    def state_need(self):
        return _needs(self.mixers[0]) + _needs(self.mixers[1]) or None

    def tokens_per_attention_tile(self):
        tiles = []
        for m in self.mixers:
            want = m.tokens_per_attention_tile()
            tiles += list(want) if isinstance(want, (tuple, list)) else [want] if want else []
        return tuple(tiles) or None

    def forward(self, ctx, x, cache, state):
        z = ops.linear(x, self.w_in, self.b_in, out_dtype=torch.float32)
        inner = self.w_o.shape[1]
        out = torch.empty((x.shape[0], (inner + 7) // 8 * 8), dtype=x.dtype, device=x.device)[:, :inner]  # 16-byte rows
        col = row = first = 0
        for m, n in zip(self.mixers, self.columns):
            count = len(_needs(m))
            own = state[first:first + count] if count else None
            if count and not isinstance(m.state_need(), tuple):
                own = own[0]
            m.heads(ctx, z[:, col:col + n], cache if m.cache_need() is not None else None, own,
                    out[:, row:row + m.out_columns])
            col, row, first = col + n, row + m.out_columns, first + count
        return ops.linear(out, self.w_o, self.b_o, out_dtype=torch.float32)
