"""Interfaces of the parts a decoder is assembled from.

A part owns its sizes and constants (constructor arguments), declares the tensors it
needs (``tensor_specs``), receives them once (``load``) and runs on a flat batch of
tokens described by a ``StepContext``.  No part knows which model it is in: what it
needs from outside arrives as an argument (another part object, a cache view, a state
view).

Roles and their required methods:

* ``Norm.forward(ctx, x, rows=None) -> y`` and
  ``Norm.forward_add(ctx, residual, delta) -> y`` (adds ``delta`` into ``residual`` in
  place in 32-bit, then normalises the sum).
* ``PositionEncoding.rotation() -> Rotation(inv_freq, rotary_dim) | None`` and
  ``PositionEncoding.score_scale() -> float``: what the attention mixer asks of it.
* ``Mixer.forward(ctx, x, cache, state) -> y``; ``cache_need()`` says which named tensors
  a call of this mixer keeps per token in the paged cache (or None), ``state_need()`` what
  fixed-size per-request state (a need, a tuple of them, or None; ``state`` is then a view, a tuple of
  views, or None).
* ``FeedForward.forward(ctx, x) -> y``.
* ``Block.forward(ctx, x, cache, state) -> x``: the arrangement of two norms, a mixer
  and a feed-forward with their residual sums.
"""
from __future__ import annotations

from dataclasses import dataclass, field
from typing import Any

import torch

from dispec_b200 import ops
from dispec_b200.cache.manager import CacheTensor, key_value_tensors  # noqa: F401  (CacheTensor re-exported)


@dataclass(frozen=True)
class TensorSpec:
    """Shape and storage class of one tensor a part needs.

    ``dtype``: "model" follows the engine (bfloat16, or float32 on the 32-bit path);
    "float32" stays 32-bit in every mode; "int32" is an integer table.
    ``init`` tells the random-weights mode how to draw it: "normal" is N(0, std),
    "one_plus_normal" is 1 + N(0, std) (gains), "zeros" is 0.
    """
    shape: tuple[int, ...]
    dtype: str = "model"
    init: str = "normal"


@dataclass(frozen=True)
class PartSpec:
    """Declarative description of one part: registered kind, constructor parameters,
    and the checkpoint tensor name behind each of the part's local tensor names."""
    role: str
    kind: str
    params: dict[str, Any] = field(default_factory=dict)
    tensors: dict[str, str] = field(default_factory=dict)  # local name -> checkpoint name


@dataclass(frozen=True)
class CacheNeed:
    """What one mixer call keeps per token in the paged cache: a tuple of named tensors
    (``CacheTensor(name, num_heads, width)``), each with its own heads and width.  Ordinary
    attention keeps two of equal shape, "key" and "value" (``CacheNeed.key_value``); a mixer
    that caches one latent tensor, or keys and values of different widths, lists those instead
    and finds them by name in ``LayerCacheView.tensors``.  ``window`` 0: every token stays;
    W > 0: only the last W positions are ever read (and the ``keep_first`` first ones), other pages
    can be given back."""
    tensors: tuple
    window: int = 0
    keep_first: int = 0

    @classmethod
    def key_value(cls, num_kv_heads: int, head_dim: int, window: int = 0) -> "CacheNeed":
        return cls(key_value_tensors(num_kv_heads, head_dim), window)


@dataclass(frozen=True)
class StateNeed:
    """Fixed-size per-request state of one mixer call: a tensor of ``shape`` per live
    request, zeroed when a request is admitted."""
    shape: tuple[int, ...]
    dtype: str = "float32"


@dataclass
class WideStream:
    """A residual stream kept in 32-bit floats (``full``, [T, width]) beside the copy rounded to
    the model type that the products read (``rounded``; the same tensor on the 32-bit path; None
    where the arrangement reads the stream through a norm only and keeps no such copy).
    Blocks that keep the stream this way pass it on as their ``x``; a norm that takes it
    (``rms_norm_f32``) reads ``full``."""
    full: torch.Tensor
    rounded: torch.Tensor | None

    @property
    def shape(self):
        return self.full.shape


class Part:
    role = ""
    kind = ""
    # False for a part whose forward decides things on the host from the step's values (such a
    # part cannot be replayed from a captured graph; the runner then runs every step eagerly)
    graph_safe = True

    def tensor_specs(self) -> dict[str, TensorSpec]:
        return {}

    def load(self, tensors: dict[str, torch.Tensor]) -> None:
        if tensors:
            raise ValueError(f"{type(self).__name__} takes no tensors")


class Norm(Part):
    def forward(self, ctx, x, rows=None):
        raise NotImplementedError

    def forward_add(self, ctx, residual, delta):
        raise NotImplementedError


@dataclass(frozen=True)
class Rotation:
    """Rotation of query and key heads: pair i of every head is turned by the angle
    position * inv_freq[i]; dimensions from ``rotary_dim`` on pass unchanged.  ``layout`` says
    which dimensions form pair i: "halves" (i, i + rotary_dim/2) or "interleaved" (2i, 2i+1).
    ``magnitude``: a factor on cosine and sine (1: a pure rotation); a mixer whose kernels do not
    apply it refuses an encoding that has one."""
    inv_freq: Any  # float32 [rotary_dim / 2] on the device
    rotary_dim: int
    layout: str = "halves"
    magnitude: float = 1.0


class PositionEncoding(Part):
    """What a mixer asks of its position encoding.  ``rotation()``: how it turns queries and
    keys before the scores (None: not at all).  ``score_scale()``: a factor the encoding puts on
    the attention scores beside the mixer's own scale.  ``prepare(device)`` (optional) builds
    device tables once the weights are loaded.  An encoding of another kind (an offset added to
    the stream, a bias on the scores) adds a method of its own and is consumed by a mixer that
    knows that method; the built-in attention mixer uses the two below."""

    def rotation(self) -> Rotation | None:
        return None

    def score_scale(self) -> float:
        return 1.0


class Mixer(Part):
    def cache_need(self) -> CacheNeed | None:
        return None

    def state_need(self) -> StateNeed | tuple | None:
        return None

    def tokens_per_attention_tile(self):
        """Query tokens per attention tile this mixer wants listed in the batch: an int, a tuple
        of them (one tile list each), or None."""
        return None

    def forward(self, ctx, x, cache, state):
        raise NotImplementedError


class JoinableMixer(Mixer):
    """A mixer of the form W_o f(W_in h + b_in) + b_o: one product into its rows, something of its own on
    those rows (``heads``), one product out of them.  Another mixer can run several of these side by
    side as one: their input matrices stacked, each one's ``heads`` on its columns, their output
    matrices joined along the input dimension (the sum over the mixers is then part of that product).
    A block can join a mixer with a feed-forward that reads the same rows in the same way.

    ``load`` sets ``w_in`` [columns, hidden], ``b_in`` (or None), ``w_o`` [hidden, out_columns] and ``b_o``
    (or None).  ``out_scale``: a factor on the mixer's result, set before ``load`` where the class says
    ``takes_out_scale``; ``heads`` applies it in 32-bit."""
    out_scale = 1.0
    takes_out_scale = False
    out_columns = 0
    w_in = b_in = w_o = b_o = None

    def heads(self, ctx, z, cache, state, out):
        """From the rows ``z`` [T, columns] of the input product (float32) to ``out`` [T, out_columns]."""
        raise NotImplementedError

    def forward(self, ctx, x, cache, state):
        z = ops.linear(x, self.w_in, self.b_in, out_dtype=torch.float32)
        out = torch.empty((x.shape[0], self.out_columns), dtype=x.dtype, device=x.device)
        self.heads(ctx, z, cache, state, out)
        return ops.linear(out, self.w_o, self.b_o, out_dtype=torch.float32)


class FeedForward(Part):
    def forward(self, ctx, x):
        raise NotImplementedError


class Block(Part):
    def forward(self, ctx, x, pending, cache, state):
        raise NotImplementedError
