"""Interfaces of the parts a layer is put together from, and one registry for each family.

A part is built from a :class:`~ginfer_b200.parts.plan.PartSpec` (``kind`` plus parameters), says
which tensors it needs (:meth:`Part.tensor_specs`), receives them (:meth:`Part.load`) and runs on
the tokens of one step.  No part knows which model it is in: sizes and constants arrive as
constructor parameters, per-step facts arrive in a :class:`StepContext`, and a mixer's cache
arrives as a binding made by the cache manager.
"""
from __future__ import annotations

from dataclasses import dataclass, field
from typing import Any, Callable

import torch

from .plan import PartSpec


# ----------------------------------------------------------------------------- tensors of a part
@dataclass(frozen=True)
class TensorSpec:
    """A tensor a part needs.  ``name`` is relative to the part's scope (the layer prefix).
    ``role`` decides how it is kept and how random weights are drawn:

    * ``matrix`` / ``embedding``: operands of matrix products, kept in the compute dtype;
      drawn N(0, 0.02).
    * ``bias``: kept in the compute dtype unless stored in 32-bit, which stays; N(0, 0.02).
    * ``norm``: like ``bias`` but drawn 1 + N(0, 0.02).
    * ``f32``: a small tensor that enters 32-bit arithmetic (a router, decay constants, norm
      weights stored around zero); always kept in 32-bit; N(0, 0.02).
    * ``norm32``: a norm weight that is always kept in 32-bit; drawn 1 + N(0, 0.02).
    * ``int``: integer table, kept as int32; drawn uniform in ``[0, int_high)``.

    A size of ``-1`` in ``shape`` stands for "whatever the file has" (a rank that only the
    tensor's own shape gives); random weights cannot be drawn for such a tensor.

    A name that starts with ``/`` is a tensor of the whole model, not of the part's scope: it is
    looked up without the layer prefix, and several parts may name the same one (a table that
    every layer reads a slice of).
    """
    name: str
    shape: tuple[int, ...]
    role: str = "matrix"
    int_high: int = 2


# ----------------------------------------------------------------------------- caches of a mixer
@dataclass(frozen=True)
class PagedKVSpec:
    """What a mixer keeps of every position (``window == 0``) or of the last ``window``
    positions (or, with ``chunk``, of the chunk the sequence is in), in pages.  By default keys and values of ``num_kv_heads`` heads of ``head_dim``
    each.  ``planes`` names another lay-out: one ``(heads, width)`` per tensor kept of a token
    (one latent vector: ``((1, width),)``; keys and values of different widths:
    ``((heads, k_width), (heads, v_width))``)."""
    num_kv_heads: int
    head_dim: int
    window: int = 0
    planes: tuple[tuple[int, int], ...] | None = None
    chunk: int = 0        # > 0: a query sees only the keys of its own chunk of this many positions

    def layout(self) -> tuple[tuple[int, int], ...]:
        return self.planes or ((self.num_kv_heads, self.head_dim),) * 2


@dataclass(frozen=True)
class StateSpec:
    """Per-request state of fixed size, kept in a slot; zeroed when a request takes the slot."""
    shape: tuple[int, ...]
    dtype: torch.dtype = torch.float32


@dataclass
class PagedKVBinding:
    # [2, num_pages, page_size, num_kv_heads, head_dim] (0 = K, 1 = V); for a spec with ``planes``
    # a tuple of tensors [num_pages, page_size, heads, width], one per plane
    pages: torch.Tensor | tuple
    block_table: torch.Tensor    # [B, W] int32, logical page -> physical page, -1 where none
    slot_mapping: torch.Tensor   # [T] int32, physical token slot (page * page_size + offset)
    page_size: int
    window: int
    write: bool
    chunk: int = 0


@dataclass
class StateBinding:
    state: torch.Tensor          # [num_slots, *shape]
    write: bool


# ----------------------------------------------------------------------------- per-step facts
@dataclass
class StepContext:
    """What one step's batch looks like.  Tokens of all requests are packed: request ``b`` owns
    rows ``cu_seqlens_q[b]:cu_seqlens_q[b+1]``; its tokens sit at absolute positions
    ``q_starts[b] ...`` and after the step the request holds ``kv_lens[b]`` tokens."""
    num_tokens: int
    num_seqs: int
    dtype: torch.dtype
    device: torch.device
    token_ids: torch.Tensor       # [T] int32 (device)
    positions: torch.Tensor       # [T] int32 (device)
    seq_of_token: torch.Tensor    # [T] int32 (device)
    cu_seqlens_q: torch.Tensor    # [B+1] int32 (device)
    kv_lens: torch.Tensor         # [B] int32 (device)
    slot_ids: torch.Tensor        # [B] int32 (device): per-request state slot
    logit_rows: torch.Tensor      # [R] int32 (device): rows whose logits are wanted
    q_lens_host: list[int] = field(default_factory=list)
    q_starts_host: list[int] = field(default_factory=list)
    slot_ids_host: list[int] = field(default_factory=list)
    max_q_len: int = 0
    max_kv_len: int = 0
    decode_only: bool = False
    all_rows_wanted: bool = False  # logit_rows is every row of the step, in order
    capturing: bool = False       # inside CUDA-graph capture: no host syncs, no allocation tricks
    extras: dict[str, Any] = field(default_factory=dict)


# ----------------------------------------------------------------------------- folded norms
@dataclass
class Summed:
    """A hidden state whose last residual addition is done: ``tensor [T, H]`` in fp32, with the
    partial sums of squares of its rows that the product which formed it left behind
    (``sumsq [parts, ld]``), so that a following RMS normalisation needs no pass of its own.
    ``scaled`` is ``tensor * gamma`` in the activation dtype for the norm whose weight is
    ``scaled_by`` (the norm the producer was told comes next), or ``None``."""
    tensor: torch.Tensor
    sumsq: torch.Tensor
    scaled: torch.Tensor | None = None
    scaled_by: torch.Tensor | None = None


@dataclass
class LazyNorm:
    """The RMS normalisation of a :class:`Summed` state, not computed yet: what is there is
    ``scaled = tensor * gamma`` and the sums of squares, and ``norm = scaled / rms`` row by row.
    A product that can multiply its accumulator by ``1 / rms`` takes it as it is (``x W^T / rms``
    is the product of the normalised rows); anything else calls :meth:`materialize`."""
    summed: Summed
    gamma: torch.Tensor
    eps: float
    dtype: torch.dtype

    @property
    def scaled(self) -> torch.Tensor | None:
        s = self.summed
        return s.scaled if s.scaled_by is self.gamma else None

    def materialize(self) -> torch.Tensor:
        from .. import ops
        return ops.add_rmsnorm(self.summed.tensor, None, self.gamma, self.eps, want_sum=False,
                               out_dtype=self.dtype)[1]


@dataclass
class PairSum:
    """The output of a routed feed-forward, not added up yet: ``rows [P, H]`` fp32 holds a row per
    (token, choice) pair in sorted order, pair ``t * top + k`` sits at ``pos_of_pair[t * top + k]``
    and a token's output is the sum of its pairs' rows times ``weights [T, top]`` (``None``: 1).
    A kernel that adds the output to the stream can add the pairs up itself; anything else calls
    :meth:`materialize`."""
    rows: torch.Tensor
    pos_of_pair: torch.Tensor
    weights: torch.Tensor | None
    top: int
    materialize: Callable[[], torch.Tensor]


@dataclass
class TermSum:
    """The output of a sublayer that is a sum, not added up yet: dense ``terms`` ``(tensor [T, H],
    constant, factors [T] fp32 or None)`` (the first one fp32, a second one fp32 or the activation
    dtype) and a routed feed-forward's ``pairs``.  A kernel that adds the output to the stream can form
    the sum itself; anything else calls :meth:`materialize`."""
    terms: list
    pairs: PairSum | None = None

    def kernel_args(self) -> dict:
        p = self.pairs
        return dict(terms=self.terms,
                    pairs=None if p is None else (p.rows, p.pos_of_pair, p.weights, p.top))

    def materialize(self) -> torch.Tensor:
        from ..ops import hyper
        some = self.terms[0][0] if self.terms else self.pairs.rows
        one = torch.ones(1, dtype=torch.float32, device=some.device)
        return hyper.update(None, 1, torch.float32, out_w=one, **self.kernel_args())[0][:, 0]


@dataclass
class MixedInput:
    """What the first sublayer of a run reads, where the model carries several residual streams: the
    norm of their sum with the fp32 ``weights [streams]``.  It takes the place of the plain norm where
    another block prepares a run's input (``then``)."""
    norm: "Norm"
    weights: torch.Tensor


@dataclass
class ShiftedInput:
    """What the first sublayer of a run reads, where that is a norm of the stream shifted towards
    the token before: ``n_t + (n_(t-1) - n_t) * weight`` with ``n = norm(x)`` and ``weight`` fp32
    ``[H]``; ``state`` holds ``n`` of the last token of earlier steps, a row a slot.  It takes the
    place of the plain norm where another block prepares a run's input (``then``)."""
    norm: "Norm"
    weight: torch.Tensor
    state: StateBinding


# ----------------------------------------------------------------------------- part interfaces
class Part:
    """Base of every part."""

    def tensor_specs(self) -> list[TensorSpec]:
        return []

    def load(self, tensors: dict[str, torch.Tensor], dtype: torch.dtype,
             device: torch.device) -> None:
        """Receive the tensors named by :meth:`tensor_specs` (already on ``device``)."""


class Norm(Part):
    def forward(self, x: torch.Tensor, delta: torch.Tensor | None = None,
                rows: torch.Tensor | None = None, want_sum: bool = True, out_dtype=None
                ) -> tuple[torch.Tensor | None, torch.Tensor]:
        """Return ``(s, norm(s))`` with ``s = x + delta`` (``s = x`` if ``delta`` is None), the
        sum formed in 32-bit.  ``rows`` (int32) selects rows of ``x``/``delta`` first.  ``s`` is
        None when ``want_sum`` is false.  ``out_dtype``: the activation dtype of ``norm(s)`` when
        it cannot be read off ``delta`` or ``x``."""
        raise NotImplementedError

    def lazy(self, summed: Summed, dtype: torch.dtype) -> LazyNorm | None:
        """The normalisation of ``summed`` as a :class:`LazyNorm`, if this norm can be folded
        into the product that consumes it; ``None`` otherwise."""
        return None

    def fused(self) -> tuple | None:
        """``(kind, weight, bias or None, eps)`` with fp32 tensors if the kernel that updates a
        32-bit stream can apply this norm in the same pass (``ops.prenorm.NORM_LAYER`` /
        ``NORM_RMS``); ``None`` (the default) if it cannot."""
        return None

    def fold_weight(self) -> torch.Tensor | None:
        """The weight ``gamma`` if this norm is ``x * gamma / rms(x)`` and so can be split into a
        multiplication by ``gamma`` in the product before it and one by ``1 / rms`` in the product
        behind it; ``None`` (the default) if it cannot."""
        return None


class PositionEncoding(Part):
    def rotary_table(self) -> tuple[torch.Tensor, int] | None:
        """``(table, rotary_dim)`` if the mixer's cache-write kernel can apply the encoding:
        ``table [max_positions, rotary_dim]`` fp32 holds cos in its first half of columns and sin
        in its second, and the first ``rotary_dim`` channels of every head are rotated in pairs
        ``(j, j + rotary_dim/2)``; ``(None, 0)`` means nothing is to be done.  ``None`` (the
        default) means the encoding has code of its own and :meth:`apply` is called instead."""
        return None

    def apply(self, q: torch.Tensor, k: torch.Tensor, ctx: StepContext) -> None:
        """Encode positions in place in ``q [T, heads, head_dim]`` and ``k``; used when
        :meth:`rotary_table` gives nothing."""
        raise NotImplementedError


class Mixer(Part):
    # A mixer (or feed-forward) that sets these takes a LazyNorm as input, and the keywords
    # ``residual`` and ``then``: given a residual it may return ``Summed(residual + output)``
    # instead of its output, with ``scaled`` made for the norm ``then`` (the one that follows).
    takes_lazy_norm = False
    adds_residual = False

    def cache_spec(self) -> PagedKVSpec | StateSpec | tuple | None:
        """What the mixer keeps; a tuple for a mixer made of several, which then gets a tuple of
        bindings."""
        return None

    # A mixer that sets this takes the keyword ``defer_terms`` and may then return a :class:`TermSum`
    # instead of its output.
    defers_terms = False

    # A mixer whose work starts with ONE product of its input, left in 32-bit, may offer it to a mixer
    # that runs several on the same input: ``input_matrix(tensors)`` (rows a multiple of 8, called
    # before ``load``, which then makes no product of its own) and ``from_projection(p, ctx, cache)``.
    shares_input_product = False

    def forward(self, x: torch.Tensor, ctx: StepContext, cache) -> torch.Tensor:
        raise NotImplementedError


class FeedForward(Part):
    takes_lazy_norm = False
    adds_residual = False
    # A feed-forward that sets this takes the keyword ``defer_terms`` and may then return a
    # :class:`TermSum` instead of its output.
    defers_terms = False
    # A feed-forward that sets this takes the keyword ``defer_sum`` and may then return a
    # :class:`PairSum` instead of its output.
    can_defer_sum = False

    def forward(self, x: torch.Tensor, ctx: StepContext) -> torch.Tensor:
        raise NotImplementedError


class Block(Part):
    """An arrangement of a mixer, a feed-forward and norms.  The hidden state travels between
    blocks as ``(x, delta)`` meaning ``x + delta``, so that a block's last addition can be fused
    into the next norm."""

    # A block that sets this takes the keyword ``then``: the norm that will consume its output
    # (the next run's first norm), so that its last product can prepare that norm's input.
    takes_next_norm = False
    # ``then`` may be a :class:`ShiftedInput`, a :class:`MixedInput`
    prepares_shifted_input = False
    prepares_mixed_input = False

    def forward(self, x: torch.Tensor, delta: torch.Tensor | None, ctx: StepContext, cache
                ) -> tuple[torch.Tensor, torch.Tensor | None]:
        raise NotImplementedError

    def first_norm(self) -> "Norm | None":
        """The norm this block applies to its input first, if another block may prepare it."""
        return None

    # A block that keeps per-request state of its own (beside its mixer's) says what it needs, and
    # its ``forward`` takes the keyword ``own_state`` (a :class:`StateBinding`).
    def state_spec(self) -> StateSpec | None:
        return None

    def first_input(self, own_state: StateBinding | None
                    ) -> "Norm | ShiftedInput | MixedInput | None":
        """What another block may prepare for this one, given the binding of its own state."""
        return self.first_norm()


class StreamInput(Part):
    """Something added to the residual stream that is not a sublayer's output: a vector that
    depends on the token, on the pass of a loop, or on the embedding output.  Two places use such
    parts: a block may end with one (``forward``), and a run of the plan may start with one
    (``enter``: :attr:`RunEntry.enter`)."""

    wants_act = False      # forward() reads the stream rounded to the activation dtype

    def forward(self, x: torch.Tensor, act: torch.Tensor | None, ctx: StepContext, mult: float,
                then: "Norm | None" = None) -> tuple[torch.Tensor, torch.Tensor | None]:
        """``x`` fp32 ``[T, H]`` -> ``(x', then(x') or None)``; ``act``: ``x`` in the activation
        dtype if the part asked for it; ``mult``: the layer's residual multiplier."""
        raise NotImplementedError

    def enter(self, x: torch.Tensor, ctx: StepContext, embedding_output: torch.Tensor,
              index: int) -> torch.Tensor:
        """``x`` before a run of the plan -> ``x'``; ``index``: the entry's number."""
        raise NotImplementedError


class Embedding(Part):
    # An embedding that depends on earlier tokens of the sequence says what it keeps of them, and its
    # ``forward`` takes the keyword ``own_state`` (a :class:`StateBinding`).
    def state_spec(self) -> StateSpec | None:
        return None

    def forward(self, token_ids: torch.Tensor, ctx: StepContext) -> torch.Tensor:
        raise NotImplementedError


class Head(Part):
    def forward(self, x: torch.Tensor, ctx: StepContext) -> torch.Tensor:
        """``x [R, hidden]`` -> logits ``[R, vocab]`` in fp32."""
        raise NotImplementedError


# ----------------------------------------------------------------------------- registries
_FAMILIES = ("mixer", "feed_forward", "norm", "position", "block", "embedding", "head",
             "stream_input")
_REGISTRY: dict[str, dict[str, Callable[..., Part]]] = {f: {} for f in _FAMILIES}


def register_part(family: str, kind: str, factory: Callable[..., Part]) -> None:
    if family not in _REGISTRY:
        raise KeyError(f"unknown part family '{family}'; families are {_FAMILIES}")
    _REGISTRY[family][kind] = factory


def make_part(family: str, spec: PartSpec, **extra) -> Part:
    try:
        factory = _REGISTRY[family][spec.kind]
    except KeyError:
        raise KeyError(f"no {family} of kind '{spec.kind}' is registered; known: "
                       f"{sorted(_REGISTRY.get(family, {}))}") from None
    return factory(**dict(spec.params), **extra)


def register_mixer(kind, factory):
    register_part("mixer", kind, factory)


def register_feed_forward(kind, factory):
    register_part("feed_forward", kind, factory)


def register_norm(kind, factory):
    register_part("norm", kind, factory)


def register_position(kind, factory):
    register_part("position", kind, factory)


def register_block(kind, factory):
    register_part("block", kind, factory)


def register_stream_input(kind, factory):
    register_part("stream_input", kind, factory)
