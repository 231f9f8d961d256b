"""Interfaces of the parts a layer is put together from, and what a step hands them.

A part is built from explicit sizes and constants (never from a model's
configuration object), lists the tensors it reads (``tensor_specs``), receives
them (``bind``) and computes on the tokens of one step (``forward``).  No part
knows which model, or which layer of it, it is in.

Activations: the residual stream ``h`` is fp32 ``[T, H]`` in both precisions;
norms read it and write the compute dtype (bf16 or fp32); mixers and
feed-forwards read the normed rows and ADD their result into ``h``.
"""

from __future__ import annotations

from dataclasses import dataclass, field
from typing import Any, Optional

import torch

from .plan import TensorSpec


# ----------------------------------------------------------------------------- cache needs
@dataclass(frozen=True)
class PagedKV:
    """The mixer keeps a key and a value of ``num_kv_heads x head_dim`` per token, in pages.
    ``window``: None = every past token is read; n = only the last n (the current one included),
    so pages that lie wholly behind the window are given back while the request runs.
    ``chunk``: positions are counted off in chunks of that many from 0 and a token reads the keys of its own chunk only, so
    the pages of chunks that are over are given back while the request runs (not together with ``window``).
    ``v_head_dim``: size of a value head where it differs from a key head's (None = the same; 0 = no value rows are
    kept, for a mixer whose keys carry their values).
    ``run`` (with ``window``): positions are counted off in runs of that many from 0, and the pages of a run that is not
    complete yet stay although the window may have passed its first positions (its rows are pooled when it is complete).
    ``keep_first`` (with ``window``): the request's first so many tokens stay readable whatever the window has passed, so their
    pages stay until the request ends.
    ``stride``: one row for every ``stride`` WHOLE tokens instead of one per token: row r stands for the tokens
    r * stride .. r * stride + stride - 1 and exists once the last of them is in the cache."""

    num_kv_heads: int
    head_dim: int
    window: Optional[int] = None
    v_head_dim: Optional[int] = None
    chunk: Optional[int] = None
    run: Optional[int] = None
    stride: int = 1
    keep_first: int = 0

    def first_needed(self, num_tokens: int) -> int:
        """The lowest row beyond the kept first ones that a query at position ``num_tokens`` or later can still read."""
        if self.chunk is not None:
            return num_tokens - num_tokens % self.chunk
        if self.window is not None:
            first = max(0, num_tokens - self.window + 1)
            return first if self.run is None else min(first, num_tokens - num_tokens % self.run)
        return 0

    def rows(self, num_tokens: int) -> int:
        """How many rows ``num_tokens`` tokens have."""
        return num_tokens // self.stride

    @property
    def span(self) -> Optional[int]:
        """The most rows that have to stay in the cache at once, whatever the request's length (None: no such bound)."""
        if self.chunk is not None:
            return self.chunk
        if self.window is not None:
            return self.keep_first + (self.window if self.run is None else max(self.window, self.run))
        return None

    @property
    def keeps_all(self) -> bool:
        """Whether every key stays readable as long as the request lives."""
        return self.window is None and self.chunk is None

    @property
    def value_dim(self) -> int:
        return self.head_dim if self.v_head_dim is None else self.v_head_dim


@dataclass(frozen=True)
class FixedState:
    """The mixer keeps a tensor of ``shape`` per request, whatever the request's length.
    It is zeroed when a request is admitted."""

    shape: tuple
    dtype: torch.dtype = torch.float32


@dataclass(frozen=True)
class CombinedNeed:
    """Several needs of one mixer (a mixer that wraps another, or one with pages AND a state): the mixer gets a
    ``LayerCache`` whose ``parts`` are the caches of ``needs``, in order."""

    needs: tuple


def leaf_needs(need) -> list:
    """The needs that ``need`` is made of (itself, unless it is a CombinedNeed); None gives none."""
    if need is None:
        return []
    if isinstance(need, CombinedNeed):
        out = []
        for n in need.needs:
            out += leaf_needs(n)
        return out
    return [need]


# ----------------------------------------------------------------------------- step context
@dataclass
class PagedMeta:
    """Device metadata of one page group for one step."""

    block_tables: torch.Tensor  # int32 [S, max_blocks]; -1 = no page
    # int32 [T]; page * page_size + slot of each token of the step; in a group with a stride the slot of the row that
    # the token completes, or -1
    slot_mapping: torch.Tensor
    page_size: int


@dataclass
class SeqInfo:
    """Host-side description of one request's share of a step."""

    request_id: Any
    q_start: int  # first row of the step's token arrays
    q_len: int
    start_pos: int  # tokens of the request that were in the cache before this step
    state_slot: int


@dataclass
class StepContext:
    """Everything a part may need about the step: device arrays and their host twins."""

    num_tokens: int
    num_seqs: int
    token_ids: torch.Tensor  # int32 [T]
    positions: torch.Tensor  # int32 [T] absolute position of each token
    token_seq: torch.Tensor  # int32 [T] index of the token's request within the step
    seq_q_start: torch.Tensor  # int32 [S + 1]
    seq_start_pos: torch.Tensor  # int32 [S]
    seq_state_slot: torch.Tensor  # int32 [S]
    seqs: list  # list[SeqInfo]
    paged: dict  # group id -> PagedMeta
    max_q_len: int
    max_kv_len: int
    act_dtype: torch.dtype
    workspace: Any  # engine.workspace.Workspace
    device: torch.device = None
    # in a step that mixes portions of prompts with single tokens: the rows (int32, device) of the
    # requests that bring exactly one token, so that kernels made for either kind can share the step
    single_rows: Optional[torch.Tensor] = None
    # what parts compute once per pass of the model and share across layers, under keys of their own; the
    # model empties it when a pass begins
    shared: dict = field(default_factory=dict)

    @property
    def all_decode(self) -> bool:
        return self.max_q_len == 1


@dataclass
class LayerCache:
    """What one run of a layer's mixer owns in the cache.

    ``group``: id of the page group (PagedKV) whose block tables address ``k`` and ``v``
    ([pages, kv heads, page size, head dim]); ``state``: [slots, *shape] for FixedState; ``parts``: the caches
    of a CombinedNeed's needs.
    """

    need: Any
    group: Optional[int] = None
    k: Optional[torch.Tensor] = None
    v: Optional[torch.Tensor] = None
    state: Optional[torch.Tensor] = None
    parts: Optional[list] = None

    def leaves(self) -> list:
        """This cache, or the caches it is made of."""
        if self.parts is None:
            return [self]
        out = []
        for p in self.parts:
            if p is not None:
                out += p.leaves()
        return out


# ----------------------------------------------------------------------------- part interfaces
class Part:
    """Base of every part."""

    def tensor_specs(self, prefix: str) -> list:
        """The tensors this part reads, named under ``prefix``."""
        return []

    def bind(self, tensors: dict, prefix: str) -> None:
        """Receive the loaded tensors (on the device, in the dtype their role gives).
        Optional tensors that the folder lacks are absent from ``tensors``."""


class Norm(Part):
    def forward(self, h: torch.Tensor, out: torch.Tensor, row_index: Optional[torch.Tensor] = None) -> None:
        """out[i] = norm(h[row_index[i]] or h[i]); h fp32, out in the compute dtype."""
        raise NotImplementedError

    def lazy(self, h: torch.Tensor, out: torch.Tensor):
        """An object that stands for norm(h): ``materialize()`` computes it into ``out`` (once).  A norm
        whose arithmetic a matrix-product kernel can do on its way returns a richer object that such a
        kernel recognises; the default is to compute at once."""
        self.forward(h, out)
        return out

    # True if add_into also takes ``ops.PairRows`` for y (a mixture's results that its own kernel adds first)
    adds_parts = False

    def add_into(self, y: torch.Tensor, h: torch.Tensor, rows: Optional[torch.Tensor], workspace) -> None:
        """h += norm(y), y and h fp32; ``rows`` (or None): h in the activations' type as well.  The default is a norm, a
        sum and a cast; a norm with a kernel for all of it overrides this."""
        from ..kernels import ops

        normed = workspace.get("norm_add", tuple(h.shape), torch.float32)
        self.forward(y, normed)
        ops.add_(h, normed)
        if rows is not None:
            ops.rmsnorm_add(None, None, 0.0, h, rows)


class PositionEncoding(Part):
    """How positions enter a mixer.  ``rotary_table`` lets the attention mixer fuse the
    rotation with its cache write; a kind without one is applied through ``apply``; a kind that acts on
    the attention scores instead of (or beside) q and k says so with ``score_slopes``."""

    # as for Mixer: True if ``apply`` may be recorded into a CUDA graph (kinds with a rotary table never run it)
    graph_safe = False

    def rotary_table(self, device=None) -> Optional[tuple]:
        """``(inv_freq, R)`` if the encoding is a rotate-half rotation of the first R dims of
        each head by ``pos * inv_freq[i]`` (inv_freq fp32 [R/2] on ``device``; ``(None, 0)`` =
        nothing to rotate), which the attention mixer fuses with its cache write.
        ``None`` = not of that form: the mixer calls ``apply`` instead."""
        return None

    def apply(self, qkv: torch.Tensor, positions: torch.Tensor, num_heads: int, num_kv_heads: int,
              head_dim: int) -> None:
        """Encode positions into the q and k heads of ``qkv`` in place."""
        raise NotImplementedError

    def score_slopes(self, num_heads: int, device=None) -> Optional[torch.Tensor]:
        """fp32 [num_heads] on ``device`` if the encoding adds ``slopes[head] * (j - P)`` to the score of the key at
        position j for the query at position P (a penalty linear in the distance; j <= P); None (the default) if it
        adds nothing to the scores.  Such scores are attended by the general kernel in every precision."""
        return None

    def score_log_penalty(self, num_heads: int, device=None) -> Optional[tuple]:
        """(r1, r2), fp32 [num_heads] each on ``device``, if the score of the key at position j for the query at position
        P loses r1[head] * ln(1 + r2[head] * (P - j)); None (the default) otherwise."""
        return None


class Mixer(Part):
    """What mixes the tokens of a request: attention over cached keys and values, a recurrence over a state
    of fixed size, or anything else that declares its need with ``cache_need``.

    A step hands the mixer all its tokens as one batch; which row belongs to which request is told twice, on
    the host (``ctx.seqs``, a list of ``SeqInfo``) and on the device.  A mixer that wants its steps recorded
    into CUDA graphs (``graph_safe``) works from the device arrays alone, because a replayed step runs no
    Python: ``ctx.token_seq`` [T] (index of each row's request within the step), ``ctx.positions`` [T],
    ``ctx.seq_q_start`` [S + 1] (first row of each request; rows of a request are consecutive and in order),
    ``ctx.seq_start_pos`` [S] (tokens the request held before the step), ``ctx.seq_state_slot`` [S] (the row
    of ``cache.state`` that is the request's, for a ``FixedState`` need) and, for a ``PagedKV`` need,
    ``ctx.paged[cache.group]`` (block tables [S, max_blocks] and the cache slot of every row).  The shapes
    T and S are those of the recorded step; the contents change from replay to replay.  A decode step may
    carry padding rows after the real ones: single tokens at position 0 of requests that do not exist, whose
    state slot and page are the cache manager's padding slot and padding page, so whatever a mixer writes
    for them lands where nobody reads.  A mixer with state must carry the state across steps through its
    slot and process a request's rows in order; it may not assume that a step holds the whole request."""

    # True if forward takes its input ``x`` either as a tensor or as the object that ``Norm.lazy`` returns
    # (which it hands to ``ops.gemm`` unchanged, or turns into a tensor with ``materialize()``).
    accepts_lazy_norm = False
    # True if forward only launches work on the current stream from device-resident metadata (no host
    # loops over requests, no synchronisation, no read of ``ctx.seqs``), so that a step can be recorded into
    # a CUDA graph.  One part that says False switches graphs off for the whole model.
    graph_safe = False
    # True if forward takes ``accumulate=False``: the result then REPLACES what ``h`` holds (h = mix(x)), which spares
    # a caller that wants the result alone (a block over several residual streams, mixers side by side) the zeroing.
    can_overwrite = False

    def cache_need(self):
        """PagedKV, FixedState, a CombinedNeed of several, or None."""
        return None

    def forward(self, x: torch.Tensor, h: torch.Tensor, ctx: StepContext, cache: Optional[LayerCache],
                owns_cache: bool) -> None:
        """h += mix(x).  ``owns_cache`` False: read ``cache`` but do not write it."""
        raise NotImplementedError


class FeedForward(Part):
    accepts_lazy_norm = False  # as for Mixer
    graph_safe = False  # as for Mixer
    can_overwrite = False  # as for Mixer

    def forward(self, x: torch.Tensor, h: torch.Tensor, ctx: StepContext) -> None:
        """h += feed_forward(x)."""
        raise NotImplementedError


class Block(Part):
    graph_safe = False
    # True for a block that keeps ctx.shared["residual_rows"] (the residual rows in the activations' type) in step with
    # the residual stream; whatever else touches the stream makes the model forget those rows
    keeps_rows = False

    def cache_need(self):
        return None

    def forward(self, h: torch.Tensor, ctx: StepContext, cache: Optional[LayerCache], owns_cache: bool) -> None:
        raise NotImplementedError


def role_dtype(role: str, compute_dtype: torch.dtype, stored: torch.dtype) -> torch.dtype:
    """Device dtype of a tensor of ``role`` stored as ``stored`` when the engine computes in
    ``compute_dtype``: matrices and embeddings in the compute dtype; vectors in fp32 (an exact
    widening of bf16; a vector stored in 32-bit stays so); integer tables int32."""
    if role in ("matrix", "embedding"):
        return compute_dtype
    if role in ("bias", "norm", "vector"):
        return torch.float32
    if role == "int_table":
        return torch.int32
    raise ValueError(f"unknown tensor role '{role}'")


__all__ = [
    "PagedKV", "FixedState", "CombinedNeed", "leaf_needs", "PagedMeta", "SeqInfo", "StepContext", "LayerCache", "Part", "Norm",
    "PositionEncoding", "Mixer", "FeedForward", "Block", "TensorSpec", "role_dtype",
]
