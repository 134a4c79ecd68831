"""What every part sees: the build environment, the step's context, and the
interfaces of the four kinds of part.

A part is built from its spec record and a :class:`BuildEnv` (compute dtype and
device), declares the tensors it wants (``param_infos``), receives them
(``load``) and then runs on packed tokens: activations are [tokens, features]
for all sequences of the step back to back, and a :class:`StepContext` says
which token belongs to which sequence, at which position, in which cache slot.

Hidden state between parts is a pair ``(resid, delta)``: the float32 residual
stream and the output of the last part in the compute dtype, not yet added.
A norm adds it while it reads it (one pass over the data instead of two).

Interfaces
----------
Norm            ``__call__(resid, delta=None, rows=None) -> normed``
PositionEncoding ``prepare(max_positions)``; either ``fused_table()`` (a float32
                [positions, rotary_dim/2, 2] cos/sin table that the attention
                kernel applies itself) or ``apply(q, k, ctx) -> (q, k)``
Mixer           ``cache_request() -> CacheRequest | None``;
                ``__call__(x, ctx, cache) -> y`` with ``cache`` the
                :class:`~..cache.LayerCache` of the schedule entry
FeedForward     ``__call__(x, ctx) -> y``
"""
from __future__ import annotations

from dataclasses import dataclass, field, replace
from typing import Dict, Optional

import torch

from .registry import ParamInfo


@dataclass(frozen=True)
class BuildEnv:
    dtype: torch.dtype            # compute dtype: torch.float32 or torch.bfloat16
    device: torch.device


@dataclass
class StepContext:
    """The packed batch of one step.  Device tensors are int32.

    tok_seq[t]   index (within this step) of the sequence token t belongs to
    tok_pos[t]   position of token t in its sequence (= cache length before it)
    seq_slot[b]  cache slot of sequence b
    seq_start[b] first packed token of sequence b (length B+1)
    seq_len[b]   length of sequence b after this step
    ids[t]       token id of token t (for parts that look something up by it; the model sets it)
    """
    tok_seq: torch.Tensor
    tok_pos: torch.Tensor
    seq_slot: torch.Tensor
    seq_start: torch.Tensor
    seq_len: torch.Tensor
    num_tokens: int
    num_seqs: int
    max_new: int                  # most tokens any sequence brings in this step
    max_len: int                  # longest sequence after this step
    host_seq_slot: tuple = ()
    host_new: tuple = ()          # tokens each sequence brings
    host_len: tuple = ()          # lengths after this step
    ids: Optional[torch.Tensor] = None

    @property
    def decode_only(self) -> bool:
        return self.max_new == 1

    @property
    def len_bucket(self) -> int:
        """``max_len`` rounded up to a multiple of 1024: what kernels size their grids
        and scratch memory by, so that a captured step stays valid while the
        sequences grow inside the bucket."""
        return -(-max(1, self.max_len) // 1024) * 1024


@dataclass(frozen=True)
class CacheRequest:
    """What a mixer needs stored per sequence.

    Keys and values: ``kv_heads`` x ``head_dim`` per token (0 for none), all of
    them (``window`` 0) or the last ``window``; ``chunk`` > 0 instead of a window: the
    keys of the query's own chunk of that many positions, counted from the sequence's
    start.  ``keep_first``: beside the window, the sequence's first tokens, which every query
    sees however far behind they are.  ``shared_kv``: the values are the keys (a latent that serves as both), so
    one pool is kept and handed out as both.
    Fixed-size state: ``state_shape`` per sequence (empty for none), zeroed when a
    slot is given out; ``more_state``: further such tensors as (shape, dtype) pairs,
    handed out in this order as ``LayerCache.more_state``."""
    kv_heads: int = 0
    head_dim: int = 0
    window: int = 0
    state_shape: tuple = ()
    state_dtype: torch.dtype = torch.float32
    shared_kv: bool = False
    chunk: int = 0
    more_state: tuple = ()
    keep_first: int = 0

    @property
    def kept(self) -> int:
        """First tokens that stay stored beside a window (0 where everything, or a chunk, stays anyway)."""
        if self.keep_first and self.chunk:
            raise ValueError("kept first tokens go with a window, not with a chunked mask")
        return self.keep_first if self.window else 0

    def for_readers(self, others) -> "CacheRequest":
        """This request of a writing layer, widened so that layers that read the same entry through masks of their own
        (``others``: their requests) find every key they see."""
        masks = [(r.window, r.chunk, r.kept) for r in (self, *others)]
        if len(set(masks)) == 1:
            return self
        if all(w > 0 for w, _, _ in masks):
            return replace(self, window=max(w for w, _, _ in masks), chunk=0, keep_first=max(k for _, _, k in masks))
        return replace(self, window=0, chunk=0, keep_first=0)

    @property
    def mask(self) -> int:
        """The one integer the kernels and the page bookkeeping take: the window, or minus the chunk size."""
        if self.window and self.chunk:
            raise ValueError("a cache entry has a window or a chunked mask, not both")
        return self.window if self.window else -self.chunk


@dataclass
class Pending:
    """A sublayer's output that has not joined the residual yet, for a residual kept as several streams: the norm in
    front of the next sublayer applies x_t <- sum_s mix[s, t] x_s + out[t] y while it reads the streams
    (``mix`` None: the identity; ``out`` None: ones).  ``more``: further outputs that join in the same pass (a layer
    whose mixer and feed-forward run side by side, a mixer that is a weighted sum of two), as pairs (tensor, weights
    [streams] or None for ones): x_t <- ... + out[t] y + w2[t] y2 + ..., the sum taken in float32."""
    y: Optional[torch.Tensor]
    mix: Optional[torch.Tensor] = None
    out: Optional[torch.Tensor] = None
    more: tuple = ()
    # float32 terms that join after the outputs (an :class:`Injection`); ``y`` may then be None (nothing pending)
    entry: object = None
    # a norm behind the sublayer, as a pair (gain float32 [width], eps): the outputs' weighted sum s joins as
    # s / sqrt(mean(s^2) + eps) * gain (``out`` and the weights in ``more`` are then float32 factors [1])
    post: object = None


@dataclass
class Injection:
    """Float32 terms that join the residual right before a layer, after whatever is pending: first the embedding's
    rows once more, table[ids] * scale (``ids`` None: not), then the vector ``vec`` [hidden] on every token."""
    ids: Optional[torch.Tensor]
    table: Optional[torch.Tensor]
    scale: float
    vec: Optional[torch.Tensor]


@dataclass
class WeightedSum:
    """A part's output given as sum_i factor_i * tensor_i, the sum not yet taken: whoever adds it to the residual adds
    the terms one by one in float32 (``parts/link.py``), so that no term is rounded a second time."""
    terms: tuple                 # ((tensor, factor), ...)


class Part:
    """Common base: parameters by local name.

    ``graph_safe``: one-token steps are captured into CUDA graphs and replayed.  A
    captured step repeats the same launches with the same host-side values, so a
    part may only be replayed if everything that changes from step to step reaches
    its kernels through device tensors (the context's int32 tables, the cache).  A
    part that reads ``ctx.host_*`` values, branches on them or indexes with them
    must leave this False; a model with such a part runs every step eagerly."""
    kind = "?"
    graph_safe = False

    def __init__(self, spec, env: BuildEnv):
        self.spec = spec
        self.env = env

    @classmethod
    def param_infos(cls, spec) -> Dict[str, ParamInfo]:
        return {}

    def load(self, tensors: Dict[str, torch.Tensor]) -> None:
        """Receives the declared tensors, already on the device and in the dtype of
        their role (matrix: compute dtype; gain: float32; table: int32)."""

    def weight_bytes(self) -> int:
        return 0

    def reads_first(self) -> Optional[torch.Tensor]:
        """The weight matrix [N, K] of the linear with which this part starts, if it starts
        with one: the norm before it may warm the cache for it (see ``Norm.takes_hint``)."""
        return None


class Norm(Part):
    """``takes_hint``: the norm's ``__call__`` has a fourth argument ``then``, the weight matrix
    that the following part reads first (a performance hint that changes no result)."""
    takes_hint = False

    def __call__(self, resid, delta=None, rows=None):
        raise NotImplementedError


class PositionEncoding(Part):
    def prepare(self, max_positions: int) -> None:
        pass

    def fused_table(self) -> Optional[torch.Tensor]:
        return None

    def apply(self, q, k, ctx: StepContext):
        return q, k


class Mixer(Part):
    def cache_request(self) -> Optional[CacheRequest]:
        return None

    def prepare(self, max_positions: int) -> None:
        pass

    def __call__(self, x, ctx: StepContext, cache):
        raise NotImplementedError


class FeedForward(Part):
    def __call__(self, x, ctx: StepContext):
        raise NotImplementedError
