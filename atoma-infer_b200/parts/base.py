"""Interfaces of the parts a model is put together from.

A model is a list of layers; a layer is a block that arranges a mixer (attention
here), a feed-forward and norms around the residual stream.  Each part takes its
sizes and constants as parameters (a plain dict in the model spec) and does not
know which model it is in.  The reference hard-wires one arrangement
(models/src/llama.rs:203-430: CausalSelfAttention, Mlp, Block); the split below is
this engine's, so that another mixer or feed-forward can stand in any layer.

Life of a part: ``__init__(params, prefix)`` from the spec; ``declare()`` lists the
checkpoint tensors it needs; ``bind(tensors, rt)`` receives them on the device;
``forward`` runs inside a step.
"""
from __future__ import annotations

from dataclasses import dataclass, field
from typing import Any, Dict, List, Optional, Sequence

import torch

from ..cache.spec import CacheNeed, LayerCache
from ..weights.loader import TensorDecl


@dataclass
class Runtime:
    """What a bound part may use: the device, the compute dtype and the kernels."""

    device: torch.device
    dtype: torch.dtype
    ops: Any


@dataclass
class EntryInfo:
    """One request's share of a step, as the host sees it."""

    req: int
    start: int        # first row of the request's tokens in the step's flat batch
    num_tokens: int
    context_len: int  # tokens of the request already in the cache
    state_slot: int
    is_new: bool      # first step of the request: fixed-size state starts from zero


@dataclass
class StepContext:
    """Everything a part may read about the step under way.

    Device arrays are int32 views into one metadata buffer that the step function
    uploads in a single copy; sizes in capitals are the launch sizes (what buffers
    are padded to), the true ones stand in the metadata header for the kernels.
    """

    rt: Runtime
    T: int                       # rows of the flat batch
    S: int                       # entries (requests) in the batch
    meta: torch.Tensor           # header + arrays (csrc/kernels/common.cuh)
    tokens: torch.Tensor         # [T]
    positions: torch.Tensor      # [T] absolute position of each token in its request
    token_entry: torch.Tensor    # [T] index of the entry a token belongs to
    cu_tokens: torch.Tensor      # [S + 1] first row of each entry
    context_lens: torch.Tensor   # [S]
    state_slots: torch.Tensor    # [S]
    entries: List[EntryInfo] = field(default_factory=list)
    max_tokens_per_entry: int = 0
    max_context: int = 0         # longest context_len + num_tokens in the batch
    decode_only: bool = False    # every entry brings exactly one token
    page_size: int = 0
    table_offsets: Sequence[int] = ()   # per cache group: where its block tables start in ``meta`` ...
    table_strides: Sequence[int] = ()   # ... and how long a request's row is
    # What one layer leaves for later layers of the same step (an earlier layer's values that later ones mix in,
    # for instance), by a name the parts agree on.  Lives as long as the step.  ``"mixer_rows"``: a block whose mixer reads the
    # stream itself leaves the float32 rows there of which the mixer's input is the rounding.
    shared: Dict[str, Any] = field(default_factory=dict)

    def block_table(self, group: int) -> torch.Tensor:
        """The block tables of a cache group as a device view [S, pages per request]: entry k's row lists its
        page ids by absolute page index (-1: no page).  For parts written with tensor operations; the
        kernels read the same memory through ``meta``."""
        off, stride = self.table_offsets[group], self.table_strides[group]
        return self.meta[off:off + self.S * stride].view(self.S, stride)


@dataclass
class PendingSum:
    """An addition to the residual stream that is still to be made: mult * (sum of ``terms``) + ``rows`` + ``vector``.
    ``terms`` are a block's sublayer outputs [T, H] in the compute dtype (at most four), ``rows`` float32 [T, H],
    ``vector`` float32 [H] (the same for every token).  ``factors``: one weight per term (None: all 1), for a mixer whose
    result is a weighted sum of several outputs; the sum is then ((f0 t0 + f1 t1) + ...) in this order.  A mixer may
    return a ``PendingSum`` of terms and factors instead of a tensor.  The norm that follows (``Norm.forward``) takes the
    sum in float32, term by term in this order, in the pass in which it also norms the updated row; a block that has no
    norm for it calls ``apply_pending``.  ``norms``: per term None, or (weight float32 [H], eps): the term is divided by its
    root mean square over the width and multiplied by the weight before it is weighed (None: no term is).  A block that
    norms a sublayer's result takes such a sum in one pass; everywhere else ``without_norms`` makes the terms first."""

    terms: Sequence[torch.Tensor] = ()
    mult: float = 1.0
    rows: Optional[torch.Tensor] = None
    vector: Optional[torch.Tensor] = None
    factors: Optional[Sequence[float]] = None
    norms: Optional[Sequence[Any]] = None

    def term_norms(self) -> Sequence[Any]:
        return tuple(self.norms) if self.norms is not None else (None,) * len(self.terms)

    def weights(self) -> Sequence[float]:
        return tuple(self.factors) if self.factors is not None else (1.0,) * len(self.terms)


@dataclass
class StreamMix:
    """What a sublayer leaves pending where the residual is several streams side by side (float32 [T, streams * H]): with
    y = ``result`` times ``scale`` (float32 [H], one factor per channel; None: none), stream k becomes sum_j ``mix``[j, k] x_j
    + ``give``[k] y, all from the old streams (``mix`` float32 [streams, streams], from and to; ``give`` float32 [streams]).
    ``result``: terms, weights, a factor and a vector.  The norm that follows (``Norm.forward_streams``) does this in
    float32 in the pass that also reads and norms the new streams."""

    result: "PendingSum"
    scale: Optional[torch.Tensor]
    mix: torch.Tensor
    give: torch.Tensor


def without_norms(ops, pending, ctx: "StepContext"):
    """The same sum with every normed term replaced by its normed rows, in the terms' type."""
    if not isinstance(pending, PendingSum) or pending.norms is None:
        return pending
    terms = []
    for t, nm in zip(pending.terms, pending.term_norms()):
        if nm is not None:
            out = torch.empty_like(t)
            ops.rms_rows(t, nm[0], nm[1], out, ctx.meta)
            t = out
        terms.append(t)
    return PendingSum(tuple(terms), pending.mult, pending.rows, pending.vector, pending.factors)


def join_terms(parts, mult: float = 1.0) -> "PendingSum":
    """One pending sum of several sublayer results, each a tensor or a ``PendingSum`` of weighted terms (whose own
    factor is folded into its terms' weights)."""
    terms, factors = [], []
    for p in parts:
        if isinstance(p, PendingSum):
            if p.rows is not None or p.vector is not None or p.norms is not None:
                raise ValueError("a sublayer's result has terms and factors only")
            terms += list(p.terms)
            factors += [p.mult * f for f in p.weights()]
        else:
            terms.append(p)
            factors.append(1.0)
    return PendingSum(tuple(terms), mult, factors=None if all(f == 1.0 for f in factors) else tuple(factors))


def apply_pending(ops, resid: torch.Tensor, delta, ctx: "StepContext") -> None:
    """Adds what a block left pending (a tensor, a ``PendingSum`` or a ``StreamMix``; None: nothing) into the float32 stream(s)."""
    if delta is None:
        return
    if isinstance(delta, StreamMix):
        ops.stream_mix_norm(resid, delta.give.numel(), delta, None, None, 0.0, None, ctx.meta, ctx.T)
    elif isinstance(delta, PendingSum):
        delta = without_norms(ops, delta, ctx)
        ops.sum_rmsnorm(resid, delta, None, 0.0, None, ctx.meta, ctx.T)
    else:
        resid.add_(delta)


class Part:
    """Base of all parts: parameters from the spec, tensors by checkpoint name."""

    def __init__(self, params: Dict[str, Any], prefix: str):
        self.params = dict(params)
        self.prefix = prefix

    def declare(self) -> List[TensorDecl]:
        return []

    def bind(self, tensors: Dict[str, torch.Tensor], rt: Runtime) -> None:
        self.rt = rt

    def streamed_weights(self) -> List[torch.Tensor]:
        """The weight matrices of the part's linears in the order ``forward`` uses them (after ``bind``).  The model
        hands the whole step's list to the kernels, which may fetch a weight ahead of its use."""
        return []

    def activation_width(self) -> int:
        """Elements per token of the widest intermediate result the part makes (0: nothing wider than the
        model's width); the engine sizes its working memory from it when it sizes the cache."""
        return 0

    def fused(self) -> Optional[Dict[str, Any]]:
        """What a kernel that runs several parts at once needs to know of this part (after ``bind``): a dict with
        ``kind``, the part's tensors and constants.  None (the default): the part only runs through ``forward``."""
        return None


class Embedding(Part):
    """The first stage: the step's token ids (and whatever else of the step's metadata it wants, positions
    for instance) become the float32 residual stream.  ``graph_safe = True`` on a subclass says that its
    ``forward`` reads the step's metadata on the device only, so a decode step may be captured in a graph."""

    graph_safe = False

    def forward(self, ctx: StepContext) -> torch.Tensor:
        """Returns the residual stream, float32 [ctx.T, hidden]."""
        raise NotImplementedError

    def table(self) -> Optional[torch.Tensor]:
        """The [vocab, hidden] matrix, for a head that is tied to it (None: there is no such matrix)."""
        return None


class Head(Part):
    """The last stage: normed rows become float32 logits over the vocabulary (``graph_safe`` as for the
    embedding)."""

    graph_safe = False

    def bind(self, tensors: Dict[str, torch.Tensor], rt: Runtime, embedding: Optional["Embedding"] = None) -> None:
        """``embedding``: the model's first stage, for a head that shares its matrix."""
        self.rt = rt

    def forward(self, h: torch.Tensor, ctx: StepContext) -> torch.Tensor:
        """``h`` [rows, hidden] in the compute dtype; returns float32 [rows, vocab]."""
        raise NotImplementedError


class Norm(Part):
    def forward(self, resid: torch.Tensor, delta: Optional[torch.Tensor], ctx: StepContext,
                rows: Optional[torch.Tensor] = None, num_rows: int = 0) -> torch.Tensor:
        """Adds ``delta`` into the float32 residual stream (if given) and returns the normed
        rows in the compute dtype.  With ``rows``: only those rows, residual left untouched."""
        raise NotImplementedError

    def forward_streams(self, resid: torch.Tensor, streams: int, delta: Optional[StreamMix], read: Optional[torch.Tensor],
                        ctx: StepContext, rows: Optional[torch.Tensor] = None, num_rows: int = 0) -> torch.Tensor:
        """The same where the residual is several streams side by side ([T, streams * size]): takes ``delta`` into them and
        returns the normed sum of the streams weighed by ``read`` (float32 [streams]; None: the plain sum)."""
        raise NotImplementedError


class SequenceFilter(Part):
    """What a sublayer reads instead of the residual rows themselves: a function of a request's rows over time that
    needs only a fixed number of earlier rows, which it keeps as state (a short causal convolution, for instance)."""

    def state_bytes(self) -> int:
        return 0

    def forward(self, resid: torch.Tensor, ctx: StepContext, state: Optional[torch.Tensor]) -> torch.Tensor:
        """``resid`` float32 [T, H]; ``state`` the part's share of the per-request state, uint8 [slots, state_bytes];
        returns the sublayer's input in the compute dtype.  Reads the state, does not write it."""
        raise NotImplementedError

    def save(self, resid: torch.Tensor, ctx: StepContext, state: Optional[torch.Tensor]) -> None:
        """The step's rows of ``resid`` (what ``forward`` was given) enter the state; called after ``forward``."""
        raise NotImplementedError


class PositionEncoding(Part):
    """How positions enter a mixer.  For attention: ``encode_and_store`` turns the fused
    q|k|v rows of a step into position-encoded queries (in place) and writes keys and
    values to the layer's pages."""

    def encode_and_store(self, qkv: torch.Tensor, ctx: StepContext, cache: LayerCache, *, num_heads: int,
                         num_kv_heads: int, head_dim: int) -> None:
        raise NotImplementedError

    def rotary(self):
        """(inv_freq on the device, rotary_dim) if the encoding is a rotation by position times
        frequency, which the decode attention kernel can apply itself; None otherwise."""
        return None


class Mixer(Part):
    """Mixes information between the tokens of a request."""

    def cache_need(self) -> Optional[CacheNeed]:
        """Keys/values per cached token, or None if the mixer keeps no pages."""
        return None

    def state_bytes(self) -> int:
        """Bytes of fixed-size state per request (0: none)."""
        return 0

    def forward(self, x: torch.Tensor, ctx: StepContext, cache: LayerCache) -> torch.Tensor:
        raise NotImplementedError


class FeedForward(Part):
    def forward(self, x: torch.Tensor, ctx: StepContext) -> torch.Tensor:
        raise NotImplementedError


class Block(Part):
    """Arranges norms, mixer and feed-forward around the residual stream.

    ``forward(resid, delta, ctx, cache)``: ``resid`` is the float32 residual stream
    [T, H], ``delta`` what the previous block left to be added (None at the first);
    returns this block's own pending addition (a tensor, or a ``PendingSum`` of several terms and a
    factor).  Keeping the last addition pending lets the next norm do it, in float32, in the same pass.  ``ctx.shared["next_run"]`` holds
    (block, cache view) of the layer run that follows, or None: a block whose last kernel can
    also leave that block's input may do so under ``ctx.shared["prepared_input"]`` =
    (that block, tensor), which the next block takes if it finds itself named."""

    mixer: Mixer
    streams = 0  # how many streams side by side the block works on ([T, streams * H]); 0: the plain stream [T, H]

    def forward(self, resid: torch.Tensor, delta: Optional[torch.Tensor], ctx: StepContext,
                cache: LayerCache) -> Optional[torch.Tensor]:
        raise NotImplementedError

    def state_bytes(self) -> int:
        """Bytes of fixed-size state per request that the block's parts keep together (the mixer's, by default);
        a block with more stateful parts hands each its share of ``cache.state``."""
        return self.mixer.state_bytes()

    def decode_fusion(self) -> Optional[Dict[str, Any]]:
        """For a kernel that runs a run of whole layers of a decode step: this block's arrangement and what its
        parts say of themselves (``Part.fused``), or None if the block, or one of its parts, cannot take part."""
        return None
