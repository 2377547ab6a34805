"""Interfaces of the parts of a layer, the context a step hands them, and the registries that
map a part's description (``config.specs``) to its implementation.

No part knows which model it is in: it gets its sizes and constants from its spec, its
tensors by the names in its spec, and everything about the running step from the
:class:`StepContext`.

A rule for parts that write the key/value cache: the decode attention kernel (``kernels.attention`` for single
tokens in bfloat16) starts copying cache pages while the two kernels launched before it may still run, and
fetches again only each token's own newest row.  A part that writes other rows of a cache shortly before that
cache is attended to (within two launches) passes ``own_rows_only=False`` to ``kernels.attention``; the
attention part does so for a schedule entry that reads another entry's cache (``cache_of``).

Interfaces
----------
Norm          ``forward(x_f32 [T,H], out_dtype, rows_index=None) -> [rows,H]``; optionally
              ``add_forward(x, y, out_dtype)``: x += y and the norm in one pass; ``add_into(x, y, then, out_dtype)``:
              x += norm(y), and the next norm of x, in one pass
Position      ``prepare(max_positions)``; ``rotate_and_store(qkv, n_q, n_kv, head_dim, ctx, kv)``
Mixer         ``cache_needs()``; ``prepare(max_positions)``; ``apply(h, ctx, entry, cache_entry,
              owns_cache) -> y``; optionally ``add_to(x, norm, ctx, ...)`` fused
FeedForward   ``apply(h, ctx) -> y``; optionally ``add_to(x, norm, ctx)`` fused
Arrangement   ``run(layer, x, ctx, entry, cache_entry, owns_cache)``: updates ``x`` in place
InputFilter   what stands between a norm and the sublayer that reads it (a short causal convolution): ``state_elems()``;
              ``apply(y_f32 [T,H], ctx, state, offset, out_dtype) -> [T,H]``, which also brings its state up to date
StreamPosition  ``prepare(max_positions)``; ``add_to(x, ctx)``: positions added to the embedded stream

State of a layer: ``ctx.state(cache_entry)`` is one float32 area [slot, elems]; the mixer's numbers come first
(``Mixer.cache_needs().state_elems``), then those of the mixer's input filter, then those of the feed-forward's
(``Layer.state_offsets``).
"""
from __future__ import annotations

from dataclasses import dataclass, field
from typing import Callable, Dict, List, Optional

import torch

from ..cache import CacheNeeds
from ..config.specs import ConfigError, PartSpec
from ..weights.loader import ParamSpec


@dataclass
class KVView:
    """Keys and values of one schedule entry for the running step."""
    k: torch.Tensor               # [page, kv head, PAGE, head_dim]
    v: torch.Tensor
    table: torch.Tensor           # int32 [B, stride]: physical page of each logical page of each batch row
    stride: int
    window: Optional[int]


@dataclass
class StepContext:
    """Everything a part may know about the running step.

    The step runs ``T`` tokens of ``B`` sequences, packed sequence after sequence.  Token t
    belongs to batch row ``tok_row[t]`` and stands at position ``tok_pos[t]`` of its sequence; row b's
    tokens are ``row_first[b] .. row_first[b + 1] - 1``.  The device arrays are what a kernel needs to
    find its rows, also inside a captured graph, where the host lists (``lens``, ``starts``,
    ``slot_ids``) are those of the step that was captured and must not be read.  A captured step
    of a fixed number of rows may carry idle rows: they bring one token at position 0 of the cache's idle
    slot, and nobody reads what they produce.
    """
    T: int
    B: int
    dtype: torch.dtype                    # dtype of activations and cache
    device: torch.device
    tok_pos: torch.Tensor                 # int32 [T], device
    tok_row: torch.Tensor                 # int32 [T], device
    slots: torch.Tensor                   # int32 [B], device: sequence slot of each batch row
    row_first: torch.Tensor               # int32 [B + 1], device: packed index of each row's first token; row_first[B] = T
    row_lens: torch.Tensor                # int32 [B], device: tokens each row brings in this step
    slot_ids: List[int]                   # the slots on the host
    lens: List[int]                       # tokens of each row in this step (host)
    starts: List[int]                     # position of each row's first token (host)
    one_token_each: bool                  # every row brings exactly one token
    cache: object                         # cache.Cache
    tables: Dict[int, torch.Tensor] = field(default_factory=dict)    # group -> int32 [B, stride]
    max_context: int = 0                  # upper bound of any row's length after the step
    scratch: Dict[str, torch.Tensor] = field(default_factory=dict)   # named buffers that live as long as the step
    pending: Optional[torch.Tensor] = None  # a product [T, hidden] that still has to be added to the residual stream
    pending_norm: Optional["Norm"] = None   # the norm that product passes on its way into the stream (None: it is added as it is)
    pending_streams: Optional["Part"] = None  # how it enters a residual of several streams (a StreamMix)
    pending_rows: Optional[tuple] = None    # (rows [T, hidden], weights [T]): rows times a number a token that are added with the pending product
    stream_source: Optional[torch.Tensor] = None  # the one matrix [T, hidden] that all streams still equal, before the first sum into them

    # A part whose product comes out of the library may leave the sum into the residual stream pending, so
    # that the norm that follows does both in one pass.  Whoever reads the stream first settles it: parts
    # that declare ``takes_pending`` through ``normed``, everyone else through the arrangement.  A sublayer's
    # output that is normed before it is added (``defer_normed_add``) waits the same way: that norm, the sum and
    # the next reader's norm are then one pass over the rows.
    def defer_add(self, x: torch.Tensor, y: torch.Tensor, rows: Optional[tuple] = None) -> None:
        """x += y, left pending; ``rows`` = (r [T, hidden], w float32 [T]): x += y + w[t] * r[t]."""
        self.settle(x)
        self.pending, self.pending_rows = y, rows

    def defer_normed_add(self, x: torch.Tensor, y: torch.Tensor, norm: "Norm") -> None:
        """x += norm(y), left pending."""
        self.settle(x)
        self.pending, self.pending_norm = y, norm

    def settle(self, x: torch.Tensor) -> None:
        if self.pending is not None:
            from ..ops import kernels
            if self.pending_streams is not None:
                self._mix_streams(x, dst=x)
                return
            y, n, rows = self.pending, self.pending_norm, self.pending_rows
            self.pending = self.pending_norm = self.pending_rows = None
            if rows is not None:
                kernels.add_layernorm(x, y.contiguous(), rows=rows[0], row_weights=rows[1])
            elif n is None:
                kernels.residual_add(x, y.contiguous())
            else:
                n.add_into(x, y.contiguous())

    def normed(self, x: torch.Tensor, norm: "Norm") -> torch.Tensor:
        """norm(x) in the step's dtype, after what is pending has been added to x."""
        if self.pending is None:
            return norm.forward(x, self.dtype)
        y, n, rows = self.pending, self.pending_norm, self.pending_rows
        self.pending = self.pending_norm = self.pending_rows = None
        if rows is not None:
            return norm.add_forward(x, y.contiguous(), self.dtype, rows)
        if n is None:
            return norm.add_forward(x, y.contiguous(), self.dtype)
        return n.add_into(x, y.contiguous(), then=norm, out_dtype=self.dtype)

    # A residual of several streams x [T, S, hidden]: a sublayer's output waits in the same place (``defer_streams``), and the pass that
    # brings it into the streams also makes what the next sublayer reads (``streams_normed``) or, behind the last layer, their sum.
    def defer_streams(self, x: torch.Tensor, y: torch.Tensor, mix: "Part") -> None:
        self.settle(x)
        self.pending, self.pending_streams = y.contiguous(), mix

    def streams_normed(self, x: torch.Tensor, mix: "Part", norm: "Norm") -> torch.Tensor:
        """norm(sum_s mix.in[s] x_s) in the step's dtype, after what is pending has entered the streams."""
        return self._mix_streams(x, x if self.pending is not None else None, mix.in_weights, norm.weight, norm.eps, self.dtype)

    def streams_sum(self, x: torch.Tensor) -> torch.Tensor:
        """The sum of the streams [T, hidden] float32, with what is pending (the streams themselves are not brought up to date)."""
        return self._mix_streams(x, None, out_dtype=torch.float32)

    def _mix_streams(self, x, dst=None, in_weights=None, norm_weight=None, eps=0.0, out_dtype=None):
        from ..ops import kernels
        y, m = self.pending, self.pending_streams
        self.pending = self.pending_streams = None
        src = x if self.stream_source is None else self.stream_source
        if dst is not None:
            self.stream_source = None                      # from here on the streams stand in x
        return kernels.stream_mix(src, x.shape[1], dst, y, None if m is None else m.mix, None if m is None else m.out_weights, in_weights,
                                  norm_weight, eps, out_dtype)

    def kv(self, cache_entry: int) -> KVView:
        g = self.cache.group_of[cache_entry]
        k, v = self.cache.pools(cache_entry)
        t = self.tables[g]
        return KVView(k, v, t, t.shape[1], self.cache.groups[g].need.window)

    def state(self, cache_entry: int) -> Optional[torch.Tensor]:
        """[slot, elems] float32; row ``slots[b]`` is batch row b's state."""
        return self.cache.state_of(cache_entry)


def normed_rows(h, x_norm, ctx, w):
    """What a part's first product reads: either rows ``h`` that are normed already, or, for a step of few rows in
    bfloat16 whose weight ``w`` the fused decode product takes, the float32 stream and its RMS norm (``x_norm`` = (x, norm)),
    which that product applies in its prologue.  Returns (h, norm_of, norm_weight, eps); exactly one of h and norm_of is set."""
    if x_norm is None:
        return h, None, None, 0.0
    from ..ops import kernels
    from .norm import RMSNorm
    x, norm = x_norm
    if ctx.dtype == torch.bfloat16 and type(norm) is RMSNorm and kernels.fused_takes(x.shape[0], w, x):
        return None, x, norm.weight, norm.eps
    return norm.forward(x, ctx.dtype), None, None, 0.0


def first_product(h, norm_of, norm_weight, eps, w, ctx):
    """The product of ``normed_rows``'s answer with ``w`` in the step's dtype."""
    from ..ops import kernels, linear
    if norm_of is not None:
        return kernels.linear_fused(None, w, out_dtype=ctx.dtype, norm_of=norm_of, norm_weight=norm_weight, eps=eps)
    return linear(h, w, out_dtype=ctx.dtype)


def last_product_into(x, a, w, scale, ctx):
    """x += scale * a . w^T on the float32 stream: in the epilogue of the fused decode product where it takes the sizes,
    else the product's float32 sums followed by the scaled sum."""
    from ..ops import kernels, linear
    if a.dtype == torch.bfloat16 and kernels.fused_takes(a.shape[0], w, a):
        kernels.linear_fused(a, w, accumulate_into=x, scale=scale)
    else:
        kernels.scaled_add(x, linear(a, w, out_dtype=torch.float32), scale)


class Part:
    def __init__(self, spec: PartSpec, dtype: torch.dtype, device):
        self.spec, self.dtype, self.device = spec, dtype, device

    def expected_tensors(self) -> Dict[str, ParamSpec]:
        return {}

    def take_tensors(self, get: Callable[[str], torch.Tensor]) -> None:
        pass

    def prepare(self, max_positions: int) -> None:
        """Called once before the first step, with the longest sequence the cache can hold."""

    def weights(self) -> List[torch.Tensor]:
        """The tensors a step reads in full (for traffic accounting)."""
        return [v for v in vars(self).values() if isinstance(v, torch.Tensor)]


class Norm(Part):
    def forward(self, x: torch.Tensor, out_dtype: torch.dtype, rows_index: Optional[torch.Tensor] = None) -> torch.Tensor:
        raise NotImplementedError

    def add_forward(self, x: torch.Tensor, y: torch.Tensor, out_dtype: torch.dtype, rows: Optional[tuple] = None) -> torch.Tensor:
        """x += y in place (``rows`` = (r, w): and w[t] * r[t]), then forward(x); norms override this to do both in one pass."""
        from ..ops import kernels
        if rows is not None:
            kernels.add_layernorm(x, y, rows=rows[0], row_weights=rows[1])
        else:
            kernels.residual_add(x, y)
        return self.forward(x, out_dtype)

    def add_into(self, x: torch.Tensor, y: torch.Tensor, then: Optional["Norm"] = None, out_dtype: Optional[torch.dtype] = None):
        """x += forward(y) in place on the float32 stream (y: a sublayer's output, float32 or the step's dtype); with ``then`` also
        returns then.forward(x) of the rows as they then stand.  Norms override this to do all of it in one pass."""
        from ..ops import kernels
        kernels.residual_add(x, self.forward(y if y.dtype == torch.float32 else y.float(), torch.float32))
        return None if then is None else then.forward(x, out_dtype)


class Position(Part):
    def rotate_and_store(self, qkv: torch.Tensor, n_q: int, n_kv: int, head_dim: int, ctx: StepContext,
                         kv: Optional[KVView]) -> None:
        raise NotImplementedError


class Mixer(Part):
    takes_pending = False      # True: add_to copes with a sum that is still pending (StepContext.normed / settle)

    def cache_needs(self) -> CacheNeeds:
        return CacheNeeds()

    def apply(self, h: torch.Tensor, ctx: StepContext, entry: int, cache_entry: int, owns_cache: bool) -> torch.Tensor:
        raise NotImplementedError

    def add_to(self, x: torch.Tensor, norm: Norm, ctx: StepContext, entry: int, cache_entry: int, owns_cache: bool) -> None:
        """x += apply(norm(x)); parts override this to fuse the norm and the residual sum."""
        from ..ops import kernels
        kernels.residual_add(x, self.apply(norm.forward(x, ctx.dtype), ctx, entry, cache_entry, owns_cache).contiguous())


class SharedProducts:
    """What a mixer offers so that it can stand beside another one on the same input with one first and one last product for both
    (``BranchSum`` without norms).  ``col`` is the first of the mixer's columns in the rows of the shared first product."""

    def can_share(self) -> bool:
        return False

    def give_input(self):
        """(weights, biases or None) of the first product, rows a multiple of 8; the mixer keeps none of its own after this."""
        raise NotImplementedError

    def give_output(self) -> torch.Tensor:
        raise NotImplementedError

    def prepare_jobs(self, proj, col: int, ctx, cache_entry: int, owns_cache: bool):
        """(kernels.NormedHeads or None, kernels.TurnedHeads or None): what has to be done to this mixer's columns first."""
        return None, None

    def mixed_rows(self, proj, col: int, turned, ctx, cache_entry: int, owns_cache: bool) -> torch.Tensor:
        """The heads' outputs, before norm and gate; ``turned``: the rows a TurnedHeads job made."""
        raise NotImplementedError

    def gate_job(self, rows, col: int, scale: float):
        """kernels.GatedRows: norm, gate and the weight of this mixer."""
        raise NotImplementedError


class JoinedProducts:
    """What a sublayer (mixer or feed-forward) offers so that it can stand beside another one that reads the same normed rows: the
    sublayers' first products are then one and so are their last products, whose sum over columns adds the sublayers up
    (``parts/joined.py``).  Between the two a sublayer reads its columns of the first product's rows and writes its columns of the rows
    of the last one."""

    def can_join(self) -> bool:
        return False

    def lend_products(self):
        """(first weight [rows, hidden], last weight [hidden, columns]); the sublayer keeps neither after this."""
        raise NotImplementedError

    def fill_side(self, proj, col: int, side, side_col: int, h, ctx, cache_entry: Optional[int] = None, owns_cache: bool = True):
        """Columns ``side_col`` .. of ``side`` from columns ``col`` .. of ``proj`` (and the normed rows h).  Returns None, or (rows, weights): rows
        [T, hidden] that the sublayer's output also contains, times a float32 number a token."""
        raise NotImplementedError


class InputFilter(Part):
    """Applied to the normed rows a sublayer reads; may keep per-sequence state (``state_elems`` float32 numbers)."""

    def state_elems(self) -> int:
        return 0

    def apply(self, y: torch.Tensor, ctx: StepContext, state: Optional[torch.Tensor], offset: int, out_dtype) -> torch.Tensor:
        raise NotImplementedError


class StreamPosition(Part):
    """Positions that enter the residual stream once, after the embedding."""

    def add_to(self, x: torch.Tensor, ctx: StepContext) -> None:
        raise NotImplementedError


class FeedForward(Part):
    takes_pending = False

    def apply(self, h: torch.Tensor, ctx: StepContext) -> torch.Tensor:
        raise NotImplementedError

    def add_to(self, x: torch.Tensor, norm: Norm, ctx: StepContext) -> None:
        from ..ops import kernels
        kernels.residual_add(x, self.apply(norm.forward(x, ctx.dtype), ctx).contiguous())


# ------------------------------------------------------------------ registries

NORMS: Dict[type, type] = {}
POSITIONS: Dict[type, type] = {}
MIXERS: Dict[type, type] = {}
FEED_FORWARDS: Dict[type, type] = {}
INPUT_FILTERS: Dict[type, type] = {}
STREAM_POSITIONS: Dict[type, type] = {}
ARRANGEMENTS: Dict[str, Callable] = {}


def _register(table: Dict[type, type], spec_class: type):
    def deco(cls):
        table[spec_class] = cls
        return cls
    return deco


def register_norm(spec_class: type):
    return _register(NORMS, spec_class)


def register_position(spec_class: type):
    return _register(POSITIONS, spec_class)


def register_mixer(spec_class: type):
    return _register(MIXERS, spec_class)


def register_feed_forward(spec_class: type):
    return _register(FEED_FORWARDS, spec_class)


def register_input_filter(spec_class: type):
    return _register(INPUT_FILTERS, spec_class)


def register_stream_position(spec_class: type):
    return _register(STREAM_POSITIONS, spec_class)


def register_arrangement(name: str):
    def deco(fn):
        ARRANGEMENTS[name] = fn
        return fn
    return deco


def build_part(table: Dict[type, type], kind: str, spec: PartSpec, dtype, device) -> Part:
    try:
        cls = table[type(spec)]
    except KeyError:
        known = ", ".join(sorted(c.__name__ for c in table)) or "none"
        raise ConfigError(f"no {kind} is registered for {type(spec).__name__}; registered: {known}") from None
    return cls(spec, dtype, device)
