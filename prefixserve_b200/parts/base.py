"""What every part of a model has in common, and what a part sees of a step.

A part is built from a ``PartSpec`` (its kind plus sizes and constants),
declares the tensors it needs by local name, receives them once, and then runs
on the tokens of a step.  It never learns which model it sits in.
"""

from __future__ import annotations

from dataclasses import dataclass, field
from typing import Any, Mapping, Sequence

import torch


@dataclass(frozen=True)
class ParamSpec:
    """One tensor a part wants from the checkpoint.

    role: "matrix" (operand of a matrix product: held in the compute dtype
    unless the file stores it in 32-bit), "vector" (norm gains and the like:
    always widened to float32, which is exact), or "table_int" (int32).
    init: how the random-weights mode fills it ("normal" or "ones").
    """

    shape: tuple[int, ...]
    role: str = "matrix"
    init: str = "normal"


@dataclass(frozen=True)
class PagedKV:
    """Keys and values for every token (or the last ``window`` of them)."""

    num_kv_heads: int
    head_dim: int
    window: int | None = None
    key_order: str = "natural"  # how a key head's elements are ordered in the pages; writer and readers must agree
    planes: int = 2  # 2: keys and values side by side; 1: one row per token that serves as both (a shared latent)
    # Chunked attention: a query sees only keys of its own run of ``chunk`` positions (runs counted from position 0), so
    # the pages before the run of the next token are never read again and go back to the pool like pages behind a window.
    chunk: int | None = None
    # With a window: the first ``keep_first`` keys of a sequence stay readable by every later query, so their pages are
    # never given back while the request lives; the pages between them and the window are.
    keep_first: int = 0

    def same_layout(self, other: "PagedKV") -> bool:
        """Whether two needs describe the same rows in the pages (they may differ in how far back they read)."""
        return (self.num_kv_heads, self.head_dim, self.key_order, self.planes) == \
               (other.num_kv_heads, other.head_dim, other.key_order, other.planes)

    def reach_of_both(self, other: "PagedKV") -> "PagedKV":
        """The need of an entry that this need writes and ``other`` also reads: nothing either still reads is let go."""
        import dataclasses
        window = None if self.window is None or other.window is None else max(self.window, other.window)
        chunk = self.chunk if self.chunk == other.chunk else None
        if chunk is None and (self.chunk is not None or other.chunk is not None):
            window = None  # a chunk mask on one side only: keep everything
        keep = max(self.keep_first, other.keep_first) if window is not None else 0
        return dataclasses.replace(self, window=window, chunk=chunk, keep_first=keep)


@dataclass(frozen=True)
class FixedState:
    """A per-request tensor of fixed shape that a mixer carries across steps."""

    shape: tuple[int, ...]
    dtype: torch.dtype = torch.float32


@dataclass(frozen=True)
class CacheNeed:
    paged: PagedKV | None = None
    state: FixedState | None = None


@dataclass
class CacheView:
    """The cache entry a mixer call works on."""

    group: int | None          # which page table of the step applies (None: no pages)
    kv: torch.Tensor | None    # [num_pages, 2, num_kv_heads, page_size, head_dim]
    state: torch.Tensor | None  # [num_slots, *shape]
    page_size: int
    writes: bool = True


@dataclass(frozen=True)
class ItemView:
    """Host-side view of one batch item: tokens [start, end) of one request."""

    slot: int
    start: int
    end: int
    first_token: int  # offset of its first token in the flat batch


@dataclass
class StepContext:
    """Everything about the current batch that parts may read."""

    num_tokens: int
    num_items: int
    compute_dtype: torch.dtype
    device: torch.device
    items: Sequence[ItemView]            # host side
    token_ids: torch.Tensor              # [T] int32
    positions: torch.Tensor              # [T] int32, absolute
    token_item: torch.Tensor             # [T] int32, index into items
    item_start: torch.Tensor             # [B+1] int32, offsets into the flat batch
    kv_len: torch.Tensor                 # [B] int32, tokens held after this step
    slots: torch.Tensor                  # [B] int32
    block_tables: Mapping[int, torch.Tensor]   # group -> [B, width] int32, by absolute page index
    max_new_tokens: int                  # longest item of the step
    max_kv_len: int                      # largest kv_len of the step
    all_decode: bool                     # every item brings exactly one token
    extras: dict[str, Any] = field(default_factory=dict)


class Part:
    """Base class; subclasses override what they need."""

    # A mixer, feed-forward or head that hands its input straight to ``ops.linear`` / ``ops.gated_linear`` sets this
    # and then receives an ``ops.NormedRows`` instead of a tensor (see ``Norm.defer``).
    takes_deferred_input = False

    # True when forward() launches the same device work for the same tensor shapes, reading everything that varies
    # from device memory (then a decode step can be captured once and replayed).  A part that loops over
    # ``ctx.items`` on the host must leave this False.
    graph_safe = False

    # A mixer or feed-forward whose result is one matrix product of rows it has made may offer those rows instead: how many
    # numbers a token they have (0: not offered).  ``forward_rows(x, ctx[, cache], out=...)`` then leaves them in ``out``
    # [T, rows_width] (may be a run of columns of a wider tensor) and ``output_weight()`` is the matrix [H, rows_width] that
    # the result is their product with.  Whoever adds the results of several such parts multiplies once, by the matrices
    # side by side (see ``Block.join_outputs``); ``drop_output_weight()`` says that nobody asks for ``forward`` any more.
    rows_width = 0

    def output_weight(self) -> torch.Tensor:
        raise NotImplementedError

    def drop_output_weight(self) -> None:
        raise NotImplementedError

    def __init__(self, spec_params: Mapping[str, Any]) -> None:
        self.params = dict(spec_params)

    def param_specs(self) -> dict[str, ParamSpec]:
        return {}

    def load(self, tensors: Mapping[str, torch.Tensor], *, compute_dtype: torch.dtype, device: torch.device) -> None:
        """Receives the tensors named in param_specs (already on the device)."""

    def prepare(self, *, max_positions: int, compute_dtype: torch.dtype, device: torch.device) -> None:
        """Builds start-up tables that depend on engine limits (e.g. rotary angles)."""


class Mixer(Part):
    def cache_need(self) -> CacheNeed:
        return CacheNeed()

    def forward(self, x: torch.Tensor, ctx: StepContext, cache: CacheView) -> torch.Tensor:  # [T,H] -> [T,H]
        raise NotImplementedError


class Gate(Part):
    """A gate on a sublayer's result, computed from the sublayer's input: ``forward`` returns the pre-activations
    [T, H]; ``bias`` (float32 [H] or None) is added and the sigmoid taken by the kernel that applies the gate."""

    bias: torch.Tensor | None = None

    def forward(self, x: torch.Tensor, ctx: StepContext) -> torch.Tensor:
        raise NotImplementedError


class FeedForward(Part):
    def forward(self, x: torch.Tensor, ctx: StepContext) -> torch.Tensor:
        raise NotImplementedError


class Norm(Part):
    def forward(self, h: torch.Tensor, delta: torch.Tensor | None, ctx: StepContext,
                rows: torch.Tensor | None = None) -> torch.Tensor:
        """h: float32 residual stream [T,H]; delta: pending sublayer output or None.

        Adds delta into h (in place, in float32) and returns the normalised
        rows in the compute dtype.  With ``rows`` only those rows are read and
        h is left untouched (last use of the stream).
        """
        raise NotImplementedError

    def defer(self, h: torch.Tensor, delta: torch.Tensor | None, ctx: StepContext, rows: torch.Tensor | None = None):
        """Same, for a consumer that declares ``takes_deferred_input``: returns an ``ops.NormedRows``, which the
        consumer passes to ``ops.linear`` / ``ops.gated_linear`` (they may do the norm inside the product) or turns
        into a tensor with ``.tensor()``.  A norm without a deferred form computes now and wraps the result."""
        from ..ops import NormedRows
        return NormedRows.ready(self.forward(h, delta, ctx, rows), h)


class PositionEncoding(Part):
    pass
