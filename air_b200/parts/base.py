"""What every part must offer.

A part is built from its description alone (sizes and constants are parameters, nothing is
read from a model's configuration), says which tensors it needs, takes them when they are
loaded, and computes.  No part knows which model it is in, which layer it is, or what the
other parts of its block are.

  Norm              forward(h, delta, rows=None) -> normalised rows in the compute dtype.  h is the
                    float32 residual stream [T, hidden]; `delta` is what the part before the norm
                    produced and has NOT yet been added to the stream: None, a tensor [T, hidden]
                    (float32 or the compute dtype), or float32 partial sums [parts, T, hidden] that
                    are to be added in the order of `parts`.  Without `rows` the norm adds delta into
                    h in place and normalises every row; with `rows` (int32 indices) it leaves h as it
                    is and returns the norm of h[rows] + delta[rows].  A norm that does not want to
                    know about the forms of delta calls `self.add_delta(h, delta)` first, which is the
                    package's kernel for exactly that sum, and then works on h alone.
  PositionEncoding  table() -> float32 [positions, rotary width] cos|sin, consumed by mixers
  Mixer             cache_needs() -> what it keeps per request (CacheNeed objects: pages of keys and
                    values, pages of something else, a state of fixed size, several, or nothing);
                    plan(batch) -> what it wants worked out on the host once per step (optional);
                    forward(x, ctx, cache, owns_cache) -> [T, hidden], or float32 [parts, T, hidden]
                    partial sums, or None after adding its output into ctx.residual itself
  FeedForward       forward(x, ctx) -> as a mixer
  RowFilter         what stands between a norm and the part that reads its rows: forward(x, ctx, view) -> rows in the
                    compute dtype from float32 rows; may keep a state per request (cache_needs)
  Block             forward(h, pending, ctx, cache, owns_cache) -> (h, pending): an arrangement of
                    parts around the residual stream; `pending` is a delta in the sense above
  Embedding         forward(ctx, cache, copies) -> the stream's first rows from the step's token ids; may keep a
                    state per request (cache_needs) like a mixer
"""
from __future__ import annotations

from dataclasses import dataclass, field
from typing import Dict, Hashable, List, Optional, Sequence, Tuple

import torch

from ..weights.loader import TensorSpec
from .spec import PartSpec


@dataclass
class Runtime:
    """Where and how the parts compute: the device, the compute dtype (bfloat16 or
    float32; float32 means no reduced-precision step anywhere) and the page size.  `shared`
    holds what equal parts of different layers make once and share (a position table)."""
    device: torch.device
    dtype: torch.dtype
    page_tokens: int = 64
    status: Optional[torch.Tensor] = None    # [1] int32 on the device: kernels report impossible states here
    shared: Dict[Hashable, object] = field(default_factory=dict)

    @property
    def is_fp32(self) -> bool:
        return self.dtype == torch.float32


# ------------------------------------------------------------------ what a mixer keeps per request
class CacheNeed:
    """One thing a mixer keeps per request.  The cache manager knows no kinds of need: it asks
    each need for the shape of its memory and hands the mixer what `view` returns.

    A *paged* need keeps something for every token: the manager makes one slab
    [pages, *page_shape(page_tokens)] per run and gives the request pages of it, through a block
    table that runs with an equal `group_key()` share.  `window` (None: everything is kept) lets
    the manager take back pages whose tokens no later query can see.  A need that is not paged
    keeps `slot_shape()` per request, zeroed when the request opens."""
    paged: bool = False
    window: Optional[int] = None
    chunk: Optional[int] = None

    def group_key(self) -> Hashable:
        return self

    def first_live(self, length: int) -> int:
        """The lowest position that a query at position `length` or later can still see: pages that hold only
        earlier tokens go back to the pool.  A window keeps the last `window` keys; chunks (a query sees the keys of
        its own chunk of `chunk` positions, counted from 0) keep the chunk that position `length` lies in."""
        if self.window is not None:
            return max(0, length - self.window + 1)
        if self.chunk is not None:
            return length - length % self.chunk
        return 0

    def page_shape(self, page_tokens: int) -> Tuple[int, ...]:
        raise NotImplementedError

    def slot_shape(self) -> Tuple[int, ...]:
        raise NotImplementedError

    def element_dtype(self, compute_dtype: torch.dtype) -> torch.dtype:
        return compute_dtype

    def view(self, tensor: Optional[torch.Tensor], group: Optional[int]):
        """What the mixer's forward() receives for this need."""
        raise NotImplementedError

    def bytes_per_page(self, page_tokens: int, compute_dtype: torch.dtype) -> int:
        n = 1
        for s in self.page_shape(page_tokens):
            n *= s
        return n * torch.empty((), dtype=self.element_dtype(compute_dtype)).element_size()


@dataclass
class PagedKVView:
    """What a mixer gets for a PagedKV need: its slab [pages, 2, kv_heads, page_tokens, head_dim]
    and the index of its group (for the step's block table)."""
    kv: Optional[torch.Tensor]
    group: int
    need: "PagedKV"


@dataclass
class SlotStateView:
    """What a mixer gets for a SlotState need: [slots, *shape]; row = the request's slot."""
    state: Optional[torch.Tensor]
    need: "SlotState"


@dataclass(frozen=True)
class PagedKV(CacheNeed):
    """Keys and values of every token, in pages.  window: None keeps all keys, a number
    keeps the last `window` of them (older pages are given back).  Layers with equal needs
    share a group: one pool of pages and one block table.  v_dim: the size of a value where it
    differs from a key's (head_dim); a page is then flat, the keys [kv_heads, page_tokens, head_dim]
    followed by the values [kv_heads, page_tokens, v_dim]."""
    kv_heads: int
    head_dim: int
    window: Optional[int] = None
    v_dim: Optional[int] = None
    chunk: Optional[int] = None
    paged = True

    def page_shape(self, page_tokens):
        if self.v_dim is None or self.v_dim == self.head_dim:
            return (2, self.kv_heads, page_tokens, self.head_dim)
        return (self.kv_heads * page_tokens * (self.head_dim + self.v_dim),)

    def view(self, tensor, group):
        return PagedKVView(tensor, group, self)


@dataclass
class PagedLatentView:
    """What a mixer gets for a PagedLatent need: its slab [pages, page_tokens, width] and the index of its group."""
    rows: Optional[torch.Tensor]
    group: int
    need: "PagedLatent"


@dataclass(frozen=True)
class PagedLatent(CacheNeed):
    """One row of `width` numbers per token, in pages [page_tokens, width], with no heads: what attention over a
    compressed latent keeps (the latent and a rotated key part that all heads share).  window as for PagedKV: the
    largest window of the layers that read the rows, None if one of them sees everything."""
    width: int
    window: Optional[int] = None
    paged = True

    def page_shape(self, page_tokens):
        return (page_tokens, self.width)

    def view(self, tensor, group):
        return PagedLatentView(tensor, group, self)


@dataclass(frozen=True)
class SlotState(CacheNeed):
    """A state of fixed size per request (zeroed when the request opens), as a recurrent
    or convolutional mixer keeps it."""
    shape: Tuple[int, ...]
    dtype: str = "float32"
    paged = False

    def slot_shape(self):
        return tuple(self.shape)

    def element_dtype(self, compute_dtype):
        return getattr(torch, self.dtype)

    def view(self, tensor, group):
        return SlotStateView(tensor, self)


# ------------------------------------------------------------------ what a part may plan on the host
@dataclass
class HostBatch:
    """One step's batch as the host knows it, for parts that work something out per step before
    the kernels run (lists of tiles, schedules).  Entry i brings counts[i] next tokens of a request
    that holds lengths[i] tokens already; its tokens are rows q_start[i] .. q_start[i + 1] of the
    step; slots[i] is the request's state slot."""
    counts: List[int]
    lengths: List[int]
    slots: List[int]
    q_start: List[int]


@dataclass
class Plan:
    """What `plan` returns: int32 arrays that the step copies to the device with the rest of the
    batch (the part finds them as device tensors under the same names), and plain host values."""
    arrays: Dict[str, "object"] = field(default_factory=dict)     # name -> numpy int32 array (any shape)
    values: Dict[str, object] = field(default_factory=dict)


@dataclass
class PreNormed:
    """Rows that an RMSNorm would produce, short of the scale per row: x = bfloat16(h * weight), and the sums
    of squares of h per row in parts (ss [parts, T], to be added in order): the row's scale is
    rsqrt(sum / width + eps).  One number per row commutes with a matrix product, so a product that takes these
    rows applies the scale to its accumulators.  A norm of the form x * scale(row) * weight writes its rows so
    (Norm.forward_prenormed) where the part behind it says that it takes them in this step
    (Part.accepts_prenormed): the kernel that writes them has no block that waits for a row's other blocks."""
    x: torch.Tensor
    ss: torch.Tensor
    eps: float

    @property
    def shape(self):
        return self.x.shape

    @property
    def dtype(self):
        return self.x.dtype

    @property
    def device(self):
        return self.x.device


@dataclass
class ScaledSum:
    """What parts that stand side by side add to the stream together: the sum of scale * gate * term over `terms`, a list
    of (float32 [T, hidden], or [parts, T, hidden] partial sums of a split product; float32 [hidden] or None: a scale
    per column; optionally float32 [T] or None: a gate per row).  A form of a norm's `delta`: the norm
    that follows completes the stream with it (Norm.add_delta, or a kernel of its own that also normalises)."""
    terms: list


@dataclass
class GatedSum:
    """a + gate[row] * b: what a feed-forward adds to the stream when one of its branches carries a gate of one number
    per token.  a, b: None, float32 [T, hidden] or partial sums [parts, T, hidden]; gate: float32 [T] or None (1).  A
    form of a norm's `delta`."""
    a: Optional[torch.Tensor]
    b: Optional[torch.Tensor]
    gate: Optional[torch.Tensor]


@dataclass
class NormedSum:
    """What a sub-layer with a norm BEHIND it adds to the stream: term / sqrt(mean(term^2) + eps) * weight, with term
    float32 [T, hidden] or [parts, T, hidden] partial sums (added in order first) and weight float32 [hidden].  A form
    of a norm's `delta`: the norm that follows takes the norm of the term, completes the stream with it and normalises
    the stream in one kernel."""
    term: torch.Tensor
    weight: torch.Tensor
    eps: float


def row_terms(delta) -> Optional[list]:
    """A delta as a list of (float32 [T, hidden] or [parts, T, hidden], gate per row float32 [T] or None) to be added up, for
    kernels that take that form; None where it has no such form (scales per column, a norm behind the sub-layer, several
    streams, 16-bit tensors, more than three terms)."""
    if delta is None:
        return []
    if isinstance(delta, torch.Tensor):
        terms = [(delta, None)]
    elif isinstance(delta, GatedSum):
        terms = [(t, g) for t, g in ((delta.a, None), (delta.b, delta.gate)) if t is not None]
    elif isinstance(delta, ScaledSum):
        if any(t[1] is not None for t in delta.terms):
            return None
        # (the kernels take a gate on every term but the first)
        terms = sorted(((t[0], t[2] if len(t) > 2 else None) for t in delta.terms), key=lambda t: t[1] is not None)
    else:
        return None
    if len(terms) > 3 or any(t.dtype != torch.float32 for t, _ in terms) or (terms and terms[0][1] is not None):
        return None
    return terms


@dataclass
class StreamSum:
    """What a sub-layer of a block with several residual streams hands on (hyper-connections): the streams
    x_0 .. x_(S-1) become x'_t = sum_s mix[s, t] x_s + out[t] * term, with term float32 [T, hidden] or partial sums
    [parts, T, hidden], mix float32 [S, S], out float32 [S].  A form of a norm's `delta` for a stream h [S, T, hidden], or
    h [T, hidden] while all streams are still equal."""
    term: torch.Tensor
    mix: torch.Tensor
    out: torch.Tensor


class Part:
    # True if forward() only launches work on the current stream from device data (no host
    # reads of the batch or of a result), so that a decode step can be captured in a CUDA graph.
    graph_safe: bool = False

    def __init__(self, spec: PartSpec, prefix: str = ""):
        self.spec = spec
        self.prefix = prefix

    def tensor_specs(self) -> List[TensorSpec]:
        return []

    def load(self, tensors: Dict[str, torch.Tensor], rt: Runtime) -> None:
        self.rt = rt

    # A part that wants something worked out on the host once per step names it with a key (parts
    # with equal keys share one plan: 28 attention layers plan once) and builds it in plan().  The
    # result is at ctx.plans[key]: a namespace with the arrays as device tensors and the values.
    def plan_key(self) -> Optional[Hashable]:
        return None

    def plan(self, batch: HostBatch) -> Optional[Plan]:
        return None

    def accepts_prenormed(self, ctx, owns_cache: bool = True) -> bool:
        """Whether forward() in this step takes its input as a PreNormed (see there)."""
        return False


class Norm(Part):
    def forward(self, h, delta, rows=None):
        raise NotImplementedError

    @staticmethod
    def add_delta(h: torch.Tensor, delta) -> torch.Tensor:
        """h += delta for every form of delta that a part may hand on (see the module's text); returns h, or for a
        StreamSum the completed streams [S, T, hidden] (h itself unless its streams were still one tensor)."""
        if delta is not None:
            from ..csrc import ops
            if isinstance(delta, StreamSum):
                S = delta.out.shape[0]
                full = h if h.dim() == 3 else torch.empty((S,) + tuple(h.shape), dtype=h.dtype, device=h.device)
                ops.stream_norm(h, S, None, None, 0.0, None, term=delta.term, mix=delta.mix, out_weights=delta.out,
                                h_out=full)
                return full
            if isinstance(delta, ScaledSum) and (len(delta.terms) > 2 or any(len(t) > 2 for t in delta.terms)):
                terms = row_terms(delta)
                if terms is None:
                    raise ops.KernelError("a sum of more than two terms, or with a gate per row, takes no scales per column")
                ops.stream_norm(h, 1, None, None, 0.0, None, term=terms[0][0], more=terms[1:], h_out=h)
            elif isinstance(delta, ScaledSum):
                ops.scaled_norm(h, delta.terms, None, 0.0, None)
            elif isinstance(delta, GatedSum):
                ops.post_norm(h, 1.0, delta.a, delta.b, delta.gate, None, 0.0, None)
            elif isinstance(delta, NormedSum):
                ops.normed_add_norm(h, delta.term, delta.weight, delta.eps, None, 0.0, None)
            else:
                ops.add_parts(h, delta)
        return h


class PositionEncoding(Part):
    rotary_dim: int = 0

    def table(self) -> Optional[torch.Tensor]:
        return None

    def frequencies(self) -> Optional[torch.Tensor]:
        """float32 [rotary_dim / 2]: the angle of pair i at position p is p * frequencies[i], for mixers whose
        kernels evaluate the angles themselves instead of reading a table (no bound on the position)."""
        return None


class Embedding(Part):
    """From token ids to rows of the stream.  forward(ctx, cache, copies) -> `copies` float32 tensors [T, hidden]
    with the same contents (the stream itself, and one more where later runs add the embedding's output again);
    `cache` holds the views of cache_needs(), as a mixer's does.  `table` is the token table [vocab, hidden], which a
    model with a tied output matrix reads again at the end."""
    table: Optional[torch.Tensor] = None

    def cache_needs(self) -> Tuple[CacheNeed, ...]:
        return ()

    def forward(self, ctx, cache, copies: int = 1):
        raise NotImplementedError


class RowFilter(Part):
    """Rows on their way from a norm (float32) to the part behind it (compute dtype).  single_tokens(ctx, cache): what
    the norm's kernel needs to apply the filter itself in a step in which every row is its request's only token, or None."""

    def cache_needs(self) -> Tuple[CacheNeed, ...]:
        return ()

    def single_tokens(self, ctx, cache):
        return None

    def forward(self, x, ctx, cache):
        raise NotImplementedError


class Mixer(Part):
    def cache_needs(self) -> Tuple[CacheNeed, ...]:
        return ()

    def forward(self, x, ctx, cache, owns_cache: bool):
        raise NotImplementedError


class FeedForward(Part):
    def forward(self, x, ctx):
        raise NotImplementedError
