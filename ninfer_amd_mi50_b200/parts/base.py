"""Interfaces that every part of a layer implements, and the step's shared metadata.

A part knows its own sizes and constants (constructor arguments that come from the
configuration through a `PartSpec`) and the names of its own tensors below a prefix.
It does not know which model it is in, how many layers there are, or what the other
parts of its block are.

Reference counterpart: ``Shard::layer_start`` / ``layer_mid`` / ``end_layer``
(src/models/model.hip:206-444) hard-wire one attention and one MLP/MoE into a
function; here the same stages are objects chosen layer by layer.
"""

from __future__ import annotations

from dataclasses import dataclass, field
from typing import Callable, Dict, List, Optional, Sequence, Tuple

import torch


# --------------------------------------------------------------------------------------
# Tensors a part needs from the checkpoint
# --------------------------------------------------------------------------------------

@dataclass(frozen=True)
class TensorSpec:
    """One checkpoint tensor a part asks for.

    role:  "matrix" - held in the engine dtype (bfloat16 or float32);
           "vector" - norm weights and biases, held in float32 in both modes (a
                      bfloat16 value widens exactly; a tensor stored in 32-bit stays so);
           "router" - routing matrices, held in float32 for the same reason;
           "table"  - integer tables, held as int32.
    init:  distribution for the random-weights mode: "linear" N(0, 0.02),
           "norm" 1 + N(0, 0.05); for a table "distinct:<n>": rows of different numbers below n.
    """
    name: str
    shape: Tuple[int, ...]
    role: str = "matrix"
    init: str = "linear"


Fetch = Callable[[str], torch.Tensor]   # tensor name -> device tensor in its role's dtype


# --------------------------------------------------------------------------------------
# What a mixer asks of the cache manager
# --------------------------------------------------------------------------------------

@dataclass(frozen=True)
class CacheSpec:
    """What one cache slot keeps per token, in pages.

    kind "full": every entry stays until the request ends.
    kind "window": only the last `window` entries are read; pages that the window has
    passed go back to the pool.  With `keep_first`, a request's first `keep_first` entries stay
    readable however far the window has moved: the pages that hold them are never given back.

    The usual form is keys and values of `num_kv_heads` heads of `head_dim`: a page is
    ``[2, num_kv_heads, page_size, head_dim]`` (keys, then values; one head's keys of a page are
    one contiguous run), which is what the attention kernels read.  A mixer that keeps
    something else per token (one compressed latent row, keys and values of different widths
    packed side by side) gives `row_width` instead: a page is then ``[page_size, row_width]``
    and the mixer reads and writes it itself.  The cache manager only ever asks `page_shape`.
    """
    kind: str
    num_kv_heads: int = 0
    head_dim: int = 0
    window: Optional[int] = None
    row_width: int = 0
    keep_first: int = 0

    def page_shape(self, page_size: int) -> Tuple[int, ...]:
        if self.row_width:
            return (page_size, self.row_width)
        return (2, self.num_kv_heads, page_size, self.head_dim)

    def elements_per_token(self) -> int:
        return self.row_width if self.row_width else 2 * self.num_kv_heads * self.head_dim

    def group_key(self) -> Tuple:
        return (self.kind, self.num_kv_heads, self.head_dim, self.window, self.row_width, self.keep_first)


@dataclass(frozen=True)
class StateSpec:
    """Per-request state of fixed size: one tensor of `shape` per live request."""
    shape: Tuple[int, ...]
    dtype: torch.dtype = torch.float32


@dataclass
class CacheView:
    """What a mixer call sees of one cache slot during a step."""
    spec: CacheSpec
    pages: torch.Tensor          # [num_pages + 1, *spec.page_shape(page_size)]
    block_table: torch.Tensor    # int32 [S, width]: page of (segment, position // page_size)
    page_size: int
    append: bool = True


# --------------------------------------------------------------------------------------
# The step's metadata, shared by all parts
# --------------------------------------------------------------------------------------

@dataclass
class StepContext:
    """Everything about a step that is not the hidden state.

    Rows are the step's tokens in order; a *segment* is one request's run of rows
    (a portion of a prompt, or one decoded token).  All index tensors are int32 on the
    device.  `seg_len_host` / `seg_pos0_host` are host copies for grid sizing; they are
    absent in graph mode, where only the bounds `max_rows_per_seg` and `max_context`
    may shape a launch.
    """
    dtype: torch.dtype
    device: torch.device
    T: int
    S: int
    token_ids: torch.Tensor        # [T]
    positions: torch.Tensor        # [T] absolute position of each row in its request
    row_seg: torch.Tensor          # [T] segment of each row
    seg_row0: torch.Tensor         # [S + 1] first row of each segment
    seg_pos0: torch.Tensor         # [S] tokens the request held before this step
    seg_slot: torch.Tensor         # [S] state slot of each segment's request
    logit_rows: torch.Tensor       # [R] rows whose logits are wanted
    block_tables: Dict[int, torch.Tensor] = field(default_factory=dict)  # per cache group
    seg_len_host: Optional[List[int]] = None
    seg_pos0_host: Optional[List[int]] = None
    max_rows_per_seg: int = 1
    max_context: int = 0           # bound on pos0 + rows over the segments of this step
    graph_mode: bool = False
    scratch: Dict[str, torch.Tensor] = field(default_factory=dict)
    _tiles: Dict[object, Tuple[torch.Tensor, int]] = field(default_factory=dict)

    @property
    def all_single(self) -> bool:
        """Every segment brings exactly one row (a decode-only step)."""
        return self.max_rows_per_seg == 1

    def _ints(self, values: Sequence[int]) -> torch.Tensor:
        """A host list as an int32 tensor on the device, without waiting for the stream (a copy from pageable
        memory would: the launches that follow could then not run ahead of the device)."""
        t = torch.tensor(values, dtype=torch.int32)
        return t.pin_memory().to(self.device, non_blocking=True) if self.device.type == "cuda" else t.to(self.device)

    def query_tiles(self, rows_per_tile: int) -> Tuple[torch.Tensor, int]:
        """Tiles of at most `rows_per_tile` consecutive rows of one segment.

        Returns (int32 [n, 2] of (segment, first row), n).  Built on the host from the
        segment lengths; not available in graph mode.
        """
        if rows_per_tile in self._tiles:
            return self._tiles[rows_per_tile]
        if self.seg_len_host is None:
            raise RuntimeError("query_tiles needs host segment lengths (not in graph mode)")
        flat: List[int] = []
        row = 0
        for s, n in enumerate(self.seg_len_host):
            for r in range(0, n, rows_per_tile):
                flat += [s, row + r]
            row += n
        n_tiles = len(flat) // 2
        t = self._ints(flat).view(n_tiles, 2)
        self._tiles[rows_per_tile] = (t, n_tiles)
        return t, n_tiles


    def chunked_query_tiles(self, rows_per_tile: int, chunk: int) -> Tuple[torch.Tensor, int]:
        """`query_tiles` for attention over chunks of `chunk` positions (0: plain causal), the tiles
        that read the most keys first: a tile's keys run from the start of its first row's chunk to
        its last row, and the device hands CTAs to SMs as they fall free, so the light tiles fill
        the end.  Built on the host; not available in graph mode."""
        key = ("chunked_query_tiles", rows_per_tile, chunk)
        if key in self._tiles:
            return self._tiles[key]
        if self.seg_len_host is None:
            raise RuntimeError("chunked_query_tiles needs host segment lengths (not in graph mode)")
        found = []
        pos0 = self.seg_pos0_host or [0] * len(self.seg_len_host)
        row = 0
        for s, n in enumerate(self.seg_len_host):
            for r in range(0, n, rows_per_tile):
                first, last = pos0[s] + r, pos0[s] + min(n, r + rows_per_tile) - 1
                start = (first // chunk) * chunk if chunk > 0 else 0
                found.append((-(last - start), s, row + r))
            row += n
        found.sort()
        flat: List[int] = [v for _, s, r in found for v in (s, r)]
        n_tiles = len(flat) // 2
        t = self._ints(flat).view(n_tiles, 2)
        self._tiles[key] = (t, n_tiles)
        return t, n_tiles

    def pair_tiles(self, heads: int, pairs_per_tile: int) -> Tuple[torch.Tensor, int]:
        """Tiles over the (row, head) pairs of every segment, `pairs_per_tile` consecutive pairs of
        one segment each (pair = row within the segment * heads + head).  Returns (int32 [n, 2] of
        (segment, first pair), n).  Built on the host; not available in graph mode."""
        key = ("pair_tiles", heads, pairs_per_tile)
        if key in self._tiles:
            return self._tiles[key]
        if self.seg_len_host is None:
            raise RuntimeError("pair_tiles needs host segment lengths (not in graph mode)")
        # heaviest first (a tile late in a long prompt reads many more keys than an early one): the
        # device hands CTAs to SMs as they fall free, so the light tiles fill the end
        found = []
        pos0 = self.seg_pos0_host or [0] * len(self.seg_len_host)
        for s, n in enumerate(self.seg_len_host):
            for p in range(0, n * heads, pairs_per_tile):
                last_row = min(n * heads, p + pairs_per_tile) - 1
                found.append((-(pos0[s] + last_row // heads), s, p))
        found.sort()
        flat: List[int] = [v for _, s, p in found for v in (s, p)]
        n_tiles = len(flat) // 2
        t = self._ints(flat).view(n_tiles, 2)
        self._tiles[key] = (t, n_tiles)
        return t, n_tiles

    def one_row_tiles(self) -> Tuple[Optional[torch.Tensor], int]:
        """A tile for every segment that brings exactly one row, as the flash kernels take them
        (int32 [n, 2, 2] of (segment, first row), the second entry (-1, -1)); (None, 0) if there is
        none.  When every segment brings one row it depends on the number of segments alone, so a
        step that is captured into a graph may use it: the tensor is made on the first (uncaptured)
        run and kept."""
        if "one_row" not in self._tiles:
            if self.seg_len_host is None:
                raise RuntimeError("one_row_tiles needs host segment lengths")
            flat, row = [], 0
            for s, n in enumerate(self.seg_len_host):
                if n == 1:
                    flat += [s, row, -1, -1]
                row += n
            n_tiles = len(flat) // 4
            self._tiles["one_row"] = ((self._ints(flat).view(n_tiles, 2, 2), n_tiles)
                                      if n_tiles else (None, 0))
        return self._tiles["one_row"]

    def single_rows(self) -> Tuple[Optional[torch.Tensor], int]:
        """Rows of the segments that bring exactly one row (decoded tokens, or a prompt's last
        token arriving alone), as (int32 tensor on the device, count); (None, 0) if there are
        none.  Attention serves such a row with its split-key kernel whatever else the step
        holds.  Built on the host; not available in graph mode."""
        if "single" in self._tiles:
            return self._tiles["single"]
        if self.seg_len_host is None:
            raise RuntimeError("single_rows needs host segment lengths (not in graph mode)")
        rows, row = [], 0
        for n in self.seg_len_host:
            if n == 1:
                rows.append(row)
            row += n
        out = (self._ints(rows), len(rows)) if rows else (None, 0)
        self._tiles["single"] = out
        return out

    def single_rows_context(self) -> Optional["StepContext"]:
        """The segments that bring exactly one row as a step of their own (rows in `single_rows` order), for a
        kernel that takes whole steps; None if there are none.  Built on the host; not in graph mode."""
        if "single_ctx" not in self._tiles:
            rows, n = self.single_rows()
            sub = None
            if n:
                segs = [s for s, m in enumerate(self.seg_len_host) if m == 1]
                idx = self.row_seg.index_select(0, rows)
                count = torch.arange(n + 1, dtype=torch.int32, device=self.device)
                pos0 = [self.seg_pos0_host[s] for s in segs]
                sub = StepContext(
                    dtype=self.dtype, device=self.device, T=n, S=n, token_ids=self.token_ids.index_select(0, rows),
                    positions=self.positions.index_select(0, rows), row_seg=count[:n], seg_row0=count,
                    seg_pos0=self.seg_pos0.index_select(0, idx), seg_slot=self.seg_slot.index_select(0, idx),
                    logit_rows=count[:0], block_tables={g: t.index_select(0, idx) for g, t in self.block_tables.items()},
                    seg_len_host=[1] * n, seg_pos0_host=pos0, max_rows_per_seg=1, max_context=max(pos0) + 1)
                sub.scratch["segments"] = idx
            self._tiles["single_ctx"] = sub
        return self._tiles["single_ctx"]

    def context_rows(self, min_rows: int) -> Tuple[torch.Tensor, int]:
        """Where each segment's whole context (what it held and what it brings) starts in a matrix that holds the
        contexts of all segments of at least `min_rows` rows one after the other: (int32 [S], -1 for the others;
        rows in all).  Built on the host; not in graph mode."""
        key = ("context_rows", min_rows)
        if key not in self._tiles:
            base, total = [], 0
            for n, p in zip(self.seg_len_host, self.seg_pos0_host):
                base.append(total if n >= min_rows else -1)
                total += p + n if n >= min_rows else 0
            self._tiles[key] = (self._ints(base), total)
        return self._tiles[key]

    def paired_query_tiles(self, rows_per_tile: int, window: int, keys_per_block: int,
                           pair: bool = True, min_rows: int = 1) -> Tuple[torch.Tensor, int]:
        """Query tiles two to a CTA, a heavy one with a light one.

        A tile late in a long prompt reads many more keys than an early one; giving each CTA
        the i-th heaviest and the i-th lightest tile makes CTAs about equally long.  Returns
        (int32 [n_pairs, 2, 2] of (segment, first row), second entry (-1, -1) if there is
        none; n_pairs).  With `pair` false every CTA gets one tile, heaviest first.  Segments
        with fewer than `min_rows` rows are left out (they are served elsewhere)."""
        if self.seg_len_host is None or self.seg_pos0_host is None:
            raise RuntimeError("paired_query_tiles needs host segment lengths (not in graph mode)")
        if min_rows > 1 and all(n >= min_rows for n in self.seg_len_host):
            min_rows = 1                         # nothing is left out: one list for all who ask
        key = ("pairs", rows_per_tile, window, keys_per_block, pair, min_rows)
        if key in self._tiles:
            return self._tiles[key]
        tiles = []
        row = 0
        for s, (n, pos0) in enumerate(zip(self.seg_len_host, self.seg_pos0_host)):
            for r in range(0, n if n >= min_rows else 0, rows_per_tile):
                first = pos0 + r
                last = pos0 + min(r + rows_per_tile, n) - 1
                lo = max(0, first - window + 1) if window > 0 else 0
                work = last // keys_per_block - lo // keys_per_block + 1
                tiles.append((work, s, row + r))
            row += n
        tiles.sort(key=lambda t: -t[0])
        flat: List[int] = []
        if not pair:
            # one tile a CTA, heaviest first: the device hands CTAs to SMs as they fall free, so
            # the light tiles fill the end
            for _, s, r in tiles:
                flat += [s, r, -1, -1]
        i, j = (0, len(tiles) - 1) if pair else (1, 0)
        while i <= j:
            flat += [tiles[i][1], tiles[i][2]]
            flat += [tiles[j][1], tiles[j][2]] if j > i else [-1, -1]
            i, j = i + 1, j - 1
        n_pairs = len(flat) // 4
        t = self._ints(flat).view(n_pairs, 2, 2)
        self._tiles[key] = (t, n_pairs)
        return t, n_pairs


# --------------------------------------------------------------------------------------
# Part interfaces
# --------------------------------------------------------------------------------------

class Part:
    """Common to all parts: which tensors it needs and how it takes them."""

    # True if `forward` only launches work on the current stream from device-side data
    # (no host reads of the step's contents), so that a step may be captured in a CUDA graph.
    graph_safe = False

    def tensor_specs(self) -> List[TensorSpec]:
        return []

    def load(self, fetch: Fetch) -> None:
        """Pull this part's tensors (`fetch(name)`), fusing or stacking as it likes."""

    def weight_bytes(self) -> int:
        """Bytes of weights one forward call reads when every row uses everything."""
        return 0

    def check_limits(self, dtype: torch.dtype, max_context: int, page_size: int) -> None:
        """Raise ValueError if this part's kernels cannot serve the engine's options.  Called
        once at start-up, so that a limit is met there and not in the middle of a request."""


@dataclass
class RoutedSum:
    """A feed-forward's output that has not been added up yet:

        out[t] = sum_j wts[t, j] * y[plan.inv[t * k + j]]  (+ sigmoid(gate[t]) * shared[t])

    A block hands it on as its pending contribution; a norm that knows the form (`takes_unsummed`)
    adds it up inside its own kernel, any other consumer calls `materialize()` first.
    """
    y: torch.Tensor                      # [T * k, hidden] expert outputs in sorted order
    plan: object                         # the routing plan (`inv` is what is used)
    wts: Optional[torch.Tensor]          # float32 [T, k]; None: every weight is 1
    shared: Optional[torch.Tensor]       # [T, hidden] or None
    gate: Optional[torch.Tensor]         # float32 [T, 1] gate logits or None
    dtype: torch.dtype = torch.bfloat16

    def materialize(self) -> torch.Tensor:
        from .. import kernels
        wts = self.wts
        if wts is None:
            wts = torch.ones((self.plan.num_tokens, self.plan.top_k), dtype=torch.float32, device=self.y.device)
        return kernels.moe_combine(self.y, self.plan, wts, self.shared, self.gate, self.dtype)


@dataclass
class StreamCopy:
    """What a block that adds its sublayers' outputs to the stream itself leaves "pending": nothing
    is left to add, and `x` is the stream as it stands, in the engine's type (None in 32-bit mode,
    where the stream itself serves) - the next such block's input, saved a pass over the stream."""
    x: Optional[torch.Tensor]


@dataclass
class BiasedOutput:
    """A sublayer's output whose bias has not been added yet: `y` [T, hidden] (float32 sums or the
    engine's type) and `bias` float32 [hidden].  A consumer that reads the rows anyway (the norm
    on a sublayer's output) adds the bias in its own pass; anything else calls `summed()`."""
    y: torch.Tensor
    bias: torch.Tensor


@dataclass
class StreamUpdate:
    """What a block over several residual streams leaves pending: its last sublayer's output `y`
    [T, hidden] with the constants of the update ``x_t <- sum_s mix[s, t] x_s + out[t] * y``
    (`mix` None: the identity; `out` None: ones).  Whoever reads the streams next applies it in its
    own pass over them (`kernels.streams_mix_norm`)."""
    y: torch.Tensor
    mix: Optional[torch.Tensor]
    out: Optional[torch.Tensor]


@dataclass
class PairSum:
    """The outputs of a mixer and a feed-forward that ran side by side on one input, both still to be added
    to the stream.  A norm that knows the form (`takes_pair`) adds both in its own pass, in 32-bit."""
    a: torch.Tensor
    b: torch.Tensor


@dataclass
class ScaledPair:
    """The outputs of two mixers that ran side by side on one input, still to be added up with fixed factors:
    ``scale_a * a + scale_b * b (+ bias)``; `bias` float32 [hidden] is a projection's, its mixer's factor included."""
    a: torch.Tensor
    scale_a: float
    b: torch.Tensor
    scale_b: float
    bias: Optional[torch.Tensor] = None


@dataclass
class NormedUpdate:
    """What a block with a norm behind each sublayer leaves pending: the stream is still to grow by
    ``delta / sqrt(mean(delta^2) + eps) * weight`` (`weight` float32 [hidden]: the norm's times the channel scale).
    `delta` is a tensor, `RoutedSum`, `ScaledPair` or `BiasedOutput`.  A norm that knows the form (`takes_normed`)
    works all of it out in its own pass over the stream; `apply` does it on its own."""
    delta: object
    weight: torch.Tensor
    eps: float

    def sources(self) -> Dict[str, object]:
        """`delta` as the arguments of `kernels.residual_norm`, with the norm it is to pass."""
        d = self.delta
        args: Dict[str, object] = {"inner_weight": self.weight, "inner_eps": self.eps}
        if isinstance(d, RoutedSum):
            if d.shared is None:
                args["routed"] = (d.y, d.plan.inv, d.wts, d.plan.top_k)
                return args
            d = d.materialize()
        if isinstance(d, ScaledPair):
            args.update(a=d.a, scale_a=d.scale_a, b=d.b, scale_b=d.scale_b, bias=d.bias)
        elif isinstance(d, BiasedOutput):
            args.update(a=d.y, bias=d.bias)
        else:
            args["a"] = d
        return args

    def apply(self, h: torch.Tensor) -> None:
        from .. import kernels
        kernels.residual_norm(h, None, 0.0, None, **self.sources())


def summed(delta):
    """`delta` as a tensor (None stays None; a `StreamCopy` means nothing is left to add)."""
    if isinstance(delta, PairSum):
        return (delta.a.to(torch.float32) + delta.b.to(torch.float32)).to(delta.a.dtype)
    if isinstance(delta, ScaledPair):
        y = delta.a.to(torch.float32) * delta.scale_a + delta.b.to(torch.float32) * delta.scale_b
        return (y if delta.bias is None else y + delta.bias).to(delta.a.dtype)
    if isinstance(delta, NormedUpdate):
        raise TypeError("an update that is still to be normed is applied to the stream, not read as a sum")
    if isinstance(delta, StreamCopy):
        return None
    if isinstance(delta, BiasedOutput):
        return delta.y + delta.bias.to(delta.y.dtype)
    if isinstance(delta, StreamUpdate):
        if delta.mix is not None or delta.out is not None:
            raise TypeError("an update of several residual streams cannot be read as one sum")
        return delta.y
    return delta.materialize() if isinstance(delta, RoutedSum) else delta


class Norm(Part):
    """Normalisation fused with the residual sum.

    The residual stream `h` is float32 in both modes; `delta` is the previous part's
    output in the engine dtype (or None).  A norm with `takes_unsummed` also accepts a
    `RoutedSum` as `delta`.
    """

    takes_unsummed = False
    takes_normed = False            # accepts a `NormedUpdate` as `delta`

    def add_norm(self, h: torch.Tensor, delta: Optional[torch.Tensor],
                 out_dtype: torch.dtype) -> torch.Tensor:
        """h += delta (in place, in 32-bit); return norm(h) in `out_dtype`."""
        raise NotImplementedError

    def add_norm_rows(self, h: torch.Tensor, delta: Optional[torch.Tensor], rows: torch.Tensor,
                      out_dtype: torch.dtype) -> torch.Tensor:
        """norm(h[rows] + delta[rows]) without changing h."""
        raise NotImplementedError


class PositionEncoding(Part):
    """How positions enter queries and keys."""

    def rotary_table(self, device: torch.device) -> Optional[Tuple[torch.Tensor, int]]:
        """(inverse frequencies float32 [rotary_dim // 2], rotary_dim) for the fused
        rotate-and-append kernel (half-split pairing), or None if the encoding is not of
        that form; then `apply` is called and the kernel appends without rotating."""
        return None

    def pair_table(self, device: torch.device) -> Optional[Tuple[torch.Tensor, int, bool]]:
        """(inverse frequencies float32 [rotary_dim // 2], rotary_dim, interleaved) for kernels that take
        either layout of pairs: (i, i + rotary_dim / 2), or (2i, 2i + 1) interleaved."""
        table = self.rotary_table(device)
        return None if table is None else (*table, False)

    # what multiplies cosine and sine of every angle (a kernel that rotates takes it with the table)
    magnitude = 1.0

    def apply(self, q: torch.Tensor, k: torch.Tensor, positions: torch.Tensor) -> None:
        """Encode in place: q [T, heads, D], k [T, kv_heads, D], positions int32 [T]."""
        raise NotImplementedError


class EmbeddingExtra(Part):
    """Something added to the token embedding before the first layer (a second table looked up by
    a hash of neighbouring tokens, for instance).  It may keep a small state per request."""

    def state_spec(self) -> Optional[StateSpec]:
        return None

    def add(self, h: torch.Tensor, ctx: StepContext, state: Optional[torch.Tensor]) -> None:
        """Add this part's rows to the float32 stream `h` [T, hidden] in place.  `state` is the
        slab [slots, *state_spec.shape] indexed by `ctx.seg_slot`, zero for a new request."""
        raise NotImplementedError

    def start(self, embedding: torch.Tensor, scale: float, h: torch.Tensor, ctx: StepContext,
              state: Optional[torch.Tensor]) -> None:
        """h = embedding[token] * scale, and this part's rows added: what the first extra is asked for, so that
        it may do both in one pass over the stream."""
        from .. import kernels
        kernels.embed_rows(embedding, ctx.token_ids, h, scale=scale)
        self.add(h, ctx, state)


class Mixer(Part):
    """Mixes information between the tokens of a request (attention here)."""

    def cache_spec(self) -> Optional[CacheSpec]:
        return None

    def state_spec(self) -> Optional[StateSpec]:
        return None

    def forward(self, x: torch.Tensor, ctx: StepContext, cache: Optional[CacheView],
                state: Optional[torch.Tensor]) -> torch.Tensor:
        """x [T, hidden] in the engine dtype -> [T, hidden] in the engine dtype.

        `cache` is the view of the slot this call reads (and appends to when
        `cache.append`); `state` is the slab [slots, *state_spec.shape] indexed by
        `ctx.seg_slot`.
        """
        raise NotImplementedError


class FeedForward(Part):
    def forward(self, x: torch.Tensor, ctx: StepContext):
        """x [T, hidden] -> [T, hidden], both in the engine dtype.  A routed feed-forward may
        return a `RoutedSum` instead of the tensor (see there); `summed()` turns either into
        the tensor."""
        raise NotImplementedError


class Block(Part):
    """Arrangement of norms, mixer and feed-forward around the residual stream.

    The model asks the block, not the mixer, what the layer keeps between steps: pages
    (`cache_spec`) and a slab of fixed-size state per request (`state_spec`).  The usual block
    passes its mixer's answers on; an arrangement whose feed-forward (or the block itself)
    keeps state answers for it and hands `state` to whichever part it belongs to.
    """

    mixer: Mixer

    def cache_spec(self) -> Optional[CacheSpec]:
        return self.mixer.cache_spec()

    def state_spec(self) -> Optional[StateSpec]:
        return self.mixer.state_spec()

    def settle(self, h: torch.Tensor, pending):
        """Add what this block's `forward` left pending to the stream now; returns what is then left
        (None, or the `StreamCopy` of an arrangement that leaves nothing).  For looking at the
        stream between layers; the step itself never calls it."""
        if isinstance(pending, StreamCopy):
            return pending
        if isinstance(pending, NormedUpdate):
            pending.apply(h)
            return None
        delta = summed(pending)
        if delta is not None:
            h.add_(delta.to(torch.float32))
        return None

    def forward(self, h: torch.Tensor, pending, ctx: StepContext,
                cache: Optional[CacheView], state: Optional[torch.Tensor]):
        """Advance the float32 residual stream `h` in place.

        `pending` is a contribution not yet added to `h` (so that the sum fuses with the
        next norm): a tensor, a `RoutedSum` or None; the return value is this block's own
        pending contribution.
        """
        raise NotImplementedError
