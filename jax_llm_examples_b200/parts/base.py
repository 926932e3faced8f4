"""Interfaces of the parts a decoder is put together from, and the step context they all see.

A part gets its sizes and constants as constructor arguments and never learns which model it
is in.  The kinds of part:

* :class:`Norm` — normalises rows of the residual stream.
* :class:`PositionEncoding` — turns projected q and k rows into position-aware ones and hands
  k and v to the cache.
* :class:`Mixer` — mixes information across a request's tokens (attention here); it says what it
  needs of the cache manager: pages of keys and values (:class:`KVNeed`) and/or per-request state
  of fixed size (:class:`StateNeed`).
* :class:`FeedForward` — acts on each token alone (dense, or routed experts).
* :class:`Block` — arranges the above (pre-norm residual block here).

All of them work on the *flattened* batch of a step: N token rows from R requests, described by
:class:`StepContext`.  The residual stream is float32 [N, D]; parts return a float32 ``delta`` that
the next norm adds to it (the sum is fused into the norm kernel).
"""

from __future__ import annotations

import dataclasses
from typing import Any, Callable

import torch

from ..cache.manager import Retention


@dataclasses.dataclass
class Runtime:
    """Where and in which precision a model runs."""

    dtype: torch.dtype  # activations and cache: torch.bfloat16, or torch.float32 for the true 32-bit path
    device: torch.device

    def __post_init__(self):
        if self.dtype not in (torch.float32, torch.bfloat16):
            raise ValueError(f"dtype must be float32 or bfloat16, not {self.dtype}")


@dataclasses.dataclass(frozen=True)
class KVNeed:
    """Pages of keys and values: heads, head size, and which keys stay readable.  ``planes``: 2 = a key and a value
    row per token and head; 1 = one row (a mixer that keeps a latent from which it makes both)."""

    num_kv_heads: int
    head_dim: int
    retention: Retention
    planes: int = 2


@dataclasses.dataclass(frozen=True)
class StateNeed:
    """Per-request state of fixed size (zeroed when a request is admitted)."""

    shape: tuple[int, ...]
    dtype: torch.dtype = torch.float32


@dataclasses.dataclass
class Rows:
    """Token rows that may still be split-K partials: ``data`` is [N, D], or float32 [splits, N, D] whose
    slices the consumer adds in ascending order (saving the launch that would add them).

    As a term of a :class:`RowSum` the rows may also lie elsewhere in ``data``: token r's row is ``base + r``, or,
    with ``index`` (int32 [N * k]), the sum of the k rows ``index[r * k + j]``, j ascending, each times
    ``weights[r, j]`` (float32 [N, k]) if there are weights, all of them times the number ``scale``."""

    data: torch.Tensor
    splits: int = 1
    index: torch.Tensor | None = None
    k: int = 1
    base: int = 0
    weights: torch.Tensor | None = None
    scale: float = 1.0


@dataclasses.dataclass
class RowSum:
    """A delta that is still a sum of terms, added in this order by a consumer that can (the RMSNorm kernel: it then
    does an expert layer's un-permute and sum, and no kernel runs for them alone).  ``materialize()`` makes the plain
    [N, D] float32 tensor for a consumer that cannot: :func:`as_rows` calls it."""

    terms: list[Rows]
    materialize: Callable[[], torch.Tensor]


@dataclasses.dataclass
class PostNormed:
    """A delta that is still to be normed before it is added: x += mult * weight * groupnorm(rows + bias), the
    closing norm of a block that norms a sublayer's output as well as its input.  A norm that can (``GroupRMSNorm``)
    does this in the same pass over the row as the residual sum and its own norm; ``materialize()`` makes the plain
    [N, D] float32 tensor for a consumer that cannot: :func:`as_rows` calls it."""

    rows: Rows
    weight: torch.Tensor  # float32 [D]
    eps: float
    groups: int
    mult: float
    bias: torch.Tensor | None = None  # float32 [D], added to the rows before the norm (a biased product's bias)

    def gather(self) -> dict:
        """The group-norm kernel's arguments for rows that lie in expert order (``Rows.index``)."""
        return dict(delta_index=self.rows.index, delta_k=self.rows.k, delta_weights=self.rows.weights)

    def materialize(self) -> torch.Tensor:
        from ..kernels import api as K

        n = self.rows.data.shape[-2] if self.rows.index is None else self.rows.index.numel() // self.rows.k
        d = self.rows.data.shape[-1]
        zero = torch.zeros((n, d), dtype=torch.float32, device=self.weight.device)
        K.group_norm(zero, self.rows.data, self.rows.splits, self.bias, self.weight, self.groups, self.mult, eps=self.eps,
                     **self.gather())
        return zero


@dataclasses.dataclass
class Scaled:
    """A delta that is still to be multiplied, channel by channel, by a vector before it is added: x += scale * rows
    (a "layer scale").  A norm that can (``GroupRMSNorm``) does it in the same pass over the row as the residual sum
    and its own norm; ``materialize()`` makes the plain [N, D] float32 tensor for a consumer that cannot."""

    rows: Rows
    scale: torch.Tensor  # float32 [D]

    def materialize(self) -> torch.Tensor:
        from ..kernels import api as K

        n, d = self.rows.data.shape[-2], self.rows.data.shape[-1]
        zero = torch.zeros((n, d), dtype=torch.float32, device=self.scale.device)
        K.group_norm(zero, self.rows.data, self.rows.splits, None, self.scale, 1, 1.0, post_norm=False)
        return zero


@dataclasses.dataclass
class StreamMixed:
    """A sublayer output that is still to be written into several residual streams: x_t <- sum_s mix[s, t] x_s +
    write[t] * rows, for all streams t at once.  Only a norm that knows the streams (``StreamRMSNorm``) can add it: it
    does so in the same pass as the next sublayer's read and norm."""

    rows: Rows
    mix: torch.Tensor  # float32 [S, S], indexed [from, to]
    write: torch.Tensor  # float32 [S]


def as_rows(x: "torch.Tensor | Rows | RowSum | PostNormed | Scaled | None") -> "Rows | None":
    if x is None or isinstance(x, Rows):
        return x
    if isinstance(x, StreamMixed):
        raise TypeError("a sublayer output pending for several residual streams can only be added by a norm that keeps the streams")
    if isinstance(x, (RowSum, PostNormed, Scaled)):
        return Rows(x.materialize(), 1)
    return Rows(x, 1)


class Workspace:
    """Named device buffers that live across steps (scratch of kernels, e.g. split-K partials).
    Kernels of one stream run in order, so a buffer can serve every layer in turn.  A buffer that was
    outgrown is kept, not freed: a captured CUDA graph may still hold its address."""

    def __init__(self, device: torch.device):
        self.device = device
        self._bufs: dict[str, torch.Tensor] = {}
        self._outgrown: list[torch.Tensor] = []
        self._side: torch.cuda.Stream | None = None

    def side_stream(self) -> torch.cuda.Stream:
        """A second stream for work that is independent of what the step's own stream does next (made on first use)."""
        if self._side is None:
            self._side = torch.cuda.Stream(device=self.device)
        return self._side

    def zeros(self, name: str, numel: int, dtype: torch.dtype) -> torch.Tensor:
        """A buffer that is zero when first handed out and is never handed out as scratch: for kernels that keep a
        small state across launches (a ticket counter that every launch leaves at zero)."""
        key = "zeros:" + name
        t = self._bufs.get(key)
        if t is None or t.numel() < numel or t.dtype != dtype:
            if t is not None:
                self._outgrown.append(t)
            t = torch.zeros(max(numel, 1), dtype=dtype, device=self.device)
            self._bufs[key] = t
        return t[:numel]

    def get(self, name: str, numel: int, dtype: torch.dtype) -> torch.Tensor:
        t = self._bufs.get(name)
        if t is None or t.numel() < numel or t.dtype != dtype:
            if t is not None:
                self._outgrown.append(t)
            t = torch.empty(max(numel, 1), dtype=dtype, device=self.device)
            self._bufs[name] = t
        return t[:numel]


@dataclasses.dataclass
class LayerCache:
    """What one run of a layer sees of the cache in this step."""

    pages: torch.Tensor | None  # [num_pages, 2, Hkv, page_size, dh]
    block_table: torch.Tensor | None  # int32 [R, width], rows in the order of the step's requests
    writes: bool  # False: the layer reads a cache that another layer fills
    state: torch.Tensor | None  # [max_slots, *StateNeed.shape]; the first slab of a mixer that has several
    states: tuple = ()  # all slabs of the run, in the order of the mixer's ``state_needs()``


@dataclasses.dataclass
class StepContext:
    """One step's batch: N tokens of R requests, portions of prompts beside single decoded tokens."""

    runtime: Runtime
    n_tokens: int
    n_requests: int
    token_ids: torch.Tensor  # int32 [N]
    positions: torch.Tensor  # int32 [N] absolute position in the request
    req_of_token: torch.Tensor  # int32 [N] index into this step's requests
    cu_q: torch.Tensor  # int32 [R + 1] token offsets of the requests
    q_start: torch.Tensor  # int32 [R] tokens the request held before this step
    kv_len: torch.Tensor  # int32 [R] tokens it holds after this step
    slot_ids: torch.Tensor  # int32 [R] cache-manager slot (indexes per-request state)
    logit_rows: torch.Tensor  # int32 [M] token rows whose logits are wanted
    n_logit_rows: int
    status: torch.Tensor  # int32 [1] error bits raised by kernels
    # host copies, for parts that plan on the host
    host_q_lens: list[int] = dataclasses.field(default_factory=list)
    host_q_start: list[int] = dataclasses.field(default_factory=list)
    host_slot_ids: list[int] = dataclasses.field(default_factory=list)
    max_q_len: int = 0
    max_kv_len: int = 0
    scratch: dict[str, Any] = dataclasses.field(default_factory=dict)  # per-step memo shared by parts
    workspace: Workspace | None = None  # buffers that outlive the step
    # What the model's step planners (see :meth:`Part.step_planners`) made of this step, by name: int32 arrays
    # on the host, and the same arrays on the device (they travel with the step's descriptor, in its one copy).
    host_arrays: dict[str, Any] = dataclasses.field(default_factory=dict)
    arrays: dict[str, torch.Tensor] = dataclasses.field(default_factory=dict)

    def plan_with(self, planners, page_size: int) -> None:
        """Runs step planners for a context made by hand (a test of one part): what the engine does while it
        packs a step, with one small copy per array instead of the descriptor's single one."""
        shape = StepShape(tuple(self.host_q_lens), tuple(self.host_q_start), page_size, self.max_kv_len)
        for planner in planners:
            for name, a in planner(shape).items():
                self.host_arrays[name] = a
                self.arrays[name] = torch.tensor(a.tolist(), dtype=torch.int32).reshape(-1).to(self.token_ids.device)


@dataclasses.dataclass(frozen=True)
class StepShape:
    """What a step planner sees of a step, on the host, before anything runs."""

    q_lens: tuple[int, ...]  # tokens each request brings
    q_start: tuple[int, ...]  # tokens each request held before
    page_size: int
    max_kv_len: int


StepPlanner = Callable[["StepShape"], "dict[str, Any]"]


class Part:
    """Base of all parts.

    ``kernel_libraries``: the kernel libraries (``csrc/<name>.cu``) this part launches in every precision;
    ``kernel_libraries_bf16``: those it launches only with bfloat16 activations (tensor-core kernels: the
    32-bit path never builds or loads them).  Libraries are built on first use.
    """

    kernel_libraries: tuple[str, ...] = ()
    kernel_libraries_bf16: tuple[str, ...] = ()
    # True: the part has work that needs only the step's tokens: ``begin_step(ctx)`` is called before the first block runs.
    begins_steps: bool = False
    # False: forward() reads the step's host copies (``ctx.host_*``) or otherwise does work that a captured
    # CUDA graph would freeze; a model with such a part is never replayed from a graph.
    capturable: bool = True

    def required_libraries(self, runtime: Runtime) -> tuple[str, ...]:
        """What this part launches in this precision."""
        if runtime.dtype == torch.bfloat16:
            return tuple(dict.fromkeys(self.kernel_libraries + self.kernel_libraries_bf16))
        return self.kernel_libraries

    def step_planners(self) -> "tuple[StepPlanner, ...]":
        """Functions ``planner(shape: StepShape) -> {name: int32 numpy array}`` that this part wants run once per
        step on the host (tile lists, row lists and the like).  The model collects the distinct planners of all
        its parts; the engine runs each once per step and sends the arrays to the device together with the step's
        descriptor: ``ctx.arrays[name]`` (device) and ``ctx.host_arrays[name]``.  A planner is a module-level
        function (parts of the same kind share it, so it runs once however many layers use it) and must return
        the same names with the same sizes for steps of the same shape when it wants to be replayed from a graph."""
        return ()

    def begin_step(self, ctx: "StepContext") -> None:
        """Work of a step that needs nothing but its description (token ids, positions), called once per step and part
        before the first block, if ``begins_steps``: a part may put it on the second stream, beside the first layers, and
        leave what it made in ``ctx.scratch``."""

    def sub_parts(self) -> "tuple[Part, ...]":
        """Parts inside this one (a block's norms, mixer and feed-forward; an attention's position encoding)."""
        return ()


def walk_parts(part: "Part"):
    yield part
    for p in part.sub_parts():
        yield from walk_parts(p)


@dataclasses.dataclass
class Dispatch:
    """What a routed feed-forward needs between the router and its experts' products: the step's (token, choice)
    pairs sorted by expert and the tokens' rows gathered (and scaled) in that order.  A feed-forward that can use
    them offers the buffers through ``router_request()``; a norm that routes for it may fill them in the same kernel
    and hands them back with the routing, which saves a decode step two dependent launches per layer."""

    counter: torch.Tensor | None  # int32 [1], zero between launches (None: the kernel that fills this keeps none)
    offsets: torch.Tensor  # int32 [groups + 1]
    sorted_pair: torch.Tensor  # int32 [pairs]
    sorted_pos: torch.Tensor  # int32 [pairs]
    tiles: "tuple[torch.Tensor, torch.Tensor] | None"  # (tile list, count) for the grouped streaming products
    a_sorted: torch.Tensor  # [pairs + extra_rows, D]
    extra_rows: int  # rows of a group appended after the experts (a shared expert that takes every token)
    tile_rows: int
    status: torch.Tensor


@dataclasses.dataclass
class CorrectedRouter:
    """A corrected, group-limited router (``K.router``'s forms of that kind) as a routed feed-forward describes it to whoever
    may route for it, with ``dispatch(ctx, n_rows)`` for the buffers of its sort and gather."""

    w_router: torch.Tensor  # float32 [E, D]
    bias: torch.Tensor | None
    correction: torch.Tensor | None
    weight_form: str
    groups: int
    keep: int
    group_top: int
    normalize: bool
    scale: float
    top_k: int
    dispatch: Callable[["StepContext", int], Dispatch]


@dataclasses.dataclass
class RowPlaces:
    """Where a feed-forward wants its input rows: row n at the rows ``index[n * copies + j]`` of [N * copies, D] (int32)."""

    index: torch.Tensor
    copies: int


class Norm(Part):
    fuses_router: bool = False  # True: forward(router=...) also routes the tokens in its kernel
    places_rows: bool = False  # True: forward(places=RowPlaces) writes its rounded rows where they are wanted

    def forward(self, ctx: StepContext, x: torch.Tensor, delta: "torch.Tensor | Rows | None", *, out_dtype: torch.dtype,
                want_f32: bool = False, row_index: torch.Tensor | None = None, router=None):
        """x += delta (if given); returns (normed rows in out_dtype, the same in float32 if asked,
        routing).  ``router`` = (w_router [E, D] float32, top_k) asks a norm with ``fuses_router`` to
        route as well: routing = (expert indices [N, k] int32, weights [N, k] float32); else None.  The request
        may have a third element, a function (ctx, n_rows) -> Dispatch or None; a norm that fills the Dispatch too
        returns it as the routing's third element."""
        raise NotImplementedError


class PositionEncoding(Part):
    accepts_partials: bool = False  # True: encode_and_store takes qkv as Rows with split-K partials

    def encode_and_store(self, ctx: StepContext, qkv: "torch.Tensor | Rows", n_heads: int, n_kv_heads: int, head_dim: int,
                         cache: LayerCache, qk_norm_eps: float | None) -> torch.Tensor:
        """qkv: [N, (Hq + 2 Hkv) * dh] projected rows.  Returns q [N, Hq, dh] ready for the score
        product; writes k and v into the cache pages when ``cache.writes``."""
        raise NotImplementedError

    def query_temperature(self) -> tuple[float, float]:
        """(attn_scale, floor_scale) of the position-dependent query scale; (0, 1) = none."""
        return (0.0, 1.0)


class Mixer(Part):
    needs_f32_input: bool = False  # True: forward() gets the normed rows unrounded (``h32=``) and no rounded ones

    def kv_need(self) -> KVNeed | None:
        return None

    def state_need(self) -> StateNeed | None:
        return None

    def state_needs(self) -> "tuple[StateNeed, ...]":
        """Every per-request state of the mixer (one slab each, ``cache.states`` in this order): a recurrence's
        state beside the last inputs of a short convolution, say.  The default is the single ``state_need()``."""
        one = self.state_need()
        return () if one is None else (one,)

    def forward(self, ctx: StepContext, h: torch.Tensor, cache: LayerCache) -> "torch.Tensor | Rows":
        """h: normed rows [N, D] in the runtime's dtype.  Returns delta [N, D] float32 (or Rows of partials)."""
        raise NotImplementedError


class ProjectedMixer(Mixer):
    """A mixer of the form  out = W_o core(W_in h):  one product into the rows ``core`` works on (float32 sums, possibly
    still split-K partials), one product out of the rows it leaves.  A combinator (``ParallelMixers``) can then stack
    the W_in of several such mixers that read the same h into one product, let each ``core`` fill its own column range
    of one buffer, and send that through the W_o laid side by side: the sum of the mixers' outputs is then made by the
    output product itself."""

    w_in: torch.Tensor  # [in_features, D]
    w_o: torch.Tensor  # [D, out_features]

    @property
    def in_features(self) -> int:
        return self.w_in.shape[0]

    @property
    def out_features(self) -> int:
        return self.w_o.shape[1]

    def core(self, ctx: StepContext, h: torch.Tensor, proj: Rows, col: int, cache: LayerCache, out: torch.Tensor, mult: float) -> None:
        """``proj``: float32 rows whose columns [col, col + in_features) are W_in h; ``h``: the mixer's input (for
        small products of its own); writes ``mult`` times the rows for W_o into ``out`` [N, out_features] (maybe a
        column range of wider rows)."""
        raise NotImplementedError

    def forward(self, ctx: StepContext, h: torch.Tensor, cache: LayerCache):
        from ..tracing import scope
        from .linear import linear

        with scope("qkv_matmul"):
            proj = as_rows(linear(ctx, h, self.w_in, torch.float32, partials=True))
        out = torch.empty((h.shape[0], self.out_features), dtype=ctx.runtime.dtype, device=h.device)
        self.core(ctx, h, proj, 0, cache, out, 1.0)
        with scope("projection"):
            return linear(ctx, out, self.w_o, torch.float32, partials=True)


class FeedForward(Part):
    needs_f32_input: bool = False  # True: forward() also gets the normed rows unrounded

    def router_request(self):
        """(w_router, top_k) if the preceding norm may route the tokens for this part, else None; optionally a third
        element, see Norm.forward."""
        return None

    def row_places(self, ctx: StepContext, n: int) -> "RowPlaces | None":
        """Where this part wants the preceding norm to write its n rows, if it knows that before it sees them and the
        norm can (``Norm.places_rows``); forward() then gets rows in that order, no ``h32``, and the places as ``routing``."""
        return None

    def corrected_router(self) -> "CorrectedRouter | None":
        """The part's router, if it is of the corrected kind and a block may route for it in the kernel that closes the
        sublayer before (``PostNormBlock`` does in decode steps)."""
        return None

    def forward(self, ctx: StepContext, h: torch.Tensor, h32: torch.Tensor | None, routing=None) -> "torch.Tensor | Rows":
        """Returns delta [N, D] float32 (or Rows of partials).  ``routing``: what a fusing norm already chose."""
        raise NotImplementedError


class Block(Part):
    mixer: "Mixer | None"  # None: a block that mixes nothing across tokens and keeps no cache or state

    def forward(self, ctx: StepContext, x: torch.Tensor, delta: "torch.Tensor | Rows | None", cache: LayerCache):
        """Runs the block on residual x with a pending ``delta`` not yet added; returns the new pending delta."""
        raise NotImplementedError


# ------------------------------------------------------------------------------ part registry
_PARTS: dict[tuple[str, str], Callable[..., Part]] = {}
KINDS = ("norm", "position", "mixer", "feed_forward", "block", "conv")


def register_part(kind: str, name: str, factory: Callable[..., Part]) -> None:
    """Makes a part available to model builders under (kind, name)."""
    if kind not in KINDS:
        raise ValueError(f"unknown kind of part {kind!r}; kinds: {KINDS}")
    _PARTS[(kind, name)] = factory


def make_part(kind: str, name: str, **kwargs: Any) -> Part:
    try:
        factory = _PARTS[(kind, name)]
    except KeyError:
        known = sorted(n for k, n in _PARTS if k == kind)
        raise KeyError(f"no {kind} part named {name!r}; known: {known}") from None
    return factory(**kwargs)


def known_parts(kind: str) -> list[str]:
    return sorted(n for k, n in _PARTS if k == kind)
