"""Feed-forward parts: dense SwiGLU and routed experts with a shared expert."""

from __future__ import annotations

import torch

from ..kernels import api as K
from ..tracing import active as tracing_active
from ..tracing import scope
from .base import CorrectedRouter, Dispatch, FeedForward, RowPlaces, Rows, RowSum, StepContext, as_rows, register_part
from .linear import (STREAM_MAX_ROWS, group_rows_hint, grouped_act_linear, grouped_linear, grouped_swiglu_linear, grouped_swiglu_streams,
                     interleave_gate_up, linear,
                     swiglu_linear)


def _can_interleave(w_gate_up: torch.Tensor) -> bool:
    return w_gate_up.dtype == torch.bfloat16 and (w_gate_up.shape[-2] // 2) % 16 == 0 and w_gate_up.shape[-1] % 8 == 0


class DenseSwiGLU(FeedForward):
    """down(silu(h gate) * (h up)) (llama4/llama4_jax/model.py:1142-1153).
    ``w_gate_up``: [2F, D], gate rows then up rows; ``w_down``: [D, F].  bfloat16 weights are re-laid in
    blocks of [16 gate rows, 16 up rows] so that the product's epilogue can apply the activation."""

    kernel_libraries = ("elementwise", "gemm_simt")
    kernel_libraries_bf16 = ("gemm_stream",)

    def __init__(self, w_gate_up: torch.Tensor, w_down: torch.Tensor, glu=K.SILU_GLU):
        """``glu``: another form of the gated activation, ``K.glu_form(alpha, limit, shift)``:
        g sigmoid(alpha g) (u + shift) with g = min(gate, limit) and u = clamp(up, -limit, limit)."""
        if w_gate_up.shape[0] != 2 * w_down.shape[1] or w_gate_up.shape[1] != w_down.shape[0]:
            raise ValueError(f"SwiGLU weights do not fit: gate_up {tuple(w_gate_up.shape)}, down {tuple(w_down.shape)}")
        self.interleaved = _can_interleave(w_gate_up)
        self.w_gate_up = interleave_gate_up(w_gate_up) if self.interleaved else w_gate_up
        self.w_down = w_down
        self.glu = tuple(glu)

    glu = K.SILU_GLU

    def forward(self, ctx: StepContext, h, h32=None, routing=None):
        with scope("gate_up_proj"):  # the reference's "gate" and "up_proj" (model.py:1145-1149) as one product
            act = swiglu_linear(ctx, h, self.w_gate_up, self.interleaved, ctx.runtime.dtype, self.glu)
        with scope("down_proj"):
            return linear(ctx, act, self.w_down, torch.float32, partials=True)


class RoutedExperts(FeedForward):
    """Sigmoid-routed top-k experts plus an optional shared expert (model.py:958-972, 999-1139).

    scores = h W_router in float32 from the unrounded normed rows; top-k of the raw scores (lower
    index wins ties); weight = sigmoid(score); each chosen expert runs SwiGLU on weight * h (the
    INPUT is scaled, model.py:1071); expert outputs are summed per token in choice order and the
    shared expert's output on the unscaled h is added (model.py:1111, 1137-1139).
    ``w_router``: [E, D]; ``we_gate_up``: [E, 2F, D] (gate rows then up rows); ``we_down``: [E, D, F]."""

    kernel_libraries = ("moe", "elementwise", "gemm_simt")
    kernel_libraries_bf16 = ("gemm_stream",)
    needs_f32_input = True
    OVERLAP_MIN_ROWS = 512  # from this many rows on (prompt portions), the shared expert runs on a second stream beside the routed ones
    FORK_MIN_ROWS = 2  # and in steps of few rows (decoding) from this many on; below, it rides as a group of the routed products

    def __init__(self, w_router: torch.Tensor, we_gate_up: torch.Tensor, we_down: torch.Tensor, top_k: int,
                 shared: DenseSwiGLU | None = None):
        E = w_router.shape[0]
        if we_gate_up.shape[0] != E or we_down.shape[0] != E or we_gate_up.shape[1] != 2 * we_down.shape[2] \
                or we_gate_up.shape[2] != we_down.shape[1] or w_router.shape[1] != we_down.shape[1]:
            raise ValueError(f"expert weights do not fit: router {tuple(w_router.shape)}, gate_up "
                             f"{tuple(we_gate_up.shape)}, down {tuple(we_down.shape)}")
        if not 1 <= top_k <= E:
            raise ValueError(f"top-{top_k} of {E} experts")
        self.w_router = w_router.to(torch.float32).contiguous()
        self.interleaved = _can_interleave(we_gate_up)
        self.we_gate_up = interleave_gate_up(we_gate_up) if self.interleaved else we_gate_up
        self.we_down, self.top_k, self.shared = we_down, top_k, shared
        self.num_experts = E
        # A shared expert of the experts' own shape rides along as group E of the grouped products when a step
        # has few rows (decoding): two launches fewer, and its weights stream at the grouped kernel's rate.
        # Its weights then live at the end of the experts' tensors; the shared part keeps views of them.
        self.merged = (shared is not None and shared.interleaved == self.interleaved
                       and shared.w_gate_up.shape == self.we_gate_up.shape[1:] and shared.w_down.shape == we_down.shape[1:]
                       and shared.w_gate_up.dtype == self.we_gate_up.dtype == torch.bfloat16 and shared.w_down.dtype == we_down.dtype)
        if self.merged:
            self.we_gate_up = torch.cat([self.we_gate_up, shared.w_gate_up[None]])
            self.we_down = torch.cat([self.we_down, shared.w_down[None]])
            shared.w_gate_up, shared.w_down = self.we_gate_up[E], self.we_down[E]

    def sub_parts(self):
        return () if self.shared is None else (self.shared,)

    def router_request(self):
        return (self.w_router, self.top_k, self.offer_dispatch)

    def placement(self, ctx: StepContext, n: int) -> tuple[bool, bool]:
        """Where the shared expert runs in a step of n rows: (on a second stream beside the routed experts, as one more
        group of the routed experts' products).  One row: as a group (two launches fewer; with so few blocks one
        kernel streams better than two).  More rows: on a second stream, beside the routed products: its weights stream
        while the routed products' few blocks leave memory bandwidth unused, or their short predecessors leave it idle
        (decode at batch 2: +7.5 %, batch 8: +3.7 %, batch 64: +6.5 %; batch 1 would lose 2 %).  Prompt portions: the routed experts stream their weights once for
        about a hundred rows each (bound by HBM), the shared expert's products are dense (bound by the tensor cores);
        side by side, the tails and the small kernels of either hide behind the other.  Between STREAM_MAX_ROWS and
        OVERLAP_MIN_ROWS: one after the other."""
        beside = self.shared is not None and ctx.workspace is not None and (
            self.FORK_MIN_ROWS <= n <= STREAM_MAX_ROWS or n >= self.OVERLAP_MIN_ROWS)
        return beside, self.merged and n <= STREAM_MAX_ROWS and not beside

    def sort_buffers(self, ctx: StepContext, n: int, extra_rows: int):
        """(offsets, sorted_pair, sorted_pos, tiles, tile_rows) for a step of n rows, not yet filled."""
        k, dev = self.top_k, self.w_router.device
        offsets = torch.empty(self.num_experts + 2, dtype=torch.int32, device=dev)
        sorted_pair = torch.empty(n * k, dtype=torch.int32, device=dev)
        sorted_pos = torch.empty(n * k, dtype=torch.int32, device=dev)
        tiles, tile_rows = None, 0
        if self.we_gate_up.dtype == torch.bfloat16 and ctx.runtime.dtype == torch.bfloat16:
            # the grouped products will run on the streaming kernel: their row tiles are listed once, by the sort
            rows, groups = n * k + extra_rows, self.num_experts + (extra_rows > 0)
            tile_rows = K.gemm_stream_token_tile(group_rows_hint(rows, groups, extra_rows))
            tiles = (torch.empty(2 * (-(-rows // tile_rows) + groups), dtype=torch.int32, device=dev),
                     torch.empty(1, dtype=torch.int32, device=dev))
        return offsets, sorted_pair, sorted_pos, tiles, tile_rows

    def offer_dispatch(self, ctx: StepContext, n: int) -> Dispatch | None:
        """The buffers that a norm which routes for this part may fill as well (see Dispatch)."""
        if ctx.workspace is None:
            return None
        extra = n if self.placement(ctx, n)[1] else 0
        offsets, sorted_pair, sorted_pos, tiles, tile_rows = self.sort_buffers(ctx, n, extra)
        a_sorted = torch.empty((n * self.top_k + extra, self.w_router.shape[1]), dtype=ctx.runtime.dtype, device=self.w_router.device)
        return Dispatch(ctx.workspace.zeros("dispatch_counter", 1, torch.int32), offsets, sorted_pair, sorted_pos, tiles, a_sorted,
                        extra, tile_rows, ctx.status)

    def route(self, ctx: StepContext, h32: torch.Tensor):
        """The router as a kernel of its own (when the norm before this part does not route)."""
        n, k, dev = h32.shape[0], self.top_k, h32.device
        topk_idx = torch.empty((n, k), dtype=torch.int32, device=dev)
        topk_w = torch.empty((n, k), dtype=torch.float32, device=dev)
        K.router(h32, self.w_router, topk_idx, topk_w)
        return topk_idx, topk_w

    def sort(self, ctx: StepContext, topk_idx: torch.Tensor, extra_rows: int = 0):
        offsets, sorted_pair, sorted_pos, tiles, tile_rows = self.sort_buffers(ctx, topk_idx.shape[0], extra_rows)
        if tiles is not None:
            K.expert_sort(topk_idx, offsets, sorted_pair, sorted_pos, self.num_experts, ctx.status, extra_rows, tile_rows, *tiles)
        else:
            K.expert_sort(topk_idx, offsets, sorted_pair, sorted_pos, self.num_experts, ctx.status, extra_rows)
        return offsets, sorted_pair, sorted_pos, tiles

    def forward(self, ctx: StepContext, h, h32, routing=None):
        rt = ctx.runtime
        n, D = h32.shape
        k, E = self.top_k, self.num_experts
        topk_idx, topk_w, *dispatched = routing if routing is not None else self.route(ctx, h32)
        done = dispatched[0] if dispatched else None  # sorted and gathered already, by the norm that routed
        if "record_routing" in ctx.scratch:  # tests compare the choices with a plain router's
            ctx.scratch["record_routing"].append(topk_idx)
        beside, merged = self.placement(ctx, n)
        extra = n if merged else 0
        shared, side = None, None
        if beside:
            main, side = torch.cuda.current_stream(), ctx.workspace.side_stream()
            side.wait_stream(main)
            with torch.cuda.stream(side), scope("moe_shared_expert"):
                shared = as_rows(self.shared.forward(ctx, h, None))
            shared.data.record_stream(main)  # made on the side stream, read (and freed) on the step's own
        with scope("moe_routed_expert"):  # the reference's names (model.py:1076-1138)
            if done is not None:
                if done.extra_rows != extra:
                    raise RuntimeError("the rows gathered with the routing do not fit this step's placement of the shared expert")
                offsets, sorted_pos, tiles, a_sorted = done.offsets, done.sorted_pos, done.tiles, done.a_sorted
            else:
                with scope("permute"):
                    offsets, sorted_pair, sorted_pos, tiles = self.sort(ctx, topk_idx, extra)
                    a_sorted = torch.empty((n * k + extra, D), dtype=rt.dtype, device=h.device)
                    K.permute_scale(h32, sorted_pair, topk_w, a_sorted, k, extra)
            groups = E + 1 if merged else E
            with scope("we_gate_up"):
                one_product = grouped_swiglu_streams(a_sorted, self.we_gate_up[:groups], self.interleaved)
                act = grouped_swiglu_linear(ctx, a_sorted, self.we_gate_up[:groups], offsets, self.interleaved, rt.dtype, extra, tiles)
            with scope("we_down"):  # (a timer's events between the two launches would come between them on the stream)
                y = grouped_linear(ctx, act, self.we_down[:groups], offsets, torch.float32, partials=True, largest_group=extra,
                                   tiles=tiles, after_grouped=one_product and not tracing_active())
        if side is not None:
            torch.cuda.current_stream().wait_stream(side)
        elif self.shared is not None and not merged:
            with scope("moe_shared_expert"):
                shared = as_rows(self.shared.forward(ctx, h, None))
        def combine() -> torch.Tensor:
            delta = torch.empty((n, D), dtype=torch.float32, device=h.device)
            with scope("unpermute"):  # with the reference's "expert_summing" in the same kernel
                K.moe_combine(y.data, None if shared is None else shared.data, sorted_pos, delta, k,
                              1 if shared is None else shared.splits, y.splits, n * k if merged else -1)
            return delta

        # The un-permute and the sum over a token's experts are left to the consumer (the next norm adds the rows
        # where it adds the residual); the order is the combine kernel's: shared expert, then the experts by choice.
        if y.data.dtype != torch.float32 or (shared is not None and shared.data.dtype != torch.float32):
            return combine()
        terms = [shared] if shared is not None else []
        if merged:
            terms.append(Rows(y.data, y.splits, None, 1, n * k))
        terms.append(Rows(y.data, y.splits, sorted_pos, k, 0))
        return RowSum(terms, combine)


register_part("feed_forward", "dense_swiglu", DenseSwiGLU)
register_part("feed_forward", "routed_experts", RoutedExperts)


class DenseBiasedMLP(FeedForward):
    """down(act(h up + b_up)) + b_down with a pointwise activation (``relu2``: the square of relu; ``silu``;
    ``gelu_tanh``; ``none``).  ``w_up``: [F, D]; ``w_down``: [D, F].  The first bias and the activation run in one
    kernel on the product's (partial) sums.  The last bias is not added here: ``bias_out`` offers it to whoever adds
    this part's output to the residual stream (a block whose closing norm takes it into its own kernel); a block
    that knows nothing of it must add it itself."""

    kernel_libraries = ("group_norm", "gemm_simt")
    kernel_libraries_bf16 = ("gemm_stream",)

    def __init__(self, w_up: torch.Tensor, b_up: torch.Tensor | None, w_down: torch.Tensor, b_down: torch.Tensor | None,
                 activation: str = "relu2"):
        if w_up.shape[0] != w_down.shape[1] or w_up.shape[1] != w_down.shape[0]:
            raise ValueError(f"MLP weights do not fit: up {tuple(w_up.shape)}, down {tuple(w_down.shape)}")
        if activation not in K.ACTIVATIONS:
            raise ValueError(f"unknown activation {activation!r}; known: {sorted(K.ACTIVATIONS)}")
        self.w_up, self.w_down, self.activation = w_up, w_down, activation
        self.b_up = None if b_up is None else b_up.to(torch.float32).contiguous()
        self.bias_out = None if b_down is None else b_down.to(torch.float32).contiguous()

    def forward(self, ctx: StepContext, h, h32=None, routing=None):
        with scope("gate_up_proj"):
            up = as_rows(linear(ctx, h, self.w_up, torch.float32, partials=True))
            act = torch.empty((h.shape[0], self.w_up.shape[0]), dtype=ctx.runtime.dtype, device=h.device)
            K.bias_act(up.data, act, self.b_up, None, self.activation, up.splits)
        with scope("down_proj"):
            return linear(ctx, act, self.w_down, torch.float32, partials=True)


register_part("feed_forward", "dense_biased", DenseBiasedMLP)


class RoutedMLPExperts(FeedForward):
    """Experts of the form down(act(up h)), their OUTPUTS weighted:

        out = sum_j weight_j * expert_j(h)  (+ shared(h): an expert of the same form that takes every token),

    chosen by a router of one of two families (``weight_form``), z = W_router h (+ bias) in float32:

    * "softmax_of_chosen": the top-k experts by z; weights = softmax over the chosen z only;
    * "sigmoid_corrected": s = sigmoid(z); the choice is made on s + ``correction``, among the ``keep`` best of ``groups``
      equal groups of neighbouring experts (a group's score is the sum of its ``group_top`` largest choice scores); weights
      = the chosen s (``normalize``: divided by their sum), times ``route_scale``.

    ``w_router``: [E, D]; ``router_bias``, ``correction``: [E] or None; ``we_up``: [E, F, D]; ``we_down``: [E, D, F];
    ``activation``: a name of ``K.ACTIVATIONS``.  The tokens' rows are gathered in expert order (unscaled), both products
    run as grouped products over that order.  The result is a :class:`RowSum` of one term, the rows in expert order with
    their weights, for a consumer that gathers them in its own kernel; else one kernel brings them back, weights them and
    adds the shared expert."""

    kernel_libraries = ("moe", "group_norm", "gemm_simt")
    kernel_libraries_bf16 = ("gemm_stream",)
    needs_f32_input = True
    MANY_ROWS = 64  # above this many rows (bfloat16) a corrected router shares each of its rows among eight tokens

    def __init__(self, w_router: torch.Tensor, router_bias: torch.Tensor | None, we_up: torch.Tensor, we_down: torch.Tensor,
                 top_k: int, activation: str = "relu2", shared: "DenseBiasedMLP | None" = None, weight_form: str = "softmax_of_chosen",
                 correction: torch.Tensor | None = None, groups: int = 1, keep: int = 1, group_top: int = 1, normalize: bool = False,
                 route_scale: float = 1.0):
        E = w_router.shape[0]
        if we_up.shape[0] != E or we_down.shape[0] != E or we_up.shape[1] != we_down.shape[2] or we_up.shape[2] != we_down.shape[1] \
                or w_router.shape[1] != we_down.shape[1] or any(t is not None and t.numel() != E for t in (router_bias, correction)):
            raise ValueError(f"expert weights do not fit: router {tuple(w_router.shape)}, up {tuple(we_up.shape)}, down {tuple(we_down.shape)}")
        if weight_form not in ("softmax_of_chosen", "sigmoid_corrected"):
            raise ValueError(f"unknown weight form {weight_form!r}")
        if weight_form == "softmax_of_chosen" and (correction is not None or groups != 1):
            raise ValueError("a softmax over the chosen scores has neither a correction nor groups")
        if groups < 1 or E % groups or not 1 <= keep <= groups or groups > K.ROUTER_MAX_GROUPS or group_top not in (1, 2):
            raise ValueError(f"{groups} groups (keep {keep}, {group_top} scores each) do not divide {E} experts evenly")
        if not 1 <= top_k <= E // groups * keep:
            raise ValueError(f"top-{top_k} of {E // groups * keep} experts")
        if activation not in K.ACTIVATIONS:
            raise ValueError(f"unknown activation {activation!r}; known: {sorted(K.ACTIVATIONS)}")
        self.w_router = w_router.to(torch.float32).contiguous()
        self.router_bias = None if router_bias is None else router_bias.to(torch.float32).contiguous()
        self.correction = None if correction is None else correction.to(torch.float32).contiguous()
        self.we_up, self.we_down = we_up.contiguous(), we_down.contiguous()
        self.top_k, self.num_experts, self.activation, self.shared = top_k, E, activation, shared
        self.weight_form, self.groups, self.keep, self.group_top = weight_form, int(groups), int(keep), int(group_top)
        self.normalize, self.route_scale = bool(normalize), float(route_scale)

    def sub_parts(self):
        return () if self.shared is None else (self.shared,)

    def corrected_router(self) -> CorrectedRouter | None:
        if self.weight_form != "sigmoid_corrected":
            return None
        return CorrectedRouter(self.w_router, self.router_bias, self.correction, self.weight_form, self.groups, self.keep, self.group_top,
                               self.normalize, self.route_scale, self.top_k, self.sort_buffers)

    def sort_buffers(self, ctx: StepContext, n: int) -> Dispatch:
        """The buffers of a step's sort and gather, not yet filled."""
        k, E, dev = self.top_k, self.num_experts, self.w_router.device
        i32 = lambda size: torch.empty(size, dtype=torch.int32, device=dev)  # noqa: E731
        tiles, tile_rows = None, 0
        if self.we_up.dtype == torch.bfloat16 and ctx.runtime.dtype == torch.bfloat16:
            tile_rows = K.gemm_stream_token_tile(group_rows_hint(n * k, E))
            tiles = (i32(2 * (-(-n * k // tile_rows) + E)), i32(1))
        a_sorted = torch.empty((n * k, self.w_router.shape[1]), dtype=ctx.runtime.dtype, device=dev)
        return Dispatch(None, i32(E + 1), i32(n * k), i32(n * k), tiles, a_sorted, 0, tile_rows, ctx.status)

    def route(self, ctx: StepContext, h32: torch.Tensor):
        n, k, dev = h32.shape[0], self.top_k, h32.device
        topk_idx = torch.empty((n, k), dtype=torch.int32, device=dev)
        topk_w = torch.empty((n, k), dtype=torch.float32, device=dev)
        if self.weight_form == "softmax_of_chosen":
            K.router(h32, self.w_router, topk_idx, topk_w, bias=self.router_bias, weight_form=self.weight_form)
        else:
            K.router(h32, self.w_router, topk_idx, topk_w, many_rows=ctx.runtime.dtype == torch.bfloat16 and n > self.MANY_ROWS,
                     bias=self.router_bias, weight_form=self.weight_form, correction=self.correction, groups=self.groups,
                     keep=self.keep, scale=self.route_scale, group_top=self.group_top, normalize=self.normalize)
        return topk_idx, topk_w

    def forward(self, ctx: StepContext, h, h32, routing=None):
        rt = ctx.runtime
        n, D = h32.shape
        k, E, dev = self.top_k, self.num_experts, h32.device
        # the block may have routed, sorted and gathered already (CorrectedRouter)
        topk_idx, topk_w, *dispatched = routing if routing is not None else self.route(ctx, h32)
        if "record_routing" in ctx.scratch:
            ctx.scratch["record_routing"].append(topk_idx)
        with scope("moe_routed_expert"):
            done = dispatched[0] if dispatched else self.sort_buffers(ctx, n)
            offsets, sorted_pos, tiles, a_sorted = done.offsets, done.sorted_pos, done.tiles, done.a_sorted
            if not dispatched:
                with scope("permute"):
                    K.expert_sort(topk_idx, offsets, done.sorted_pair, sorted_pos, E, ctx.status, 0,
                                  *((done.tile_rows, *tiles) if tiles is not None else ()))
                    K.permute_scale(h32, done.sorted_pair, None, a_sorted, k)
            with scope("we_gate_up"):
                act, one_product = grouped_act_linear(ctx, a_sorted, self.we_up, offsets, self.activation, rt.dtype, tiles)
            with scope("we_down"):
                y = as_rows(grouped_linear(ctx, act, self.we_down, offsets, torch.float32, partials=True, tiles=tiles,
                                           after_grouped=one_product and not tracing_active()))
        shared = None
        if self.shared is not None:
            with scope("moe_shared_expert"):
                shared = as_rows(self.shared.forward(ctx, h, None))

        def combine() -> torch.Tensor:
            delta = torch.empty((n, D), dtype=torch.float32, device=dev)
            with scope("unpermute"):
                K.moe_combine(y.data, None if shared is None else shared.data, sorted_pos, delta, k,
                              1 if shared is None else shared.splits, y.splits, -1, pair_weights=topk_w)
            return delta

        if shared is not None:
            return combine()
        return RowSum([Rows(y.data, y.splits, sorted_pos, k, 0, topk_w)], combine)


class SoftmaxRoutedMLPExperts(RoutedMLPExperts):
    """The form with a biased router and a softmax over the chosen logits (see :class:`RoutedMLPExperts`)."""


register_part("feed_forward", "softmax_routed_mlp", SoftmaxRoutedMLPExperts)
register_part("feed_forward", "routed_mlp", RoutedMLPExperts)


class GroupLimitedGLUExperts(FeedForward):
    """Gated experts chosen by a softmax router whose choice is corrected and limited to groups, their OUTPUTS weighted:

        s = softmax(W_router h) over ALL router outputs (float32);  the choice is made on s + correction, among the
        ``keep`` best of ``groups`` equal groups of neighbouring outputs (a group's score is its largest choice score);
        weights = the chosen s / (their sum + 1e-20) * ``route_scale``;
        out = sum_j weight_j * expert_j(h)  (+ shared(h): an expert that takes every token).

    The last ``identity`` router outputs are experts without weights whose output is their input.  An expert is
    down(act(gate h, up h)) with the gated activation ``glu`` (``K.glu_form``).  ``w_router``: [E + identity, D];
    ``correction``: [E + identity] or None; ``we_gate_up``: [E, 2F, D] (gate rows then up rows); ``we_down``: [E, D, F].
    The tokens' rows are gathered in expert order (unscaled; the identity experts' pairs sort behind the real ones and
    no product sees them), both products run as grouped products, and the kernel that brings the rows back applies
    the weights, puts the token's own row in an identity expert's place and adds the shared expert."""

    kernel_libraries = ("moe", "elementwise", "gemm_simt")
    kernel_libraries_bf16 = ("gemm_stream",)
    needs_f32_input = True
    MANY_ROWS = 64  # above this many rows (bfloat16) the router shares each of its rows among eight tokens

    def __init__(self, w_router: torch.Tensor, correction: torch.Tensor | None, we_gate_up: torch.Tensor, we_down: torch.Tensor,
                 top_k: int, identity: int = 0, groups: int = 1, keep: int = 1, route_scale: float = 1.0, glu=K.SILU_GLU,
                 shared: "DenseSwiGLU | None" = None):
        E = we_gate_up.shape[0]
        total = E + identity
        if w_router.shape[0] != total or we_down.shape[0] != E or we_gate_up.shape[1] != 2 * we_down.shape[2] \
                or we_gate_up.shape[2] != we_down.shape[1] or w_router.shape[1] != we_down.shape[1] \
                or (correction is not None and correction.numel() != total):
            raise ValueError(f"expert weights do not fit: router {tuple(w_router.shape)} for {E} experts + {identity} that hand their "
                             f"input on, gate_up {tuple(we_gate_up.shape)}, down {tuple(we_down.shape)}")
        if not 1 <= top_k <= total:
            raise ValueError(f"top-{top_k} of {total} router outputs")
        if groups < 1 or total % groups or not 1 <= keep <= groups or groups > K.ROUTER_MAX_GROUPS:
            raise ValueError(f"{groups} groups (keep {keep}) do not divide {total} router outputs evenly")
        self.w_router = w_router.to(torch.float32).contiguous()
        self.correction = None if correction is None else correction.to(torch.float32).contiguous()
        self.interleaved = _can_interleave(we_gate_up)
        self.we_gate_up = interleave_gate_up(we_gate_up) if self.interleaved else we_gate_up.contiguous()
        self.we_down = we_down.contiguous()
        self.top_k, self.num_experts, self.identity, self.total = top_k, E, int(identity), total
        self.groups, self.keep, self.route_scale, self.glu, self.shared = int(groups), int(keep), float(route_scale), tuple(glu), shared

    def sub_parts(self):
        return () if self.shared is None else (self.shared,)

    def forward(self, ctx: StepContext, h, h32, routing=None):
        rt = ctx.runtime
        n, D = h32.shape
        k, E, T, dev = self.top_k, self.num_experts, self.total, h32.device
        topk_idx = torch.empty((n, k), dtype=torch.int32, device=dev)
        topk_w = torch.empty((n, k), dtype=torch.float32, device=dev)
        K.router(h32, self.w_router, topk_idx, topk_w, many_rows=rt.dtype == torch.bfloat16 and n > self.MANY_ROWS,
                 weight_form="softmax_normalized", correction=self.correction, groups=self.groups, keep=self.keep,
                 scale=self.route_scale)
        if "record_routing" in ctx.scratch:
            ctx.scratch["record_routing"].append(topk_idx)
        with scope("moe_routed_expert"):
            with scope("permute"):
                offsets = torch.empty(T + 1, dtype=torch.int32, device=dev)
                sorted_pair = torch.empty(n * k, dtype=torch.int32, device=dev)
                sorted_pos = torch.empty(n * k, dtype=torch.int32, device=dev)
                tiles = None
                if self.we_gate_up.dtype == torch.bfloat16 and rt.dtype == torch.bfloat16:
                    tile_rows = K.gemm_stream_token_tile(group_rows_hint(n * k, E))
                    tiles = (torch.empty(2 * (-(-n * k // tile_rows) + T), dtype=torch.int32, device=dev),
                             torch.empty(1, dtype=torch.int32, device=dev))
                    K.expert_sort(topk_idx, offsets, sorted_pair, sorted_pos, T, ctx.status, 0, tile_rows, *tiles, tile_groups=E)
                else:
                    K.expert_sort(topk_idx, offsets, sorted_pair, sorted_pos, T, ctx.status)
                a_sorted = torch.empty((n * k, D), dtype=rt.dtype, device=dev)
                K.permute_scale(h32, sorted_pair, None, a_sorted, k)
            # the grouped products see the first E groups only: offsets[0..E]
            with scope("we_gate_up"):
                one_product = grouped_swiglu_streams(a_sorted, self.we_gate_up, self.interleaved)
                act = grouped_swiglu_linear(ctx, a_sorted, self.we_gate_up, offsets, self.interleaved, rt.dtype, 0, tiles, self.glu)
            with scope("we_down"):
                y = as_rows(grouped_linear(ctx, act, self.we_down, offsets, torch.float32, partials=True, tiles=tiles,
                                           after_grouped=one_product and not tracing_active()))
        shared = None
        if self.shared is not None:
            with scope("moe_shared_expert"):
                shared = as_rows(self.shared.forward(ctx, h, None))
        delta = torch.empty((n, D), dtype=torch.float32, device=dev)
        with scope("unpermute"):
            ident = self.identity > 0
            K.moe_combine(y.data, None if shared is None else shared.data, sorted_pos, delta, k,
                          1 if shared is None else shared.splits, y.splits, -1, pair_weights=topk_w,
                          topk_idx=topk_idx if ident else None, n_real=E, h_rows=h32 if ident else None)
        return delta


register_part("feed_forward", "group_limited_glu_experts", GroupLimitedGLUExperts)


class TableRoutedGLUExperts(FeedForward):
    """Gated experts without a router: a table gives every token id its experts, whose outputs count alike,

        out = (1 / k) * sum_j expert_(table[token, j])(h).

    ``table``: int32 [vocab, k], the entries of a row differ; ``we_gate_up``: [E, 2F, D] (gate rows then up rows); ``we_down``:
    [E, D, F]; ``glu``: the gated activation (``K.glu_form``).

    Which rows go where depends on the step's token ids alone.  The sort of the (token, expert) pairs therefore runs ahead of
    the layers, on the second stream beside whatever comes first (``begin_step``), once per step however many layer runs
    share this part; and the norm in front of it writes its rows straight to their places in expert order
    (``row_places``), so that neither a router, nor a sort, nor a gather stands between the norm and the experts' products.
    The result is a :class:`RowSum` of one scaled term, the rows still in expert order."""

    kernel_libraries = ("moe", "elementwise", "gemm_simt")
    kernel_libraries_bf16 = ("gemm_stream",)
    begins_steps = True
    needs_f32_input = True  # behind a norm that does not place its rows
    MAX_COPIES = 16  # places per row that the norm's kernel takes (csrc/elementwise.cu)

    def __init__(self, table: torch.Tensor, we_gate_up: torch.Tensor, we_down: torch.Tensor, glu=K.SILU_GLU):
        E = we_gate_up.shape[0]
        if we_down.shape[0] != E or we_gate_up.shape[1] != 2 * we_down.shape[2] or we_gate_up.shape[2] != we_down.shape[1]:
            raise ValueError(f"expert weights do not fit: gate_up {tuple(we_gate_up.shape)}, down {tuple(we_down.shape)}")
        if table.dim() != 2 or table.is_floating_point() or not 1 <= table.shape[1] <= E:
            raise ValueError(f"a table of experts is integers [vocab, k] with k of at most {E} experts, not {table.dtype} {tuple(table.shape)}")
        if int(table.min()) < 0 or int(table.max()) >= E:
            raise ValueError(f"the table names experts {int(table.min())}..{int(table.max())}; there are {E}")
        ordered = table.sort(dim=1).values
        if bool((ordered[:, 1:] == ordered[:, :-1]).any()):
            raise ValueError("a row of the table names an expert twice")
        self.table = table.to(torch.int32).contiguous()
        self.interleaved = _can_interleave(we_gate_up)
        self.we_gate_up = interleave_gate_up(we_gate_up) if self.interleaved else we_gate_up.contiguous()
        self.we_down = we_down.contiguous()
        self.top_k, self.num_experts, self.glu = table.shape[1], E, tuple(glu)

    def begin_step(self, ctx: StepContext) -> None:
        n, k, E, dev = ctx.n_tokens, self.top_k, self.num_experts, self.table.device
        i32 = lambda size: torch.empty(size, dtype=torch.int32, device=dev)  # noqa: E731
        tiles, tile_rows = None, 0
        if self.we_gate_up.dtype == torch.bfloat16 and ctx.runtime.dtype == torch.bfloat16:
            tile_rows = K.gemm_stream_token_tile(group_rows_hint(n * k, E))
            tiles = (i32(2 * (-(-n * k // tile_rows) + E)), i32(1))
        chosen = i32(n * k) if "record_routing" in ctx.scratch else None
        routing = {"offsets": i32(E + 1), "pair": i32(n * k), "pos": i32(n * k), "tiles": tiles, "chosen": chosen, "ready": None}

        def sort():
            with scope("permute"):
                K.expert_sort(chosen, routing["offsets"], routing["pair"], routing["pos"], E, ctx.status, 0,
                              *((tile_rows, *tiles) if tiles is not None else ()), token_ids=ctx.token_ids, table=self.table)

        if ctx.workspace is None:
            sort()
        else:  # the buffers were made on the step's own stream, which joins the second one before they are read or freed
            main, side = torch.cuda.current_stream(), ctx.workspace.side_stream()
            side.wait_stream(main)
            with torch.cuda.stream(side):
                sort()
                routing["ready"] = side.record_event()
        ctx.scratch[("table_routing", id(self))] = routing

    def _routing(self, ctx: StepContext) -> dict:
        key = ("table_routing", id(self))
        if key not in ctx.scratch:
            self.begin_step(ctx)
        routing = ctx.scratch[key]
        if routing["ready"] is not None:
            torch.cuda.current_stream().wait_event(routing["ready"])
            routing["ready"] = None
        return routing

    def row_places(self, ctx: StepContext, n: int) -> RowPlaces | None:
        return RowPlaces(self._routing(ctx)["pos"], self.top_k) if self.top_k <= self.MAX_COPIES else None

    def forward(self, ctx: StepContext, h, h32, routing=None):
        rt, k, E = ctx.runtime, self.top_k, self.num_experts
        r = self._routing(ctx)
        offsets, pos, tiles = r["offsets"], r["pos"], r["tiles"]
        n, D = ctx.n_tokens, self.we_down.shape[1]
        if "record_routing" in ctx.scratch:
            ctx.scratch["record_routing"].append(r["chosen"].view(n, k))
        with scope("moe_routed_expert"):
            if isinstance(routing, RowPlaces):
                a_sorted = h
            else:
                a_sorted = torch.empty((n * k, D), dtype=rt.dtype, device=h32.device)
                K.permute_scale(h32, r["pair"], None, a_sorted, k)
            with scope("we_gate_up"):
                one_product = grouped_swiglu_streams(a_sorted, self.we_gate_up, self.interleaved)
                act = grouped_swiglu_linear(ctx, a_sorted, self.we_gate_up, offsets, self.interleaved, rt.dtype, 0, tiles, self.glu)
            with scope("we_down"):
                y = as_rows(grouped_linear(ctx, act, self.we_down, offsets, torch.float32, partials=True, tiles=tiles,
                                           after_grouped=one_product and not tracing_active()))

        def combine() -> torch.Tensor:
            delta = torch.empty((n, D), dtype=torch.float32, device=y.data.device)
            with scope("unpermute"):
                K.moe_combine(y.data, None, pos, delta, k, 1, y.splits, -1,
                              pair_weights=torch.full((n, k), 1.0 / k, dtype=torch.float32, device=y.data.device))
            return delta

        return RowSum([Rows(y.data, y.splits, pos, k, 0, None, 1.0 / k)], combine)


register_part("feed_forward", "table_routed_glu_experts", TableRoutedGLUExperts)
