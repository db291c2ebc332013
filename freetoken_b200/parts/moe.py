"""Top-k routed gated-linear-unit experts.

Router, all float32 (python/freetoken/models/minimax_m3/moe.py:71-81;
softmax variant python/freetoken/moe/fused.py:27-31):
``logits = x @ Wg^T``; ``s = sigmoid(logits)`` or ``softmax(logits)``;
experts are chosen by ``s + bias`` (the bias only chooses), weights are the
unbiased ``s`` of the chosen, optionally renormalised to sum 1, times ``scale``.

Experts (python/freetoken/moe/fused.py:267-337,
python/freetoken/layers/moe.py:83-92): routes are sorted by expert;
``m = act(Wgate_e x) * (Wup_e x)`` from one product against ``[gate; up]``;
``y_route = w_route * (Wdown_e m)`` with the weight applied to the float32
accumulator; ``y = sum over the k routes`` in float32, slot order.
Two options no model of the reference has: ``identity`` - the last outputs of the router stand for
experts without weights that hand the input back, times the route's weight (their routes are sorted
behind all others and no product touches them) - and ``shared``, a gated feed-forward every token
passes, added (``shared_gate``: times ``sigmoid(w h)``, one number per token, whose row rides behind the
router's in one float32 product).  With either the result is :class:`ops.RoutedRows`: the consumer's kernel adds the
routed rows, the handed-back input and the shared row in float32, in one pass.
Activation ``silu`` or ``swigluoai``
(python/freetoken/kernel/triton/activation.py:96-107).
"""

from __future__ import annotations

from typing import Dict, List

import torch

from ..csrc import ops
from ..weights.spec import Cat, Init, Name, Stack, TensorSpec
from . import linear
from .base import FEED_FORWARDS, FeedForward, StepContext, register_feed_forward


# Above this many rows per expert (on average) the experts run on the tcgen05
# grouped GEMM; below it the weight-streaming kernel reads each expert once.
# Measured on a B200 with 256 experts, top-8 (decode batches of 32 .. 512): at an
# average of 4 rows the two are level, at 6 the grouped GEMM is 6 % ahead, at 8 rows
# 20 % (the streaming kernel then reads many experts twice, 8 rows a pass).
TC_MIN_ROWS_PER_EXPERT = 4

# Up to this many tokens the router's logits come from the one-warp-per-expert
# kernel; above it from the tiled float32 product.
ROUTER_SMALL_T = 64


def bf16_terms(w: torch.Tensor) -> torch.Tensor:
    """``[terms * E, H]`` bfloat16 whose ``terms`` row blocks sum exactly to the
    float32 matrix ``w``: hi = bf16(w), mid = bf16(w - hi), lo = bf16(w - hi - mid)
    (three 8-bit pieces cover a 24-bit significand; the differences are exact in
    float32).  A product of bfloat16 activations with each term is exact in
    float32, so a tensor-core product with float32 accumulation over the terms
    computes the float32 router logits without rounding the weight."""
    if w.dtype == torch.bfloat16:
        return w
    terms, rest = [], w.float()
    for _ in range(3):
        t = rest.to(torch.bfloat16)
        terms.append(t)
        rest = rest - t.float()
    return torch.cat(terms, 0).contiguous()


@register_feed_forward("routed_experts")
class RoutedExperts(FeedForward):
    """params: ``hidden_size, intermediate_size, num_experts, top_k, scoring``
    (sigmoid | softmax), ``use_bias, renormalize, scale, activation`` (silu |
    swigluoai), ``act_alpha, act_limit, scope`` and ``checkpoint_names``
    (router, bias, gate_up, down: model-side names below the scope; gate, up,
    down_each: per-expert checkpoint names with ``{e}``).  ``groups`` and ``keep_groups``
    (default 1, 1: no groups): the experts form ``groups`` equal groups of neighbours, a group's
    value is the sum of its two largest choice scores (score plus bias; ``group_top`` 1: the largest), and
    only experts of the ``keep_groups`` best groups can be chosen.  ``identity`` (default 0): so many router outputs behind
    the ``num_experts`` experts' hand the input back.  ``shared`` (a PartSpec of a feed-forward, or
    None): one that runs for every token beside the routed experts; ``shared_gate`` (default False) gates
    it per token (``checkpoint_names`` then also has shared_gate, ``[1, hidden]``, and router_gate, the name
    of the merged matrix the model keeps)."""

    graph_capturable = True

    def __init__(self, spec, prefix):
        super().__init__(spec, prefix)
        p = spec.params
        self.hidden = int(p["hidden_size"])
        self.inter = int(p["intermediate_size"])
        self.E = int(p["num_experts"])
        self.k = int(p["top_k"])
        self.softmax = p.get("scoring", "sigmoid") == "softmax"
        self.use_bias = bool(p.get("use_bias", False))
        self.renorm = bool(p.get("renormalize", True))
        self.scale = float(p.get("scale", 1.0))
        self.act = p.get("activation", "silu")
        self.act_alpha = float(p.get("act_alpha", 1.702))
        self.act_limit = float(p.get("act_limit", 7.0))
        self.identity = int(p.get("identity") or 0)
        self.outputs = self.E + self.identity          # of the router
        if self.k > self.outputs:
            raise ValueError(f"top_k {self.k} exceeds the router's {self.outputs} outputs")
        self.groups = int(p.get("groups", 1))
        self.keep_groups = int(p.get("keep_groups", self.groups))
        if (self.groups < 1 or self.outputs % self.groups or not 1 <= self.keep_groups <= self.groups
                or self.keep_groups * (self.outputs // self.groups) < self.k or self.groups > 256):
            raise ValueError(f"{self.groups} groups of which {self.keep_groups} are kept do not fit "
                             f"{self.outputs} experts, top-{self.k}")
        self.group_top = int(p.get("group_top", 2))
        if self.group_top not in (1, 2):
            raise ValueError("a group's value is made of its largest one or two choice scores")
        self.shared = None
        self.shared_gate = bool(p.get("shared_gate", False))
        if self.shared_gate and (p.get("shared") is None or self.identity):
            raise ValueError("a gate on the shared feed-forward needs one (and no identity experts beside it)")
        if p.get("shared") is not None:
            self.shared = FEED_FORWARDS.get(p["shared"].kind)(p["shared"], prefix)
            if not self.shared.writes_into_out:
                raise ValueError("the shared feed-forward must be able to leave its result in a given place")
        names = p["checkpoint_names"]
        self.scope = self.name(p["scope"])
        self.n_router = f"{self.scope}.{names['router']}"
        self.n_bias = f"{self.scope}.{names['bias']}"
        self.n_gate_up = f"{self.scope}.{names['gate_up']}"
        self.n_down = f"{self.scope}.{names['down']}"
        if self.shared_gate:
            self.n_shared_gate = f"{self.scope}.{names['shared_gate']}"
            self.n_router_gate = f"{self.scope}.{names['router_gate']}"
        self.logit_rows = self.outputs + (1 if self.shared_gate else 0)
        self._each = {key: f"{self.scope}.{names[key]}" for key in ("gate", "up", "down_each")}
        self.w_router = self.w_router_terms = self.w_bias = self.w_gate_up = self.w_down = None

    def children(self):
        return [self.shared] if self.shared is not None else []

    def tensor_specs(self) -> List[TensorSpec]:
        E, I, H = self.E, self.inter, self.hidden
        gate_up = Stack(tuple(
            Cat((Name(self._each["gate"].format(e=e), (I, H)),
                 Name(self._each["up"].format(e=e), (I, H))), 0) for e in range(E)))
        down = Stack(tuple(Name(self._each["down_each"].format(e=e), (H, I)) for e in range(E)))
        router = TensorSpec(self.n_router, (self.outputs, H), role="small32", keep_float32_in_file=True)
        if self.shared_gate:
            router = TensorSpec(self.n_router_gate, (self.outputs + 1, H), role="small32", keep_float32_in_file=True,
                                sources=(Cat((Name(self.n_router, (self.outputs, H)),
                                              Name(self.n_shared_gate, (1, H))), 0),))
        return [
            router,
            TensorSpec(self.n_bias, (self.outputs,), role="small32", keep_float32_in_file=True,
                       init=Init(0.0, 0.01 if self.use_bias else 0.0), tag="router_bias",
                       optional=not self.use_bias),
            TensorSpec(self.n_gate_up, (E, 2 * I, H), sources=(gate_up,)),
            TensorSpec(self.n_down, (E, H, I), sources=(down,), tag="residual_out"),
        ] + (self.shared.tensor_specs() if self.shared is not None else [])

    def bind(self, tensors: Dict[str, torch.Tensor], dtype) -> None:
        self.w_router = tensors[self.n_router_gate if self.shared_gate else self.n_router]
        self.w_router_terms = bf16_terms(self.w_router) if dtype == torch.bfloat16 else None
        # The bias is part of the routing whenever the checkpoint carries it: the
        # reference's block always adds it (python/freetoken/models/minimax_m3/moe.py:75,
        # weight.py:220).  ``use_bias`` only decides whether its absence is an error.
        self.w_bias = tensors.get(self.n_bias)
        self.w_gate_up = tensors[self.n_gate_up]
        self.w_down = tensors[self.n_down]
        if self.shared is not None:
            self.shared.bind(tensors, dtype)

    def libraries(self, dtype) -> List[str]:
        libs = ["gemm_simt", "moe_route", "elementwise"] + (["rowwise"] if self.identity or self.shared else [])
        libs += [lib for lib in (self.shared.libraries(dtype) if self.shared else []) if lib not in libs]
        return libs + (["skinny_gemm", "moe_gemm_tc"] if dtype == torch.bfloat16 else [])

    # ---- forward ----------------------------------------------------------------
    def route(self, ctx: StepContext, x: torch.Tensor, sort_into=None):
        """``(ids [T,k] int32, weights [T,k] float32)``.  With ``sort_into``
        (counts, offsets, sorted_route, sorted_token, active) the routes may be
        sorted as well: returns ``(ids, weights, sorted?)``, the flag saying
        whether that was done here (a handful of tokens: one launch for both)."""
        T = x.shape[0]
        ws = ctx.workspace
        logits = ws.get("moe.logits", (T, self.logit_rows), torch.float32)
        terms = 1
        if ctx.dtype == torch.bfloat16 and T <= ROUTER_SMALL_T and ops.router_logits_takes(x, self.w_router):
            ops.router_logits(x, self.w_router, logits)
        elif ctx.dtype == torch.bfloat16 and self.w_router_terms is not None and linear.library_f32_out(
                x, self.w_router_terms, ws.get("moe.logit_terms", (T, self.w_router_terms.shape[0]),
                                               torch.float32)):
            # many rows: tensor-core products of the bfloat16 activations with the exact
            # bfloat16 terms of the float32 router weight; the terms are summed by the selection
            terms = self.w_router_terms.shape[0] // self.logit_rows
            logits = ws.get("moe.logit_terms", (T, self.w_router_terms.shape[0]), torch.float32)
        else:
            ops.gemm_rows(x, self.w_router, logits)
        ids = ws.get("moe.ids", (T, self.k), torch.int32)
        weights = ws.get("moe.weights", (T, self.k), torch.float32)
        gate = ws.get("moe.shared_gate", (T,), torch.float32) if self.shared_gate else None
        if sort_into is not None and ops.route_small_takes(T, self.outputs, self.k):
            ops.route_small(logits, self.w_bias, ids, weights, *sort_into, self.k, self.softmax,
                            self.renorm, self.scale, terms, self.groups, self.keep_groups, busy_of=self.E,
                            group_top=self.group_top, tail=gate)
            return ids, weights, True
        ops.router_select(logits, self.w_bias, ids, weights, self.k, self.softmax, self.renorm,
                          self.scale, terms, self.groups, self.keep_groups, self.group_top, gate)
        return (ids, weights) if sort_into is None else (ids, weights, False)

    def forward(self, ctx: StepContext, x: torch.Tensor):
        T = x.shape[0]
        R = T * self.k
        ws = ctx.workspace
        counts = ws.get("moe.counts", (self.outputs,), torch.int32)
        offsets = ws.get("moe.offsets", (self.outputs + 1,), torch.int32)
        sorted_route = ws.get("moe.sorted_route", (R,), torch.int32)
        sorted_token = ws.get("moe.sorted_token", (R,), torch.int32)
        active = ws.get("moe.active", (self.E + 1,), torch.int32)
        ids, weights, is_sorted = self.route(ctx, x, (counts, offsets, sorted_route, sorted_token, active))
        if not is_sorted:
            scratch = None
            if R >= ops.MOE_SORT_CHUNKED_FROM:
                scratch = ws.get("moe.sort_scratch", (ops.moe_sort_scratch(R, self.outputs),), torch.int32)
            ops.moe_sort(ids.view(-1), counts, offsets, sorted_route, sorted_token, active, self.outputs,
                         self.k, scratch, busy_of=self.E)
        if ctx.probe is not None:
            if "router_ids" in ctx.probe:
                ctx.probe["router_ids"].append(ids.clone())
            else:
                ctx.probe.setdefault("experts_touched", []).append(int((counts[:self.E] > 0).sum()))
        mid = ws.get("moe.mid", (R, self.inter), ctx.dtype)
        parts = ws.get("moe.parts", (R, self.hidden), ctx.dtype)
        self.experts(ctx, x, mid, parts, offsets, active, sorted_route, sorted_token,
                     weights.view(-1), R)
        # the k partial rows of a token are summed by whoever consumes them
        # (the next norm adds them into the residual in slot order)
        parts = parts.view(T, self.k, self.hidden)
        if self.shared is None and not self.identity:
            return parts
        extra = None
        if self.shared is not None:
            extra = self.shared.forward(ctx, x, out=ws.get("moe.shared", (T, self.hidden), ctx.dtype))
        if not self.identity:
            gate = ws.get("moe.shared_gate", (T,), torch.float32) if self.shared_gate else None
            return ops.RoutedRows(parts, extra=extra, extra_gate=gate)
        return ops.RoutedRows(parts, ids, weights, self.E, x, extra)

    def experts(self, ctx, x, mid, parts, offsets, active, sorted_route, sorted_token, route_weight, R):
        if ctx.dtype == torch.bfloat16 and R > TC_MIN_ROWS_PER_EXPERT * self.E \
                and ops.moe_gemm_tc_takes(x, self.w_gate_up, mid) \
                and ops.moe_gemm_tc_takes(mid, self.w_down, parts):
            # many rows per expert: tcgen05 grouped GEMM over the rows sorted by expert
            ops.moe_experts_tc(x, self.w_gate_up, self.w_down, mid, parts, offsets, active, sorted_route,
                               sorted_token, route_weight, R, self.act, self.act_alpha, self.act_limit,
                               ctx.workspace)
            return
        if ctx.dtype == torch.bfloat16 and ops.skinny_gemm_takes(x, self.w_gate_up, mid) \
                and ops.skinny_gemm_takes(mid, self.w_down, parts):
            per_pass = ops.pass_rows(-(-R // self.E))
            ops.skinny_gemm(x, self.w_gate_up, mid, group_offsets=offsets, active=active,
                            a_rows=sorted_token,
                            rows=R, glu=True, act=self.act, act_alpha=self.act_alpha,
                            act_limit=self.act_limit, rows_per_pass=per_pass)
            ops.skinny_gemm(mid, self.w_down, parts, group_offsets=offsets, active=active,
                            c_rows=sorted_route,
                            row_scale=route_weight, rows=R, rows_per_pass=per_pass)
            return
        ops.gemm_rows(x, self.w_gate_up, mid, group_offsets=offsets, a_rows=sorted_token, rows=R,
                      glu=True, act=self.act, act_alpha=self.act_alpha, act_limit=self.act_limit)
        ops.gemm_rows(mid, self.w_down, parts, group_offsets=offsets, c_rows=sorted_route,
                      row_scale=route_weight, rows=R)
