"""Attention mixers that keep ONE tensor per token in the cache.

Both run causal softmax attention through the kernels of :mod:`.attention`
over pages that hold a single plane, read as keys and again as values.

``shared_kv_attention`` - grouped-query attention whose values are its keys::

    q_t = Wq h_t  (heads x dim),   k_t = Wk h_t  (kv_heads x dim),   v_t = k_t
    q_t <- q_t * (1 + coef * ln(floor((t + 1) / every) + 1))      (query temperature)
    o_t,i = sum_{j <= t} softmax_j(q_t,i . k_j,g(i) * scale) k_j,g(i);   y_t = Wo o_t

No rotation: the temperature is the only way a position enters.

``latent_attention`` - keys and values are made from a cached latent vector::

    c_t = rms(Wdkv h_t) * w_c                (rank numbers: all the cache keeps)
    k_j,i = Wuk,i c_j,   v_j,i = Wuv,i c_j,   score = q_t,i . k_j,i * scale
    o_t,i = sigmoid(Wg h_t)_i * sum_j softmax_j(score) v_j,i;   y_t = Wo o_t

Since ``q . (Wuk c) = (Wuk^T q) . c`` and ``sum_j p_j Wuv c_j = Wuv (sum_j p_j c_j)``,
the mixer multiplies the queries by ``Wuk^T`` per head, attends over the latent
pages as ONE shared key/value head of size ``rank``, and multiplies the result by
``Wuv`` per head: the keys and values themselves are never formed, for a prompt
portion no more than for a decoded token, so the logits at a position do not
depend on how the prompt was cut.

``latent_attention`` also takes the fuller form of the same idea: queries through a normed latent
of their own (``c_q = rms(Wdq h) w_q``, ``q = Wuq c_q``), a key part of ``rot_dim`` values that is not
made from the latent but projected directly, rotated by the position and shared by all heads (every
head's query carries ``rot_dim`` rotated values for it), a sliding window, and a gate per output
value instead of per head::

    score = (q_i[:dq] . Wuk,i c_j + rot(q_i[dq:]) . rot(k_j)) * scale

The cache keeps ``[c_j | rot(k_j)]`` per token, the absorbed query is ``[Wuk,i^T q_i[:dq] | rot(q_i[dq:])]``,
and attention runs over rows of ``rank + rot_dim`` values, of which the first ``rank`` are the "values".

In bfloat16, rows of other sizes than the paged kernels' (32, 64, 128) take two kernels of their own:
single tokens and short portions the absorbed form on tensor cores over rows of any width (each cached
row fetched once, used as key and as value); portions of :data:`EXPAND_FROM` tokens and more the expanded form - the
context's cached rows are gathered, ``Wuk`` and ``Wuv`` applied in one product, and every head scores its own
``dq + rot`` values on tcgen05: per query and key ``dq + rot + dv`` instead of ``2 rank + rot`` products, for
``rank (dq + dv)`` a key once.  Both compute the same function; which one a token takes depends on the
length of its portion, its logits do not beyond rounding.

The reference's models have neither mixer; its attention layer
(python/freetoken/models/minimax_m2/attention.py:29-84) is the pattern both follow.
"""

from __future__ import annotations

from typing import Dict, List

import numpy as np
import torch

from ..cache.manager import PagedKeyNeed
from ..csrc import ops
from ..weights.spec import Cat, Init, Name, TensorSpec
from . import linear
from .attention import PagedSoftmaxCore
from .base import POSITIONS, CacheView, Mixer, StepContext, StepPlan, StepShape, register_mixer

# portions of at least this many tokens make their context's keys and values (the expanded form)
EXPAND_FROM = 64
# largest buffer of expanded keys and values; contexts that do not fit stay with the absorbed form
EXPAND_BYTES = 1 << 30


def _both_planes(pages: torch.Tensor) -> torch.Tensor:
    """``[pages, kv_heads, page, d]`` seen as the kernels' ``[2 (K, V), ...]``: the same
    plane twice."""
    return pages.unsqueeze(0).expand(2, *pages.shape)


@register_mixer("shared_kv_attention")
class SharedKVAttention(PagedSoftmaxCore, Mixer):
    """params: ``hidden_size, num_heads, num_kv_heads, head_dim, sm_scale``,
    ``q_temp_coef`` (0: no temperature), ``q_temp_every``, ``sliding_window`` (None: all
    keys), ``scope`` and ``names`` (q, k, o and the merged qk tensor below the scope)."""

    graph_capturable = True
    writes_into_out = True

    def __init__(self, spec, prefix):
        super().__init__(spec, prefix)
        p = spec.params
        self.hidden = int(p["hidden_size"])
        self.nq = int(p["num_heads"])
        self.nkv = int(p["num_kv_heads"])
        self.d = int(p["head_dim"])
        self.scale = float(p["sm_scale"])
        self.temp_coef = float(p.get("q_temp_coef", 0.0))
        self.temp_every = int(p.get("q_temp_every", 1))
        self.window = p.get("sliding_window")
        if self.nkv <= 0 or self.nq % self.nkv:
            raise ValueError(f"num_heads {self.nq} is not a multiple of num_kv_heads {self.nkv}")
        if self.d > 1024:
            raise ValueError(f"head_dim {self.d} exceeds what the attention kernels take (1024)")
        if self.temp_coef != 0.0 and self.temp_every <= 0:
            raise ValueError("q_temp_every must be positive")
        names = p["names"]
        scope = self.name(p["scope"])
        self.n_qk = f"{scope}.{names['qk']}"
        self.n_q, self.n_k, self.n_o = (f"{scope}.{names[k]}" for k in ("q", "k", "o"))
        self.w_qk = self.w_o = None

    def cache_need(self):
        return PagedKeyNeed(self.nkv, self.d, self.window)

    def tensor_specs(self) -> List[TensorSpec]:
        qn, kn = self.nq * self.d, self.nkv * self.d
        return [
            TensorSpec(self.n_qk, (qn + kn, self.hidden), sources=(Cat((
                Name(self.n_q, (qn, self.hidden)), Name(self.n_k, (kn, self.hidden))), 0),)),
            TensorSpec(self.n_o, (self.hidden, qn), tag="residual_out"),
        ]

    def bind(self, tensors: Dict[str, torch.Tensor], dtype) -> None:
        self.w_qk = tensors[self.n_qk]
        self.w_o = tensors[self.n_o]

    def libraries(self, dtype) -> List[str]:
        return ["rowwise"] + self.attention_libraries(dtype) + linear.libraries(dtype)

    def forward(self, ctx: StepContext, x: torch.Tensor, cache: CacheView, out=None) -> torch.Tensor:
        T = x.shape[0]
        ws = ctx.workspace
        qn, kn = self.nq * self.d, self.nkv * self.d
        qk = linear.linear(x, self.w_qk, ws.get("kattn.qk", (T, qn + kn), ctx.dtype))
        q = ws.get("kattn.q", (T, qn), ctx.dtype)
        table = ctx.block_tables[cache.block_table_index]
        ops.key_store(qk, q, cache.pages if cache.writes else None, None, ctx.token_pos, ctx.token_seg,
                      table, q_off=0, k_off=qn, num_heads=self.nq, q_dim=self.d, num_kv_heads=self.nkv,
                      k_dim=self.d, temp_coef=self.temp_coef, temp_every=self.temp_every)
        o = ws.get("kattn.o", (T, qn), ctx.dtype)
        self.attend(ctx, q, o, _both_planes(cache.pages), table)
        if out is None:
            out = ws.get("kattn.y", (T, self.hidden), ctx.dtype)
        return linear.linear(o, self.w_o, out)


@register_mixer("latent_attention")
class LatentAttention(PagedSoftmaxCore, Mixer):
    """params: ``hidden_size, num_heads, qk_dim, v_dim, rank, sm_scale, norm_eps``,
    ``output_gate`` (a sigmoid gate per head, read from the mixer's input),
    ``scope`` and ``names`` (q, down, gate, latent_norm, up_k, up_v, o and the merged input
    projection below the scope).

    Options of the fuller form (module docstring): ``q_rank`` (queries through a normed latent of
    that size; ``names`` then also has q_down, q_norm, q_up), ``rot_dim`` with ``position`` (a PartSpec;
    the rotated key part and the rotated tail of every head's query), ``sliding_window``, ``gate_per``
    (``"head"``, the default, or ``"element"``: one gate per output value)."""

    graph_capturable = True
    writes_into_out = True

    def __init__(self, spec, prefix):
        super().__init__(spec, prefix)
        p = spec.params
        self.hidden = int(p["hidden_size"])
        self.nq = int(p["num_heads"])
        self.nkv = 1                       # every head attends over the one latent
        self.dq = int(p["qk_dim"])
        self.dv = int(p["v_dim"])
        self.d = self.rank = int(p["rank"])
        self.scale = float(p["sm_scale"])
        self.eps = float(p["norm_eps"])
        self.gated = bool(p.get("output_gate", True))
        self.window = p.get("sliding_window")
        self.q_rank = int(p["q_rank"]) if p.get("q_rank") else None
        self.rot = int(p.get("rot_dim") or 0)
        self.gate_per = str(p.get("gate_per", "head"))
        if self.gate_per not in ("head", "element"):
            raise ValueError("gate_per must be 'head' or 'element'")
        self.d = self.rank + self.rot          # a cached row, and the head size the kernels see
        self.position = None
        if self.rot:
            pos_spec = p["position"]
            self.position = POSITIONS.get(pos_spec.kind)(pos_spec, prefix)
            if self.position.rotary_dim != self.rot:
                raise ValueError(f"latent_attention: the position part turns {self.position.rotary_dim} "
                                 f"dimensions, the rotated key part has {self.rot}")
        self.full = bool(self.rot or self.q_rank or self.gate_per == "element" or not self.gated)
        if self.d > 1024:
            raise ValueError(f"latent rank plus rotated part {self.d} exceeds what the attention kernels take (1024)")
        names = p["names"]
        scope = self.name(p["scope"])
        self.n = {k: f"{scope}.{v}" for k, v in names.items()}
        self.w_in = self.w_norm = self.w_uk = self.w_uv = self.w_ukt = self.w_o = None
        self.w_qnorm = self.w_uq = None
        self.n_up = f"{scope}.{names.get('up', 'up_kv')}"        # [Wuk ; Wuv], one matrix of the model
        self.w_up = None
        self.own_kernels = False           # rows the paged kernels have no size for (bind decides)
        self.expands = False

    def _takes_own_kernels(self, dtype) -> bool:
        return (self.full and self.d not in ops.DECODE_HEAD_DIMS and self.dq % 8 == 0
                and ops.attn_latent_takes(dtype, self.d, self.rank))

    def _expands(self, dtype) -> bool:
        return (self._takes_own_kernels(dtype) and ops.attn_prefill_mha_takes(dtype, self.dq, self.rot, self.dv)
                and self.w_in_width() % 8 == 0)

    def w_in_width(self) -> int:
        return (self.q_rank or self.nq * (self.dq + self.rot)) + self.rank + self.rot + self._gate_width()

    # ---- step metadata of the kernels of its own ----------------------------------------
    def step_plan_key(self):
        if not self.own_kernels:
            return super().step_plan_key()
        return ("latent_attention", self.nq, self.dq + self.dv, self.d, self.rank, self.window, self.expands)

    def plan_step(self, shape: StepShape) -> StepPlan:
        """Which segments take which form, the row tiles of the absorbed one, the query tiles, context
        blocks and plain rows of the expanded one."""
        if not self.own_kernels:
            return super().plan_step(shape)
        rt = ops.latent_row_tile(self.nq, self.d, self.rank)
        room = EXPAND_BYTES // (2 * self.nq * (self.dq + self.dv)) // 64 * 64
        flat, tiles, blocks = [], [], []
        rows, flat_kv, first, last = 0, 0, None, 0
        for i, s in enumerate(shape.segments):
            base = max(0, s.pos0 - self.window + 1) // 64 * 64 if self.window else 0
            context = -(-(s.pos0 + s.n - base) // 64) * 64
            if self.expands and s.n >= EXPAND_FROM and rows + context <= room:
                tiles += [(i, q0, rows - base) for q0 in range(0, s.n, ops.MHA_QUERY_TILE)]
                blocks += [(i, base + k, rows + k) for k in range(0, context, 64)]
                rows += context
                continue
            flat += [(i, r) for r in range(0, s.n * self.nq, rt)]
            flat_kv = max(flat_kv, s.pos0 + s.n)
            first, last = s.q_start if first is None else first, s.q_start + s.n
        if shape.max_q_len == 1:           # whole block-table rows: a captured graph stays put while contexts grow
            flat_kv = shape.table_width * shape.page_size
        arrays = {}
        for names, items in ((("flat_seg", "flat_row"), flat), (("x_seg", "x_q0", "x_row0"), tiles),
                             (("g_seg", "g_key0", "g_row0"), blocks)):
            table = np.asarray(items, dtype=np.int32).reshape(-1, len(names))
            for c, name in enumerate(names):
                arrays[name] = np.ascontiguousarray(table[:, c])
        return StepPlan(arrays=arrays, host={"flat": len(flat), "flat_kv": flat_kv, "flat_tokens": (first or 0, last),
                                             "expanded": len(tiles), "rows": rows})

    def children(self):
        return [self.position] if self.position is not None else []

    def cache_need(self):
        return PagedKeyNeed(1, self.d, self.window)

    def _gate_width(self) -> int:
        if not self.gated:
            return 0
        return self.nq if self.gate_per == "head" else self.nq * self.dv

    def tensor_specs(self) -> List[TensorSpec]:
        H, W, R = self.nq, self.hidden, self.rank
        q_width = H * (self.dq + self.rot)
        if self.q_rank:
            pieces = [Name(self.n["q_down"], (self.q_rank, W))]
        else:
            pieces = [Name(self.n["q"], (q_width, W))]
        pieces.append(Name(self.n["down"], (R + self.rot, W)))
        if self.gated:
            pieces.append(Name(self.n["gate"], (self._gate_width(), W)))
        specs = [
            TensorSpec(self.n["in"], (sum(piece.shape[0] for piece in pieces), W), sources=(Cat(tuple(pieces), 0),)),
            TensorSpec(self.n["latent_norm"], (R,), role="small32", init=Init(mean=1.0, std=0.0), tag="norm"),
            TensorSpec(self.n_up, (H * (self.dq + self.dv), R), sources=(Cat((
                Name(self.n["up_k"], (H * self.dq, R)), Name(self.n["up_v"], (H * self.dv, R))), 0),)),
            TensorSpec(self.n["o"], (W, H * self.dv), tag="residual_out"),
        ]
        if self.q_rank:
            specs += [TensorSpec(self.n["q_norm"], (self.q_rank,), role="small32", init=Init(mean=1.0, std=0.0),
                                 tag="norm"),
                      TensorSpec(self.n["q_up"], (q_width, self.q_rank))]
        return specs

    def bind(self, tensors: Dict[str, torch.Tensor], dtype) -> None:
        H, R = self.nq, self.rank
        self.w_in = tensors[self.n["in"]]
        self.w_norm = tensors[self.n["latent_norm"]]
        self.w_up = tensors[self.n_up]
        self.w_uk = self.w_up[:H * self.dq].view(H, self.dq, R)      # [head][dq, R]
        self.w_uv = self.w_up[H * self.dq:].view(H, self.dv, R)      # [head][dv, R]
        self.own_kernels, self.expands = self._takes_own_kernels(dtype), self._expands(dtype)
        # the CUDA-core product wants [N, K] rows: Wuk^T per head
        self.w_ukt = self.w_uk.transpose(1, 2).contiguous() if dtype == torch.float32 else None
        self.w_o = tensors[self.n["o"]]
        if self.q_rank:
            self.w_qnorm = tensors[self.n["q_norm"]]
            self.w_uq = tensors[self.n["q_up"]]

    def libraries(self, dtype) -> List[str]:
        if self._takes_own_kernels(dtype):
            return (["rowwise", "attention_latent"] + (["attention_prefill_mha"] if self._expands(dtype) else [])
                    + linear.libraries(dtype))
        return ["rowwise"] + self.attention_libraries(dtype) + linear.libraries(dtype)

    def _attend_own(self, ctx: StepContext, z, q, at: int, cache: CacheView, table) -> torch.Tensor:
        """Cache rows, then both forms of the attention, each on its segments; the heads' values ``[T, H * dv]``."""
        T, ws = z.shape[0], ctx.workspace
        H, R, dq, dv, rot, d = self.nq, self.rank, self.dq, self.dv, self.rot, self.d
        plan = ctx.plan(self)
        host, lists = plan.host, plan.tensors
        q_abs = ws.get("lattn.q", (T, H, d), ctx.dtype) if host["flat"] else None
        cos_sin = self.position.table(ctx.device, ctx.max_positions) if rot else None
        ops.latent_store(z[:, at:at + R + rot], q, q_abs, cache.pages if cache.writes else None, self.w_norm,
                         cos_sin, ctx.token_pos, ctx.token_seg, table, heads=H, q_dim=dq, rank=R, rot=rot,
                         interleaved=bool(rot and self.position.interleaved), eps=self.eps,
                         turn_q=host["expanded"] > 0)
        y = ws.get("lattn.v", (T, H * dv), ctx.dtype)
        if host["flat"]:
            # the tokens from the first to the last absorbed segment; whatever lies between is overwritten below
            t0, t1 = host["flat_tokens"]
            q_heads = q[t0:t1].unflatten(1, (H, dq + rot))[:, :, :dq]
            torch.bmm(q_heads.transpose(0, 1), self.w_uk, out=q_abs[t0:t1, :, :R].transpose(0, 1))
            o = ws.get("lattn.o", (T, H, R), ctx.dtype)
            ops.attn_latent(q_abs, o, cache.pages, lists["flat_seg"], lists["flat_row"], ctx.seg_q_start,
                            ctx.seg_pos0, table, H, R, self.scale, self.window, host["flat_kv"], ws)
            torch.bmm(o[t0:t1].transpose(0, 1), self.w_uv.transpose(1, 2),
                      out=y.view(T, H, dv)[t0:t1].transpose(0, 1))
        if host["expanded"]:
            rows = host["rows"]
            plain = ws.get("lattn.rows", (rows, d), ctx.dtype)
            ops.latent_gather(cache.pages, plain, lists["g_seg"], lists["g_key0"], lists["g_row0"], ctx.seg_kv_len,
                              ctx.seg_pos0, table, self.window)
            made = ws.get("lattn.kv", (rows, H * (dq + dv)), ctx.dtype)
            torch.matmul(plain[:, :R], self.w_up.t(), out=made)
            ops.attn_prefill_mha(q, made[:, :H * dq].unflatten(1, (H, dq)), plain[:, R:] if rot else None,
                                 made[:, H * dq:].unflatten(1, (H, dv)), y, lists["x_seg"], lists["x_q0"],
                                 lists["x_row0"], ctx.seg_q_start, ctx.seg_pos0, H, dq, rot, dv, self.scale,
                                 self.window)
        return y

    def _gate(self, y, z, at: int) -> None:
        gate = z[:, at + self.d:]
        if self.gate_per == "head":
            ops.gate_heads(y, gate, self.nq, self.dv)
        else:
            ops.gate_heads(y, gate, self.nq * self.dv, 1)

    def _forward_full(self, ctx: StepContext, x: torch.Tensor, cache: CacheView, out=None) -> torch.Tensor:
        """The fuller form: a query latent, a rotated key part, a window, a gate per value."""
        T, ws = x.shape[0], ctx.workspace
        H, R, dq, dv, rot, d = self.nq, self.rank, self.dq, self.dv, self.rot, self.d
        z = linear.linear(x, self.w_in, ws.get("lattn.in", (T, self.w_in.shape[0]), ctx.dtype))
        q_width = H * (dq + rot)
        if self.q_rank:
            cq = ws.get("lattn.cq", (T, self.q_rank), ctx.dtype)
            ops.rms_rows(z[:, :self.q_rank], self.w_qnorm, cq, self.eps)
            q = linear.linear(cq, self.w_uq, ws.get("lattn.q_up", (T, q_width), ctx.dtype))
            at = self.q_rank
        else:
            q, at = z[:, :q_width], q_width
        table = ctx.block_tables[cache.block_table_index]
        if self.own_kernels:
            y = self._attend_own(ctx, z, q, at, cache, table)
            if self.gated:
                self._gate(y, z, at)
            return linear.linear(y, self.w_o, ws.get("lattn.y", (T, self.hidden), ctx.dtype) if out is None else out)
        q_abs = ws.get("lattn.q", (T, H, d), ctx.dtype)
        cos_sin = self.position.table(ctx.device, ctx.max_positions) if rot else None
        ops.latent_store(z[:, at:at + R + rot], q, q_abs, cache.pages if cache.writes else None, self.w_norm,
                         cos_sin, ctx.token_pos, ctx.token_seg, table, heads=H, q_dim=dq, rank=R, rot=rot,
                         interleaved=bool(rot and self.position.interleaved), eps=self.eps)
        # the unrotated part of every head's query into the latent's space: Wuk^T q per head
        q_heads = q.view(T, H, dq + rot)[:, :, :dq] if q.is_contiguous() else \
            q.unflatten(1, (H, dq + rot))[:, :, :dq]
        if ctx.dtype == torch.float32:
            ops.gemm_heads(q_heads, self.w_ukt, q_abs[:, :, :R])
        else:
            torch.bmm(q_heads.transpose(0, 1), self.w_uk, out=q_abs[:, :, :R].transpose(0, 1))
        o = ws.get("lattn.o", (T, H * d), ctx.dtype)
        self.attend(ctx, q_abs.view(T, H * d), o, _both_planes(cache.pages), table)
        # the first rank values of a head's result are the weighted latents: Wuv per head, then the gate
        y = ws.get("lattn.v", (T, H * dv), ctx.dtype)
        o_latent = o.view(T, H, d)[:, :, :R]
        if ctx.dtype == torch.float32:
            ops.gemm_heads(o_latent, self.w_uv, y.view(T, H, dv))
        else:
            torch.bmm(o_latent.transpose(0, 1), self.w_uv.transpose(1, 2), out=y.view(T, H, dv).transpose(0, 1))
        if self.gated:
            self._gate(y, z, at)
        if out is None:
            out = ws.get("lattn.y", (T, self.hidden), ctx.dtype)
        return linear.linear(y, self.w_o, out)

    def forward(self, ctx: StepContext, x: torch.Tensor, cache: CacheView, out=None) -> torch.Tensor:
        if self.full:
            return self._forward_full(ctx, x, cache, out)
        T = x.shape[0]
        ws = ctx.workspace
        H, R, dq, dv = self.nq, self.rank, self.dq, self.dv
        width = self.w_in.shape[0]
        z = linear.linear(x, self.w_in, ws.get("lattn.in", (T, width), ctx.dtype))
        table = ctx.block_tables[cache.block_table_index]
        # the latent: RMS norm in float32, into the token's place of the page
        ops.key_store(z, None, cache.pages if cache.writes else None, self.w_norm, ctx.token_pos,
                      ctx.token_seg, table, q_off=0, k_off=H * dq, num_heads=H, q_dim=dq, num_kv_heads=1,
                      k_dim=R, eps=self.eps)
        # queries into the latent's space: q' = Wuk^T q per head
        q = ws.get("lattn.q", (T, H * R), ctx.dtype)
        q_heads = z[:, :H * dq].view(T, H, dq)
        if ctx.dtype == torch.float32:
            ops.gemm_heads(q_heads, self.w_ukt, q.view(T, H, R))
        else:
            torch.bmm(q_heads.transpose(0, 1), self.w_uk, out=q.view(T, H, R).transpose(0, 1))
        o = ws.get("lattn.o", (T, H * R), ctx.dtype)
        self.attend(ctx, q, o, _both_planes(cache.pages), table)
        # back out of the latent's space: Wuv per head, then the gate
        y = ws.get("lattn.v", (T, H * dv), ctx.dtype)
        if ctx.dtype == torch.float32:
            ops.gemm_heads(o.view(T, H, R), self.w_uv, y.view(T, H, dv))
        else:
            torch.bmm(o.view(T, H, R).transpose(0, 1), self.w_uv.transpose(1, 2),
                      out=y.view(T, H, dv).transpose(0, 1))
        if self.gated:
            ops.gate_heads(y, z[:, H * dq + R:], H, dv)
        if out is None:
            out = ws.get("lattn.y", (T, self.hidden), ctx.dtype)
        return linear.linear(y, self.w_o, out)
