"""RMSNorm with the residual add folded in.

``z = delta + residual; residual <- z; y = z * rsqrt(mean(z^2) + eps) * w``
in float32 (python/freetoken/kernel/triton/norm.py:101-112); ``plus_one``
selects the ``(1 + w)`` form (norm.py:69-72, python/freetoken/layers/norm.py:120-147).
The residual stream itself stays float32 between layers here (the reference
rounds it to the activation dtype each time it is stored, norm.py:108-109).
"""

from __future__ import annotations

from typing import Dict, List, Optional

import torch

from ..csrc import ops
from ..weights.spec import Init, TensorSpec
from .base import Norm, StepContext, register_norm


@register_norm("rmsnorm")
class RMSNorm(Norm):
    """params: ``size``, ``eps``, ``plus_one``, and ``scope`` (the tensor is ``<scope>.weight``
    below the prefix) or ``tensor`` (its whole name below the prefix).  ``scale_tensor`` (None: none):
    a second vector the normed values are multiplied by element by element (a layer scale behind a
    sublayer's output norm); the product of both vectors is formed once, in float32, at binding."""

    graph_capturable = True

    def __init__(self, spec, prefix):
        super().__init__(spec, prefix)
        self.size = int(spec.params["size"])
        self.eps = float(spec.params["eps"])
        self.plus_one = bool(spec.get("plus_one", False))
        self.weight_name = self.name(spec.get("tensor") or f"{spec.params['scope']}.weight")
        self.scale_name = self.name(spec.get("scale_tensor")) if spec.get("scale_tensor") else None
        if self.scale_name and self.plus_one:
            raise ValueError("a scale beside a one-plus norm weight is not offered")
        self.weight: Optional[torch.Tensor] = None

    def tensor_specs(self) -> List[TensorSpec]:
        mean = 0.0 if self.plus_one else 1.0
        return [TensorSpec(name, (self.size,), role="small32", init=Init(mean=mean, std=0.0), tag="norm")
                for name in (self.weight_name, self.scale_name) if name]

    def bind(self, tensors: Dict[str, torch.Tensor], dtype) -> None:
        self.weight = tensors[self.weight_name]
        if self.scale_name:
            self.weight = self.weight * tensors[self.scale_name]

    def libraries(self, dtype) -> List[str]:
        return ["elementwise", "rowwise"]

    def forward(self, ctx: StepContext, delta, residual: torch.Tensor) -> torch.Tensor:
        if isinstance(delta, NormedBranch):
            # the branch's own norm, the sum and this norm in one launch
            return delta.norm.add_normed(ctx, delta.y, residual, delta.mult, then=self)
        out = ctx.workspace.get("norm.out", residual.shape, ctx.dtype)
        ops.rmsnorm(plain_branch(ctx, delta), residual, self.weight, out, self.eps, self.plus_one)
        return out

    def add_normed(self, ctx: StepContext, branch, residual: torch.Tensor, mult: float,
                   then: Optional["RMSNorm"] = None, copy_out: Optional[torch.Tensor] = None
                   ) -> Optional[torch.Tensor]:
        """``residual += mult * norm(branch)`` in float32, this norm being the branch's own
        (``branch`` is ``[T, H]`` or ``[T, k, H]`` partial rows or :class:`ops.RoutedRows`, summed first).
        With ``then`` the new residual rows are normed by that norm in the same launch and returned;
        with ``copy_out`` they also leave as they are, in the activation type."""
        if then is None:
            ops.norm_add(branch, residual, self.weight, self.eps, self.plus_one, mult, copy_out=copy_out)
            return None
        out = ctx.workspace.get("norm.out", residual.shape, ctx.dtype)
        ops.norm_add(branch, residual, self.weight, self.eps, self.plus_one, mult, next_weight=then.weight,
                     next_eps=then.eps, next_plus_one=then.plus_one, next_out=out, copy_out=copy_out)
        return out


class NormedBranch:
    """A sublayer's output that has not joined the residual stream yet and passes a norm of its own
    first: ``x <- x + mult * norm(y)``.  A sandwich block hands it on where other blocks hand on a plain
    branch output; the next :class:`RMSNorm` (the next layer's or the model's last) folds it in with
    its own norm in one launch, :func:`add_pending` does it where no norm follows."""

    __slots__ = ("y", "norm", "mult")

    def __init__(self, y, norm: "RMSNorm", mult: float):
        self.y, self.norm, self.mult = y, norm, mult


def plain_branch(ctx: StepContext, delta):
    """``delta`` as a tensor of (partial) rows: a routed feed-forward's unsummed result is summed."""
    if isinstance(delta, ops.RoutedRows):
        rows = delta.rows
        out = ctx.workspace.get("norm.branch", (rows.shape[0], rows.shape[-1]), ctx.dtype)
        ops.branch_sum(delta, out)
        return out
    return delta


def add_pending(ctx: StepContext, delta, residual: torch.Tensor, copy_out: torch.Tensor) -> None:
    """Whatever a block left pending joins the plain residual stream; the new rows also leave, in the
    activation type, through ``copy_out`` (``[T, H]``, rows may lie further apart)."""
    if isinstance(delta, NormedBranch):
        delta.norm.add_normed(ctx, delta.y, residual, delta.mult, copy_out=copy_out)
        return
    if isinstance(delta, PendingBranch):
        raise ValueError("a branch with connection weights joins several streams, not the plain residual")
    ops.cast_rows(residual, copy_out, delta)


class PendingBranch:
    """A sublayer's output that has not joined the residual streams yet, with the connection
    weights it joins them by: ``x_t <- sum_s mix[s, t] x_s + out[t] y``.  A hyper-connected block
    hands it on where other blocks hand on a plain branch output; the next :class:`HyperNorm`
    (the next sublayer's, the next layer's or the model's last norm) folds it in."""

    __slots__ = ("y", "mix", "out")

    def __init__(self, y: torch.Tensor, mix: torch.Tensor, out: torch.Tensor):
        self.y, self.mix, self.out = y, mix, out


@register_norm("layer_norm")
class LayerNorm(Norm):
    """Layer norm with the residual add folded in: the pending branch joins, then ``(x - mean) / sqrt(variance +
    eps) * weight [+ bias]``, the variance being the mean of the squared deviations.  params: ``size``, ``eps``,
    ``tensor`` (the weight's name below the prefix), ``bias_tensor`` (None: no bias), ``factor`` (default 1): a
    constant on the result - in front of a head, a factor on the logits that costs no pass over them; it is
    multiplied into weight and bias at binding, in float32."""

    graph_capturable = True

    def __init__(self, spec, prefix):
        super().__init__(spec, prefix)
        p = spec.params
        self.size = int(p["size"])
        self.eps = float(p["eps"])
        self.factor = float(p.get("factor", 1.0))
        self.weight_name = self.name(p["tensor"])
        self.bias_name = self.name(p["bias_tensor"]) if p.get("bias_tensor") else None
        self.weight = self.bias = None

    def tensor_specs(self) -> List[TensorSpec]:
        specs = [TensorSpec(self.weight_name, (self.size,), role="small32", init=Init(mean=1.0, std=0.0), tag="norm")]
        if self.bias_name:
            specs.append(TensorSpec(self.bias_name, (self.size,), role="small32", init=Init(0.0, 0.02), tag="bias"))
        return specs

    def bind(self, tensors: Dict[str, torch.Tensor], dtype) -> None:
        self.weight = tensors[self.weight_name]
        self.bias = tensors[self.bias_name] if self.bias_name else None
        if self.factor != 1.0:
            self.weight = self.weight * self.factor
            self.bias = self.bias * self.factor if self.bias is not None else None

    def libraries(self, dtype) -> List[str]:
        return ["rowwise"]

    def _join(self, ctx: StepContext, delta, residual: torch.Tensor):
        """What is left to join: a branch with a norm of its own joins by a launch of its own."""
        if isinstance(delta, PendingBranch):
            raise ValueError("a branch with connection weights joins several streams, not the plain residual")
        if isinstance(delta, NormedBranch):
            delta.norm.add_normed(ctx, delta.y, residual, delta.mult)
            return None
        return delta

    def forward(self, ctx: StepContext, delta, residual: torch.Tensor) -> torch.Tensor:
        out = ctx.workspace.get("norm.out", residual.shape, ctx.dtype)
        ops.join_layer_norm(self._join(ctx, delta, residual), residual, self.weight, self.eps, out, self.bias)
        return out

    def forward_pair(self, ctx: StepContext, delta, residual: torch.Tensor, other: "LayerNorm"):
        """``(this norm's rows, other's rows)`` of the same new residual rows, in one launch."""
        out = ctx.workspace.get("norm.out", residual.shape, ctx.dtype)
        out2 = ctx.workspace.get("norm.out2", residual.shape, ctx.dtype)
        ops.join_layer_norm(self._join(ctx, delta, residual), residual, self.weight, self.eps, out, self.bias,
                            other.weight, other.eps, out2, other.bias)
        return out, out2


@register_norm("hyper_norm")
class HyperNorm(Norm):
    """The norm in front of a sublayer of a model with several residual streams
    (hyper-connections).  The residual is ``[T, streams, H]`` float32; the sublayer reads ``u =
    sum_s in[s] x_s``, normed here, and its output ``y`` later joins every stream: ``x_t <- sum_s
    mix[s, t] x_s + out[t] y`` (``mix`` is indexed ``[from, to]``).  One launch folds in the branch
    that is still pending, forms ``u`` and norms it.

    params: ``size``, ``eps``, ``streams``, ``tensor`` (the norm weight's name below the prefix),
    ``bias_tensor`` (None: no bias), ``center`` (default True: layer norm - the mean is taken off and
    the variance is the mean of the squared deviations; False: RMS norm), ``connection`` (the prefix
    of the ``in``, ``out`` and ``mix`` tensors below the layer's; None: the norm reads the plain sum
    of the streams and no branch leaves through it - the model's last norm; ``"identity"``: no
    tensors, every weight is one - with one stream the plain pre-norm residual ``x <- x + y``)."""

    graph_capturable = True

    def __init__(self, spec, prefix):
        super().__init__(spec, prefix)
        p = spec.params
        self.size = int(p["size"])
        self.eps = float(p["eps"])
        self.streams = int(p.get("streams", 1))
        self.center = bool(p.get("center", True))
        self.weight_name = self.name(p["tensor"])
        self.bias_name = self.name(p["bias_tensor"]) if p.get("bias_tensor") else None
        conn = p.get("connection")
        self.identity = conn == "identity"
        if self.identity and self.streams != 1:
            raise ValueError("connection weights of one are the plain residual: they need streams = 1")
        self.conn = {k: self.name(f"{conn}.{k}") for k in ("in", "out", "mix")} if conn and not self.identity else None
        self.weight = self.bias = self.w_in = self.w_out = self.w_mix = None

    def tensor_specs(self) -> List[TensorSpec]:
        S = self.streams
        specs = [TensorSpec(self.weight_name, (self.size,), role="small32", init=Init(mean=1.0, std=0.0), tag="norm")]
        if self.bias_name:
            specs.append(TensorSpec(self.bias_name, (self.size,), role="small32", init=Init(0.0, 0.02), tag="bias"))
        if self.conn:
            # near the plain residual sum: every stream keeps itself, reads and writes are spread evenly
            specs += [TensorSpec(self.conn["in"], (S,), role="small32", init=Init(1.0 / S, 0.1 / S), tag="connection"),
                      TensorSpec(self.conn["out"], (S,), role="small32", init=Init(1.0, 0.1), tag="connection"),
                      TensorSpec(self.conn["mix"], (S, S), role="small32", init=Init(0.0, 0.1 / S, eye=1.0), tag="connection_mix")]
        return specs

    def bind(self, tensors: Dict[str, torch.Tensor], dtype) -> None:
        self.weight = tensors[self.weight_name]
        self.bias = tensors[self.bias_name] if self.bias_name else None
        if self.conn:
            self.w_in, self.w_out, self.w_mix = (tensors[self.conn[k]] for k in ("in", "out", "mix"))
        elif self.identity:
            ones = torch.ones(1, dtype=torch.float32, device=self.weight.device)
            self.w_in, self.w_out, self.w_mix = ones, ones, ones.view(1, 1)

    def libraries(self, dtype) -> List[str]:
        return ["rowwise"]

    def pending(self, y: torch.Tensor) -> PendingBranch:
        """``y`` (this norm's sublayer's output) with the weights it joins the streams by."""
        if not self.conn and not self.identity:
            raise ValueError("a norm without connection weights has no sublayer whose output could leave through it")
        return PendingBranch(y, self.w_mix, self.w_out)

    def forward(self, ctx: StepContext, delta, residual: torch.Tensor) -> torch.Tensor:
        if residual.dim() == 2 and self.streams == 1:
            residual = residual.unsqueeze(1)          # one stream: the plain residual [T, H]
        if residual.dim() != 3 or residual.shape[1] != self.streams:
            raise ValueError(f"hyper_norm: the residual must be [T, {self.streams}, H]")
        if delta is not None and not isinstance(delta, PendingBranch):
            raise ValueError("hyper_norm: a branch reaches the streams through its connection weights "
                             "(PendingBranch), not as a plain tensor")
        T, _, H = residual.shape
        out = ctx.workspace.get("norm.out", (T, H), ctx.dtype)
        y, mix, w_out = (plain_branch(ctx, delta.y), delta.mix, delta.out) if delta is not None else (None, None, None)
        ops.hyper_norm(residual, y, mix, w_out, self.w_in, self.weight, self.bias, self.eps, self.center, out)
        return out
