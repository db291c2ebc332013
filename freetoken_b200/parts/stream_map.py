"""Maps of the residual stream between layers.

``embedding_mix`` - the stream and the embedded row go through one matrix (in front of every pass of
a span of layers that runs several times)::

    x <- W [x ; x0]        x0: the stream as the embedding left it

``[x ; x0]`` is one row of 2 H activations per token: the second half is written once a step, the
first half by the launch that joins what the layer before left pending (its norm, the sum and the
copy in one).  The product leaves its float32 accumulator in the stream's place.

The reference's models have no such map; its layers follow each other directly
(python/freetoken/models/minimax_m2/model.py:48-52).
"""

from __future__ import annotations

from typing import Dict, List

import torch

from ..csrc import ops
from ..weights.spec import TensorSpec
from . import linear
from .base import StepContext, StreamMap, register_stream_map
from .norm import add_pending


@register_stream_map("embedding_mix")
class EmbeddingMix(StreamMap):
    """params: ``hidden_size``, ``tensor`` (the matrix ``[H, 2 H]``, the stream's columns first)."""

    graph_capturable = True

    def __init__(self, spec, prefix):
        super().__init__(spec, prefix)
        self.hidden = int(spec.params["hidden_size"])
        self.weight_name = self.name(spec.params["tensor"])
        self.weight = None

    def tensor_specs(self) -> List[TensorSpec]:
        return [TensorSpec(self.weight_name, (self.hidden, 2 * self.hidden))]

    def bind(self, tensors: Dict[str, torch.Tensor], dtype) -> None:
        self.weight = tensors[self.weight_name]

    def libraries(self, dtype) -> List[str]:
        return ["rowwise"] + linear.libraries(dtype)

    def _pair(self, ctx: StepContext) -> torch.Tensor:
        return ctx.workspace.get(f"stream_map.{self.weight_name}", (ctx.num_tokens, 2 * self.hidden), ctx.dtype)

    def begin(self, ctx: StepContext, residual: torch.Tensor) -> None:
        ops.cast_rows(residual, self._pair(ctx)[:, self.hidden:])

    def forward(self, ctx: StepContext, delta, residual: torch.Tensor) -> None:
        pair = self._pair(ctx)
        add_pending(ctx, delta, residual, pair[:, :self.hidden])
        linear.linear(pair, self.weight, residual)
