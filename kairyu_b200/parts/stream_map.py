"""Maps of the whole residual stream that run between two layers (``ModelSpec.stream_map``)."""

from __future__ import annotations

from typing import Any, Mapping, Optional

import torch

from kairyu_b200 import kernels
from kairyu_b200.parts.base import STREAM_MAPS, StepContext, StreamMap, TensorSpec


@STREAM_MAPS.register("origin_concat")
class OriginConcat(StreamMap):
    """``x <- W [x; x0]``: the stream and the embedding output side by side through one matrix ([hidden, 2 * hidden],
    the stream's columns first), as a looped model feeds its input to every pass anew.

    What the layer before left to add is added on the way, in 32-bit, by the kernel that writes the product's rows; the
    product's result is the new fp32 stream."""

    graph_safe = True

    def __init__(self, *, name: str, hidden_size: int, dtype: torch.dtype, device: str, **_: object) -> None:
        self.name = name
        self.hidden_size = hidden_size
        self.dtype = dtype
        self.weight: Optional[torch.Tensor] = None

    def tensor_specs(self) -> list[TensorSpec]:
        return [TensorSpec(self.name, (self.hidden_size, 2 * self.hidden_size))]

    def load(self, tensors: Mapping[str, torch.Tensor]) -> None:
        self.weight = tensors[self.name].contiguous()

    def bytes_streamed(self) -> int:
        return self.weight.numel() * self.weight.element_size()

    def apply(self, residual: torch.Tensor, delta: Any, origin: torch.Tensor, ctx: StepContext) -> torch.Tensor:
        if delta is not None and not isinstance(delta, kernels.PendingGated):
            raise ValueError("this stream map follows blocks that leave a gated sum or nothing to add")
        both = ctx.workspace.buffer("stream_map.rows", residual.shape[0], 2 * self.hidden_size, self.dtype)
        kernels.gated_residual_norm(residual, delta, None, 0.0, both, origin=origin)
        kernels.linear(both, self.weight, None, residual)
        return residual
