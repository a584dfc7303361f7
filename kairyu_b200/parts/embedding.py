"""Token embedding and output head (kairyu/models/llama.py:217, 261-273, 612-614)."""

from __future__ import annotations

from typing import Mapping, Optional

import torch

from kairyu_b200 import kernels
from kairyu_b200.parts.base import EMBEDDINGS, HEADS, NORMS, Part, PartSpec, StepContext, TensorSpec


@EMBEDDINGS.register("token_embedding")
class TokenEmbedding(Part):
    """``x = E[token_ids] * scale`` (``scale`` 1 unless given); the residual it starts is fp32.  ``norm``: an RMS norm
    (``rmsnorm``) on those rows, in the gather's kernel.  ``keep_origin``: the rows are also kept, unchanged for the
    whole step, for a stream map that reads the embedding output again (``origin``)."""

    graph_safe = True

    def __init__(self, *, name: str, vocab_size: int, hidden_size: int, dtype: torch.dtype, device: str, scale: float = 1.0,
                 norm: Optional[PartSpec] = None, keep_origin: bool = False, **_: object) -> None:
        if norm is not None and norm.kind != "rmsnorm":
            raise ValueError(f"the embedding's kernel takes an RMS norm, not {norm.kind!r}")
        self.norm = NORMS.build(norm, dtype=dtype, device=device) if norm is not None else None
        self.keep_origin = bool(keep_origin)
        self.name = name
        self.scale = float(scale)
        self.vocab_size = vocab_size
        self.hidden_size = hidden_size
        self.weight: Optional[torch.Tensor] = None

    def tensor_specs(self) -> list[TensorSpec]:
        return [TensorSpec(self.name, (self.vocab_size, self.hidden_size))] + (self.norm.tensor_specs() if self.norm is not None else [])

    def load(self, tensors: Mapping[str, torch.Tensor]) -> None:
        self.weight = tensors[self.name].contiguous()
        if self.norm is not None:
            self.norm.load(tensors)

    def origin(self, ctx: StepContext) -> torch.Tensor:
        """The step's embedding output, as ``forward`` left it."""
        if not self.keep_origin:
            raise ValueError("this embedding keeps no copy of its output")
        return ctx.workspace.buffer("embedding.origin", ctx.num_tokens, self.hidden_size, torch.float32)

    def forward(self, ctx: StepContext) -> torch.Tensor:
        out = ctx.workspace.buffer("residual", ctx.num_tokens, self.hidden_size, torch.float32)
        if self.norm is None and not self.keep_origin:
            kernels.embedding(self.weight, ctx.token_ids, out, ctx.error_flag, scale=self.scale)
            return out
        kernels.embedding_norm(self.weight, ctx.token_ids, out, weight=self.norm.weight if self.norm is not None else None,
                               eps=self.norm.eps if self.norm is not None else 0.0, scale=self.scale,
                               origin=self.origin(ctx) if self.keep_origin else None, flag=ctx.error_flag)
        return out


@HEADS.register("linear_head")
class LinearHead(Part):
    """``logits = h @ W^T`` in fp32 output; ``tied_to`` names the embedding
    tensor to share when the file has no head tensor of its own."""

    graph_safe = True

    def __init__(
        self,
        *,
        name: str,
        vocab_size: int,
        hidden_size: int,
        tied_to: Optional[str],
        dtype: torch.dtype,
        device: str,
        **_: object,
    ) -> None:
        self.name = name
        self.vocab_size = vocab_size
        self.hidden_size = hidden_size
        self.tied_to = tied_to
        self.weight: Optional[torch.Tensor] = None

    def tensor_specs(self) -> list[TensorSpec]:
        return [TensorSpec(self.name, (self.vocab_size, self.hidden_size), alias_of=self.tied_to)]

    def load(self, tensors: Mapping[str, torch.Tensor]) -> None:
        self.weight = tensors[self.name]

    def bytes_streamed(self) -> int:
        return self.weight.numel() * self.weight.element_size()

    def forward(self, hidden: torch.Tensor, ctx: StepContext) -> torch.Tensor:
        logits = ctx.workspace.buffer("logits", hidden.shape[0], self.vocab_size, torch.float32)
        kernels.linear(hidden, self.weight, None, logits)
        return logits
