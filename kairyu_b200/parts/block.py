"""Arrangements of norms, mixer and feed-forward around the residual stream."""

from __future__ import annotations

from typing import Mapping, Optional

import torch

from kairyu_b200 import kernels
from kairyu_b200.parts.base import (
    BLOCKS,
    FEED_FORWARDS,
    MIXERS,
    NORMS,
    Block,
    CacheView,
    LayerSpec,
    Norm,
    StepContext,
    TensorSpec,
)


@BLOCKS.register("pre_norm")
class PreNormBlock(Block):
    """``x += mixer(norm(x)); x += ffn(norm(x))`` (kairyu/models/llama.py:88-101).

    The residual is fp32.  Each sub-layer's output is handed on as a pending
    delta and added by the next norm's kernel.

    For a few bf16 rows (decode) the norms have no kernel of their own: the product before a
    norm adds its result to the residual and leaves the rows weighted and their sums of squares
    (``kernels.ResidualNorm``), the product after it scales by the root mean square
    (``kernels.PreNormed``).  That needs norms that offer ``fold_target`` (RMSNorm does) and a
    mixer and feed-forward that offer ``fusable_norm``; any other part gets the plain flow.

    ``LayerSpec.options["scale_names"]`` (two tensors, a factor a column each): the sub-layers' outputs are scaled by them
    as they are added, ``x += s1 * mixer(norm(x)); x += s2 * ffn(norm(x))``; the scaling rides in whichever kernel adds
    (``kernels.PendingScaled``, ``ResidualNorm.scale``), in 32-bit.  A layer may have no feed-forward.
    """

    graph_safe = True

    takes_next_norm = True  # forward accepts the norm of the block that runs next

    def __init__(self, *, layer: LayerSpec, dtype: torch.dtype, device: str, shared: dict, **_: object) -> None:
        context = dict(dtype=dtype, device=device, shared=shared)
        self.mixer_norm = NORMS.build(layer.mixer_norm, **context)
        self.mixer = MIXERS.build(layer.mixer, **context)
        # a layer may have no feed-forward: the block is then x += mixer(norm(x)) alone
        self.ffn_norm = NORMS.build(layer.ffn_norm, **context) if layer.ffn is not None else None
        self.ffn = FEED_FORWARDS.build(layer.ffn, **context) if layer.ffn is not None else None
        self._parts = tuple(part for part in (self.mixer_norm, self.mixer, self.ffn_norm, self.ffn) if part is not None)
        names = layer.options.get("scale_names")
        self.scale_names = tuple(names)[: 1 if self.ffn is None else 2] if names is not None else ()
        self.size = int(layer.mixer_norm.params["size"]) if self.scale_names else 0
        self._scales: list[Optional[torch.Tensor]] = [None, None]  # fp32: they enter the residual sum

    def tensor_specs(self) -> list[TensorSpec]:
        scales = [TensorSpec(name, (self.size,), role="vector", init="norm") for name in self.scale_names]
        return [spec for part in self._parts for spec in part.tensor_specs()] + scales

    def load(self, tensors: Mapping[str, torch.Tensor]) -> None:
        for part in self._parts:
            part.load(tensors)
        for index, name in enumerate(self.scale_names):
            self._scales[index] = tensors[name].float().contiguous()

    def bytes_streamed(self) -> int:
        return sum(part.bytes_streamed() for part in self._parts) + sum(4 * s.numel() for s in self._scales if s is not None)

    def _pending(self, index: int, output: torch.Tensor):
        return output if self._scales[index] is None else kernels.PendingScaled(output, self._scales[index])

    def _fused(self, ctx: StepContext) -> bool:
        if ctx.dtype != torch.bfloat16 or not kernels.fused_norm_available():
            return False
        # a norm offers ``fold_target`` when the products around it can take its two halves
        for norm, part in ((self.mixer_norm, self.mixer), (self.ffn_norm, self.ffn)):
            if part is None:
                continue
            fusable = getattr(part, "fusable_norm", None)
            if not hasattr(norm, "fold_target") or fusable is None or not fusable(ctx.num_tokens):
                return False
        return True

    def prenorm_target(self, ctx: StepContext) -> Optional[Norm]:
        """The norm the block before this one may fold into its last product, or None."""
        return self.mixer_norm if self._fused(ctx) else None

    def forward(
        self,
        residual: torch.Tensor,
        delta,
        ctx: StepContext,
        cache: CacheView,
        next_norm: Optional[Norm] = None,
    ):
        if isinstance(delta, kernels.PreNormed):  # the block before has added its output and begun our norm
            normed = delta
        else:
            normed = self.mixer_norm.apply(residual, delta, ctx)
        fused = self._fused(ctx)
        if self.ffn is None:
            if not fused or next_norm is None:
                return residual, self._pending(0, self.mixer.forward(normed, ctx, cache))
            # (its own input may lie in the same buffer: the products that read it are done when the last one writes)
            fold = next_norm.fold_target(residual, ctx, "mixer", self._scales[0])
            return residual, self.mixer.forward(normed, ctx, cache, fold=fold)
        if not fused:
            mixed = self.mixer.forward(normed, ctx, cache)
            normed = self.ffn_norm.apply(residual, self._pending(0, mixed), ctx)
            return residual, self._pending(1, self.ffn.forward(normed, ctx))
        mixed = self.mixer.forward(normed, ctx, cache, fold=self.ffn_norm.fold_target(residual, ctx, "ffn", self._scales[0]))
        fold = next_norm.fold_target(residual, ctx, "mixer", self._scales[1]) if next_norm is not None else None
        output = self.ffn.forward(mixed, ctx, fold=fold)
        return residual, output if fold is not None else self._pending(1, output)


@BLOCKS.register("output_norm")
class OutputNormBlock(Block):
    """``x += norm1(mixer(x)); x += norm2(ffn(x))``: the norms sit on the sub-layers' outputs, and the
    sub-layers read the stream itself.  A layer may have no feed-forward.

    The residual is fp32; one kernel per sub-layer norms the output, adds it to the residual and
    leaves the residual's rows in the activation dtype for the next products (``Norm.add_normed``).
    That copy travels to the next block in place of a pending delta (``kernels.ResidualCopy``).  A
    feed-forward that can hand over its rows before their weighted sum (a mixture of experts) does,
    and the same kernel adds them.
    """

    graph_safe = True

    def __init__(self, *, layer: LayerSpec, dtype: torch.dtype, device: str, shared: dict, **_: object) -> None:
        context = dict(dtype=dtype, device=device, shared=shared)
        self.dtype = dtype
        self.mixer = MIXERS.build(layer.mixer, **context)
        self.mixer_norm = NORMS.build(layer.mixer_norm, **context)
        self.ffn = FEED_FORWARDS.build(layer.ffn, **context) if layer.ffn is not None else None
        self.ffn_norm = NORMS.build(layer.ffn_norm, **context) if layer.ffn is not None else None
        self._parts = tuple(part for part in (self.mixer, self.mixer_norm, self.ffn, self.ffn_norm) if part is not None)
        for norm in (self.mixer_norm, self.ffn_norm):
            if norm is not None and not hasattr(norm, "add_normed"):
                raise ValueError("this arrangement needs norms that offer add_normed (rmsnorm does)")

    def tensor_specs(self) -> list[TensorSpec]:
        return [spec for part in self._parts for spec in part.tensor_specs()]

    def load(self, tensors: Mapping[str, torch.Tensor]) -> None:
        for part in self._parts:
            part.load(tensors)

    def bytes_streamed(self) -> int:
        return sum(part.bytes_streamed() for part in self._parts)

    def forward(self, residual: torch.Tensor, delta, ctx: StepContext, cache: CacheView):
        if isinstance(delta, kernels.ResidualCopy):
            rows = delta.values
        elif delta is not None:
            raise ValueError("an output-norm block cannot follow a block that leaves a sum to be added")
        elif self.dtype == torch.float32:
            rows = residual
        else:  # the model's first block: the embedding's rows
            rows = ctx.workspace.buffer("residual.copy", residual.shape[0], residual.shape[1], self.dtype)
            kernels.residual_copy(residual, rows)
        rows = self.mixer_norm.add_normed(residual, self.mixer.forward(rows, ctx, cache), ctx)
        if self.ffn is not None:
            if getattr(self.ffn, "weighted_rows", False):
                output = self.ffn.forward(rows, ctx, combine=False)
            else:
                output = self.ffn.forward(rows, ctx)
            rows = self.ffn_norm.add_normed(residual, output, ctx)
        return residual, (None if rows is residual else kernels.ResidualCopy(rows))


@BLOCKS.register("parallel")
class ParallelBlock(Block):
    """``h = norm(x); x += mixer(h) + ffn(h)``: one norm a layer, and both sub-layers read its output.  A layer may have no
    feed-forward.

    The residual is fp32.  The two outputs are handed on unsummed (``kernels.PendingSums``) and the next norm's kernel adds
    them to the residual, in 32-bit, on its way, so the layer's sum costs no kernel of its own; the norm must be one that
    takes two pending sums (``layernorm`` does)."""

    graph_safe = True

    def __init__(self, *, layer: LayerSpec, dtype: torch.dtype, device: str, shared: dict, **_: object) -> None:
        context = dict(dtype=dtype, device=device, shared=shared)
        self.mixer_norm = NORMS.build(layer.mixer_norm, **context)
        self.mixer = MIXERS.build(layer.mixer, **context)
        self.ffn = FEED_FORWARDS.build(layer.ffn, **context) if layer.ffn is not None else None
        if layer.ffn_norm is not None:
            raise ValueError("a parallel layer has one norm; its feed-forward reads the mixer's input")
        self._parts = tuple(part for part in (self.mixer_norm, self.mixer, self.ffn) if part is not None)

    def tensor_specs(self) -> list[TensorSpec]:
        return [spec for part in self._parts for spec in part.tensor_specs()]

    def load(self, tensors: Mapping[str, torch.Tensor]) -> None:
        for part in self._parts:
            part.load(tensors)

    def bytes_streamed(self) -> int:
        return sum(part.bytes_streamed() for part in self._parts)

    def forward(self, residual: torch.Tensor, delta, ctx: StepContext, cache: CacheView):
        normed = self.mixer_norm.apply(residual, delta, ctx)
        mixed = self.mixer.forward(normed, ctx, cache)
        if self.ffn is None:
            return residual, mixed
        return residual, kernels.PendingSums(mixed, self.ffn.forward(normed, ctx))


@BLOCKS.register("gated_residual")
class GatedResidualBlock(Block):
    """``h = norm1(x); x += m * sigmoid(R1 h + b1) * mixer(h);  h = norm2(x); x += m * sigmoid(R2 h + b2) * ffn(h)``: each
    sub-layer's result is gated element by element by a product of what the sub-layer reads, and scaled by one constant
    (``LayerSpec.options``: ``gate_names``, the two gates' tensors, each with a bias ``.b``, and ``residual_mult``).  A layer
    may have no feed-forward.

    The residual is fp32.  A sub-layer's output, its gate's rows and its bias travel on (``kernels.PendingGated``), and the kernel
    of the norm that reads the stream next forms the gate, adds and norms, so a gated sum costs no kernel of its own; a mixture
    hands over its experts' rows before their sum and that kernel adds them too.  A mixer that takes further rows into its own
    input product (``carry_rows``) computes the gate there; elsewhere it is a product of its own."""

    graph_safe = True

    def __init__(self, *, layer: LayerSpec, dtype: torch.dtype, device: str, shared: dict, **_: object) -> None:
        context = dict(dtype=dtype, device=device, shared=shared)
        self.dtype = dtype
        self.gate_names = tuple(layer.options["gate_names"])
        self.mult = float(layer.options.get("residual_mult", 1.0))
        self.size = int(layer.mixer_norm.params["size"])
        self.mixer_norm = NORMS.build(layer.mixer_norm, **context)
        self.mixer = MIXERS.build(layer.mixer, **context)
        self.ffn_norm = NORMS.build(layer.ffn_norm, **context) if layer.ffn is not None else None
        self.ffn = FEED_FORWARDS.build(layer.ffn, **context) if layer.ffn is not None else None
        self._parts = tuple(part for part in (self.mixer_norm, self.mixer, self.ffn_norm, self.ffn) if part is not None)
        self._carried = hasattr(self.mixer, "carry_rows")
        self._gates: list[Optional[torch.Tensor]] = [None, None]  # weights of gates that are products of their own
        self._biases: list[Optional[torch.Tensor]] = [None, None]

    def _sub_layers(self) -> int:
        return 1 if self.ffn is None else 2

    def tensor_specs(self) -> list[TensorSpec]:
        specs = [spec for part in self._parts for spec in part.tensor_specs()]
        for name in self.gate_names[: self._sub_layers()]:
            specs += [TensorSpec(name, (self.size, self.size)), TensorSpec(f"{name}.b", (self.size,), role="vector", init="normal")]
        return specs

    def load(self, tensors: Mapping[str, torch.Tensor]) -> None:
        for index, name in enumerate(self.gate_names[: self._sub_layers()]):
            self._gates[index] = tensors[name].contiguous()
            self._biases[index] = tensors[f"{name}.b"].contiguous()
        if self._carried:
            self.mixer.carry_rows(self._gates[0])
            self._gates[0] = None
        for part in self._parts:
            part.load(tensors)

    def bytes_streamed(self) -> int:
        own = sum(t.numel() * t.element_size() for t in (*self._gates, *self._biases) if t is not None)
        return own + sum(part.bytes_streamed() for part in self._parts)

    def _gate(self, index: int, h: torch.Tensor, ctx: StepContext) -> torch.Tensor:
        rows = ctx.workspace.buffer(f"block.gate{index}", h.shape[0], self.size, self.dtype)
        kernels.linear(h, self._gates[index], None, rows)
        return rows

    def forward(self, residual: torch.Tensor, delta, ctx: StepContext, cache: CacheView):
        normed = self.mixer_norm.apply(residual, delta, ctx)
        gate = None if self._carried else self._gate(0, normed, ctx)
        mixed = self.mixer.forward(normed, ctx, cache)
        pending = kernels.PendingGated(mixed, self.mixer.carried_rows(ctx) if self._carried else gate, self._biases[0], self.mult)
        if self.ffn is None:
            return residual, pending
        normed = self.ffn_norm.apply(residual, pending, ctx)
        gate = self._gate(1, normed, ctx)
        if getattr(self.ffn, "weighted_rows_and_extra", False):
            output = self.ffn.forward(normed, ctx, combine=False)
        else:
            output = self.ffn.forward(normed, ctx)
        return residual, kernels.PendingGated(output, gate, self._biases[1], self.mult)


@BLOCKS.register("sandwich_norm")
class SandwichNormBlock(Block):
    """``x += post1(mixer(pre1(x))); x += post2(ffn(pre2(x)))``: a norm before and a norm after each sub-layer.  A layer
    may have no feed-forward.

    The residual is fp32.  A sub-layer's output is handed on with its post-norm still to be applied
    (``kernels.PendingNormed``), and the kernel of the norm that reads the stream next norms it, adds it to the
    residual and norms the sum, so a sub-layer costs one norm kernel although it has two norms.  The norms must
    offer ``pending`` and take what it returns as ``delta`` (``rmsnorm`` does)."""

    graph_safe = True

    def __init__(self, *, layer: LayerSpec, dtype: torch.dtype, device: str, shared: dict, **_: object) -> None:
        context = dict(dtype=dtype, device=device, shared=shared)
        if layer.mixer_post_norm is None or (layer.ffn is not None and (layer.ffn_norm is None or layer.ffn_post_norm is None)):
            raise ValueError("this arrangement needs a norm before and a norm after each sub-layer")
        self.mixer_norm = NORMS.build(layer.mixer_norm, **context)
        self.mixer = MIXERS.build(layer.mixer, **context)
        self.mixer_post_norm = NORMS.build(layer.mixer_post_norm, **context)
        self.ffn_norm = NORMS.build(layer.ffn_norm, **context) if layer.ffn is not None else None
        self.ffn = FEED_FORWARDS.build(layer.ffn, **context) if layer.ffn is not None else None
        self.ffn_post_norm = NORMS.build(layer.ffn_post_norm, **context) if layer.ffn is not None else None
        self._parts = tuple(part for part in (self.mixer_norm, self.mixer, self.mixer_post_norm, self.ffn_norm, self.ffn, self.ffn_post_norm)
                            if part is not None)
        for norm in (self.mixer_post_norm, self.ffn_post_norm):
            if norm is not None and not hasattr(norm, "pending"):
                raise ValueError("this arrangement needs output norms that offer pending (rmsnorm does)")

    def tensor_specs(self) -> list[TensorSpec]:
        return [spec for part in self._parts for spec in part.tensor_specs()]

    def load(self, tensors: Mapping[str, torch.Tensor]) -> None:
        for part in self._parts:
            part.load(tensors)

    def bytes_streamed(self) -> int:
        return sum(part.bytes_streamed() for part in self._parts)

    def forward(self, residual: torch.Tensor, delta, ctx: StepContext, cache: CacheView):
        normed = self.mixer_norm.apply(residual, delta, ctx)
        pending = self.mixer_post_norm.pending(self.mixer.forward(normed, ctx, cache))
        if self.ffn is None:
            return residual, pending
        normed = self.ffn_norm.apply(residual, pending, ctx)
        return residual, self.ffn_post_norm.pending(self.ffn.forward(normed, ctx))
