"""A recurrent block around a real-gated linear recurrent unit (the block of De et al., "Griffin: Mixing Gated Linear Recurrences
with Local Attention for Efficient Language Models").

Two branches of ``width`` columns come from one product with biases, ``y | x``; x passes a causal convolution over time per channel
(``conv_taps`` taps, the last one the current token's, zeros before the start, with a bias, no activation), u.  u is cut into
``parts`` equal parts of ``width / parts`` columns, and per channel one number S (fp32) is carried from token to token::

    r  = sigmoid(ra[b] u_b + ra.b[b])      i = sigmoid(ri[b] u_b + ri.b[b])       a square matrix a part b
    la = -8 r softplus(lam)                a = exp(la)
    S  <- a S + sqrt(1 - a^2) i u          from S = 0, the first token like every other
    out = W_o (S * gelu(y))                gelu in its tanh form

What a request keeps between steps is S and the convolution's last inputs: two per-request state tensors, no pages.  The inputs
are kept as a ring of ``conv_taps`` rows (row p % taps holds position p's), so that single tokens write a row no other block of
their kernel reads.  Everything between the input product and the output product is 32-bit.  The kernels are in ``csrc/rglru.cu``.

Tensors under ``prefix``: ``y``, ``x`` [width, hidden], each with ``.b``, ``conv`` [width, taps], ``conv.b``, ``ra``, ``ri`` [parts,
width/parts, width/parts] as [out, in], each with ``.b`` [parts, width/parts], ``lam`` [width], ``o`` [hidden, width].
"""

from __future__ import annotations

from typing import Any, Mapping, Optional

import torch

from kairyu_b200 import kernels
from kairyu_b200.parts.base import MIXERS, CacheView, Mixer, StateSpec, StepContext, TensorSpec

DECAY_SCALE = 8.0  # log a = -DECAY_SCALE * r * softplus(lam)


@MIXERS.register("rglru")
class RealGatedLRU(Mixer):
    graph_safe = True

    def __init__(
        self,
        *,
        prefix: str,
        hidden_size: int,
        width: int,
        parts: int,
        conv_taps: int,
        dtype: torch.dtype,
        device: str,
        **_: object,
    ) -> None:
        if width % parts:
            raise ValueError(f"{width} columns do not split into {parts} equal parts")
        self.prefix = prefix
        self.hidden_size = hidden_size
        self.width = width
        self.parts = parts
        self.conv_taps = conv_taps
        self.dtype = dtype
        self.w_in: Optional[torch.Tensor] = None        # [y | x rows, hidden]
        self.b_in: Optional[torch.Tensor] = None
        self.taps: Optional[torch.Tensor] = None        # [taps, width]
        self.conv_bias: Optional[torch.Tensor] = None
        self.gates: Optional[torch.Tensor] = None       # bfloat16: [2, parts, np, np] as [gate, part, out, in], n rounded up to 16
        self.gates_t: Optional[torch.Tensor] = None     # float32: [2, parts, n, n] as [gate, part, in, out]
        self.gate_bias: Optional[torch.Tensor] = None   # [2, width]
        self.rate: Optional[torch.Tensor] = None        # [width]: -8 softplus(lam)
        self.w_o: Optional[torch.Tensor] = None

    def tensor_specs(self) -> list[TensorSpec]:
        p, h, w, n = self.prefix, self.hidden_size, self.width, self.width // self.parts
        specs = []
        for name in ("y", "x"):
            specs += [TensorSpec(f"{p}.{name}", (w, h)), TensorSpec(f"{p}.{name}.b", (w,), role="bias", init="normal")]
        specs += [TensorSpec(f"{p}.conv", (w, self.conv_taps), role="vector", init="taps"), TensorSpec(f"{p}.conv.b", (w,), role="vector", init="normal")]
        for name in ("ra", "ri"):
            specs += [TensorSpec(f"{p}.{name}", (self.parts, n, n)), TensorSpec(f"{p}.{name}.b", (self.parts, n), role="vector", init="normal")]
        return specs + [TensorSpec(f"{p}.lam", (w,), role="vector", init="normal"), TensorSpec(f"{p}.o", (h, w))]

    def load(self, tensors: Mapping[str, torch.Tensor]) -> None:
        p = self.prefix
        self.w_in = torch.cat([tensors[f"{p}.y"], tensors[f"{p}.x"]], dim=0).contiguous()
        self.b_in = torch.cat([tensors[f"{p}.y.b"], tensors[f"{p}.x.b"]], dim=0).contiguous()
        # what enters the recurrence is 32-bit whatever the compute dtype
        self.taps = tensors[f"{p}.conv"].float().t().contiguous()
        self.conv_bias = tensors[f"{p}.conv.b"].float().contiguous()
        gates = torch.stack([tensors[f"{p}.ra"], tensors[f"{p}.ri"]])
        n = self.width // self.parts
        if self.dtype == torch.bfloat16:
            padded = kernels.rglru_padded(n)
            self.gates = torch.zeros((2, self.parts, padded, padded), dtype=gates.dtype, device=gates.device)
            self.gates[:, :, :n, :n] = gates
        else:
            self.gates_t = gates.transpose(2, 3).contiguous()
        self.gate_bias = torch.stack([tensors[f"{p}.ra.b"].float().reshape(-1), tensors[f"{p}.ri.b"].float().reshape(-1)]).contiguous()
        lam = tensors[f"{p}.lam"].double()
        self.rate = (-DECAY_SCALE * torch.nn.functional.softplus(lam, threshold=40.0)).float().contiguous()
        self.w_o = tensors[f"{p}.o"].contiguous()

    def bytes_streamed(self) -> int:
        gates = self.gates if self.gates is not None else self.gates_t
        held = (self.w_in, self.b_in, self.taps, self.conv_bias, gates, self.gate_bias, self.rate, self.w_o)
        return sum(t.numel() * t.element_size() for t in held)

    def cache_specs(self) -> tuple[Any, ...]:
        specs = [StateSpec((self.width,), "float32")]
        if self.conv_taps > 1:
            specs.append(StateSpec((self.conv_taps, self.width), "float32"))
        return tuple(specs)

    def fusable_norm(self, tokens: int) -> bool:
        """Whether the input and the output product can take the norms around them into their epilogues."""
        return kernels.fused_norm_shapes_ok(tokens, self.hidden_size, self.width)

    def forward(self, x, ctx: StepContext, cache: CacheView, fold=None):
        """``x``: rows, or a ``kernels.PreNormed``; ``fold`` (a ``kernels.ResidualNorm``): the output
        product adds its result to the residual and returns the ``PreNormed`` for the next norm."""
        tokens = x.shape[0]
        ws = ctx.workspace
        states = cache.state if isinstance(cache.state, (list, tuple)) else [cache.state]
        memory = states[0]
        rings = states[1] if self.conv_taps > 1 else None
        packed = ws.buffer("rglru.packed", tokens, 2 * self.width, self.dtype)
        kernels.linear(x, self.w_in, self.b_in, packed)
        y_branch, x_branch = packed[:, : self.width], packed[:, self.width :]
        mixed = ws.buffer("rglru.mixed", tokens, self.width, self.dtype)
        slots = dict(row_ids=ctx.row_ids, state_slots=ctx.state_slots)
        step = dict(slots, qo_indptr=ctx.qo_indptr, positions=ctx.positions)
        single = tokens == ctx.num_rows and tokens <= kernels.RGLRU_STEP_MAX_TOKENS  # every row carries one token
        if self.gates is not None:
            wide = self.parts * self.gates.shape[2]
            hi, lo = (ws.buffer(f"rglru.{name}", tokens, wide, self.dtype) for name in ("hi", "lo"))
            kernels.rglru_convolve(x_branch, self.taps, self.conv_bias, rings, hi, lo, self.parts, update_rings=single, flag=ctx.error_flag, **step)
            if single:
                kernels.rglru_step(hi, lo, y_branch, memory, self.gates, self.gate_bias, self.rate, mixed, flag=ctx.error_flag, **slots)
        if self.gates is None or not single:
            a = ws.buffer("rglru.a", tokens, self.width, torch.float32)
            into = ws.buffer("rglru.into", tokens, self.width, torch.float32)
            if self.gates is not None:
                kernels.rglru_gates_tc5(hi, lo, self.gates, self.gate_bias, self.rate, a, into, flag=ctx.error_flag)
            else:
                kernels.rglru_gates(x_branch, self.taps, self.conv_bias, rings, self.gates_t, self.gate_bias, self.rate, a, into, flag=ctx.error_flag, **step)
            # 32-bit mode walks a request's tokens one by one, so that a result does not depend on where a prompt was cut
            kernels.rglru_scan(a, into, x_branch, y_branch, memory, rings, self.conv_taps, mixed, qo_indptr=ctx.qo_indptr, positions=ctx.positions,
                               state_slots=ctx.state_slots, segments=(1, 1) if self.dtype == torch.float32 else None)
        if fold is not None:
            kernels.linear(mixed, self.w_o, None, None, fold=fold)
            return fold.result()
        out = ws.buffer("rglru.out", tokens, self.hidden_size, self.dtype)
        kernels.linear(mixed, self.w_o, None, out)
        return out
