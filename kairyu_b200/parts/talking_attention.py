"""Grouped-query attention whose heads' scores are mixed before the softmax ("talking heads"), over the paged cache.

One product gives ``q | k | v`` (``values="keys"``: ``q | k``, a value is the key as projected, before its turn).  Per token::

    the first ``rotary_dim`` columns of every head of q and k turn by the token's position, pairs (i, i + rotary_dim/2)
    s_g(i, j) = q_g(i) . k_c(g)(j) * scale                  c(g) = g // (num_heads / num_kv_heads)
    s_h(i, j) <- sum_g T[h, g] s_g(i, j)                    T: the tensor ``talk``, over ALL the layer's heads
    p_h(i, .) = softmax over the keys i sees: itself and the ``window - 1`` before it (None: all before it), and the
                sequence's first ``keep_first`` tokens
    o_h(i)    = sum_j p_h(i, j) v_c(h)(j), the heads side by side through the output product

The mix is linear in the queries, so it costs no pass over the scores: ``kernels.talking_prepare`` mixes the turned queries
in 32-bit (head h gets one row that spans every key/value head's key, ``num_kv_heads * head_dim`` columns) and attention
is that of heads which share one wide key row a position and take their values from their own key/value head.  Cached per
token and key/value head: the turned key and the value.  bfloat16 of sizes ``kernels.talking_attention_supported`` names runs
on tensor cores (prompt portions in tiles of queries, single tokens with their keys split over blocks); everything else
runs the 32-bit-arithmetic kernel.

Tensors under ``prefix``: ``q``, ``k``, ``o``, ``talk`` [heads, heads], and ``v`` with ``values="projection"``.
``carry_rows`` takes further weight rows into the input product for the block around the mixer (a gate that reads
the same rows); ``carried_rows`` gives their columns of the step."""

from __future__ import annotations

from typing import Any, Mapping, Optional

import torch

from kairyu_b200 import kernels
from kairyu_b200.parts.base import MIXERS, POSITION_ENCODINGS, CacheView, Mixer, PagedKVSpec, PartSpec, StepContext, TensorSpec


@MIXERS.register("talking_attention")
class TalkingAttention(Mixer):
    graph_safe = True

    def __init__(
        self,
        *,
        prefix: str,
        hidden_size: int,
        num_heads: int,
        num_kv_heads: int,
        head_dim: int,
        scale: float,
        position: Optional[PartSpec] = None,
        window: Optional[int] = None,
        keep_first: int = 0,
        values: str = "keys",
        dtype: torch.dtype,
        device: str,
        shared: Optional[dict] = None,
        **_: object,
    ) -> None:
        if num_heads % num_kv_heads:
            raise ValueError(f"{num_heads} query heads are not a multiple of {num_kv_heads} KV heads")
        if values not in ("keys", "projection"):
            raise ValueError(f"values are the 'keys' or a 'projection', not {values!r}")
        self.prefix = prefix
        self.hidden_size = hidden_size
        self.num_heads = num_heads
        self.num_kv_heads = num_kv_heads
        self.head_dim = head_dim
        self.scale = float(scale)
        self.window = window
        self.keep_first = int(keep_first) if window is not None else 0
        self.own_values = values == "projection"
        self.dtype = dtype
        self.device = device
        self.position = None
        if position is not None:
            table = shared if shared is not None else {}
            key = ("position", position)
            if key not in table:  # one table for all layers that ask for the same encoding
                table[key] = POSITION_ENCODINGS.build(position, device=device, dtype=dtype)
            self.position = table[key]
            if self.position.rotary_dim > head_dim:
                raise ValueError(f"{self.position.rotary_dim} rotated columns in a head of {head_dim}")
        self.q_size = num_heads * head_dim
        self.kv_size = num_kv_heads * head_dim
        self.k_offset = self.q_size
        self.v_offset = self.k_offset + (self.kv_size if self.own_values else 0)
        self.carried_offset = self.v_offset + self.kv_size
        self.packed_width = self.carried_offset
        self._carried: Optional[torch.Tensor] = None
        self.w_in: Optional[torch.Tensor] = None  # [q | k | v | carried rows, hidden]
        self.w_o: Optional[torch.Tensor] = None
        self.talk: Optional[torch.Tensor] = None  # fp32: it enters the scores

    # -- weights
    def carry_rows(self, weight: torch.Tensor) -> None:
        """Rows [n, hidden] that the input product computes too; given before ``load``."""
        self._carried = weight
        self.packed_width = self.carried_offset + weight.shape[0]

    def carried_rows(self, ctx: StepContext) -> torch.Tensor:
        return self._packed(ctx)[:, self.carried_offset :]

    def tensor_specs(self) -> list[TensorSpec]:
        p = self.prefix
        specs = [TensorSpec(f"{p}.q", (self.q_size, self.hidden_size)), TensorSpec(f"{p}.k", (self.kv_size, self.hidden_size))]
        if self.own_values:
            specs.append(TensorSpec(f"{p}.v", (self.kv_size, self.hidden_size)))
        return specs + [
            TensorSpec(f"{p}.talk", (self.num_heads, self.num_heads), role="vector", init="normal"),
            TensorSpec(f"{p}.o", (self.hidden_size, self.q_size)),
        ]

    def load(self, tensors: Mapping[str, torch.Tensor]) -> None:
        p = self.prefix
        rows = [tensors[f"{p}.q"], tensors[f"{p}.k"]] + ([tensors[f"{p}.v"]] if self.own_values else [])
        if self._carried is not None:
            rows.append(self._carried)
            self._carried = None  # the packed weight holds it from here on
        self.w_in = torch.cat(rows, dim=0).contiguous()
        self.w_o = tensors[f"{p}.o"].contiguous()
        self.talk = tensors[f"{p}.talk"].float().contiguous()

    def bytes_streamed(self) -> int:
        return sum(t.numel() * t.element_size() for t in (self.w_in, self.w_o, self.talk))

    # -- cache
    def cache_specs(self) -> tuple[Any, ...]:
        return (PagedKVSpec(self.num_kv_heads, self.head_dim, self.window, keep_first=self.keep_first),)

    def _tensor_cores(self) -> bool:
        """bfloat16 and sizes the tensor-core kernels take; float32 and other sizes run the 32-bit-arithmetic kernel."""
        return self.dtype == torch.bfloat16 and kernels.talking_attention_supported(self.num_heads, self.num_kv_heads, self.head_dim)

    def query_tile_sizes(self) -> tuple[int, ...]:
        return (kernels.talking_attention_tile(self.num_heads, self.num_kv_heads),) if self._tensor_cores() else ()

    # -- compute
    def _packed(self, ctx: StepContext) -> torch.Tensor:
        return ctx.workspace.buffer("talk.packed", ctx.num_tokens, self.packed_width, self.dtype)

    def forward(self, x: torch.Tensor, ctx: StepContext, cache: CacheView) -> torch.Tensor:
        tokens = x.shape[0]
        ws = ctx.workspace
        packed = self._packed(ctx)
        kernels.linear(x, self.w_in, None, packed)
        block_table = ctx.block_tables[cache.group]
        cos, sin = self.position.rotary_tables() if self.position is not None else (None, None)
        queries = ws.buffer("talk.queries", tokens, self.num_heads * self.kv_size, self.dtype)
        kernels.talking_prepare(
            packed, self.talk, queries, num_q_heads=self.num_heads, num_kv_heads=self.num_kv_heads, head_dim=self.head_dim, k_offset=self.k_offset,
            v_offset=self.v_offset, positions=ctx.positions, row_ids=ctx.row_ids, cos=cos, sin=sin,
            block_table=block_table if cache.writes else None, write_from=ctx.write_from if cache.writes else None,
            k_cache=cache.k if cache.writes else None, v_cache=cache.v if cache.writes else None, flag=ctx.error_flag,
        )
        mixed = ws.buffer("talk.mixed", tokens, self.q_size, self.dtype)
        constants = dict(num_q_heads=self.num_heads, scale=self.scale, window=self.window or 0, keep_first=self.keep_first, flag=ctx.error_flag)
        if self._tensor_cores() and not ctx.extras.get("force_generic_attention", False):
            kernels.talking_attention(queries, mixed, cache.k, cache.v, ctx=ctx, block_table=block_table, **constants)
        else:
            # a position's keys side by side are one key row that all heads share
            wide_keys = cache.k.view(cache.k.shape[0], cache.k.shape[1], 1, self.kv_size)
            kernels.diff_attention_generic(queries, mixed, wide_keys, cache.v, positions=ctx.positions, row_ids=ctx.row_ids, block_table=block_table,
                                           maps=1, **constants)
        out = ws.buffer("talk.out", tokens, self.hidden_size, self.dtype)
        kernels.linear(mixed, self.w_o, None, out)
        return out
