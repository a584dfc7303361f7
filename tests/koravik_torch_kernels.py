"""Plain torch statements of the kernels that Koravik's parts call beyond those of the other ``*_torch_kernels`` modules, with
the signatures of ``kairyu_b200.kernels``, for CPU runs of the cache manager, the step function, the scheduler and the
command line (32-bit only).  ``install`` puts them all in place of the kernels for one test.  They are test code: the
package has no implementation but its kernels."""

from __future__ import annotations

import torch

import tapasun_torch_kernels
from mapalorn_torch_kernels import _place, _turn


def embedding_norm(table, ids, out, *, weight=None, eps=0.0, scale=1.0, origin=None, flag=None):
    rows = table[ids.long()].float() * scale
    if weight is not None:
        rows = rows * torch.rsqrt(rows.pow(2).mean(-1, keepdim=True) + eps) * weight.float()
    out.copy_(rows)
    if origin is not None:
        origin.copy_(rows)


def gated_residual_norm(residual, pending, weight, eps, out, *, rows=None, origin=None):
    picked = rows.long() if rows is not None else slice(None)
    total = residual.clone()
    if pending is not None:
        values = pending.values
        if hasattr(values, "weights"):  # a mixture's rows before their sum
            tokens, top = values.weights.shape
            parts = values.rows.float() if values.at is None else values.rows.float()[values.at.long()]
            summed = (parts.view(tokens, top, -1) * values.weights.unsqueeze(-1)).sum(1)
            values = summed + (values.extra.float() if values.extra is not None else 0.0)
        bias = pending.bias.float() if pending.bias is not None else 0.0
        total = total + pending.mult * torch.sigmoid(pending.gate.float() + bias) * values.float()
        if rows is None:
            residual.copy_(total)
    total = total[picked]
    result = total if weight is None else total * torch.rsqrt(total.pow(2).mean(-1, keepdim=True) + eps) * weight.float()
    if origin is not None:
        result = torch.cat([result, origin[picked]], dim=-1)
    out[: result.shape[0]].copy_(result.to(out.dtype))


def talking_prepare(packed, talk, mixed, *, num_q_heads, num_kv_heads, head_dim, k_offset, v_offset, positions, row_ids, cos=None, sin=None,
                    block_table=None, write_from=None, k_cache=None, v_cache=None, flag=None):
    H, G, D = num_q_heads, num_kv_heads, head_dim
    group = H // G
    for t in range(packed.shape[0]):
        position, row = int(positions[t]), int(row_ids[t])

        def turned(head):
            return _turn(head.float(), cos[position], sin[position], False) if cos is not None else head.float()

        q = torch.stack([turned(packed[t, h * D : (h + 1) * D]) for h in range(H)])
        wide = torch.zeros(H, G, D)
        for h in range(H):
            for g in range(H):
                wide[h, g // group] += talk[h, g] * q[g]
        mixed[t] = wide.reshape(-1).to(mixed.dtype)
        if k_cache is None:
            continue
        place = _place(k_cache, block_table, write_from, row, position)
        if place is None:
            continue
        page, at = place
        for c in range(G):
            k_cache[page, at, c] = turned(packed[t, k_offset + c * D : k_offset + (c + 1) * D]).to(k_cache.dtype)
            v_cache[page, at, c] = packed[t, v_offset + c * D : v_offset + (c + 1) * D]


def diff_attention_generic(q, out, k_cache, v_cache, *, positions, row_ids, block_table, num_q_heads, maps, scale, softcap=0.0, window=0,
                           keep_first=0, lam=0.0, head_norm_eps=None, out_scale=1.0, flag=None, sinks=None, gate=None):
    """One map, without cap, sinks and gate: what this design uses."""
    assert maps == 1 and softcap == 0.0 and sinks is None and gate is None and head_norm_eps is None
    page_size, dim, vdim = k_cache.shape[1], k_cache.shape[3], v_cache.shape[3]
    for t in range(q.shape[0]):
        position, row = int(positions[t]), int(row_ids[t])
        seen = [j for j in range(position + 1) if window <= 0 or position - j < window or j < keep_first]
        places = [(int(block_table[row, j // page_size]), j % page_size) for j in seen]
        assert all(0 < page < k_cache.shape[0] for page, _ in places)
        keys = torch.stack([k_cache[page, at] for page, at in places]).float()
        values = torch.stack([v_cache[page, at] for page, at in places]).float()
        for h in range(num_q_heads):
            s = keys[:, h // (num_q_heads // keys.shape[1])] @ q[t, h * dim : (h + 1) * dim].float() * scale
            a = torch.softmax(s, dim=0) @ values[:, h // (num_q_heads // values.shape[1])]
            out[t, h * vdim : (h + 1) * vdim] = a.to(out.dtype)


_NAMES = ["embedding_norm", "gated_residual_norm", "talking_prepare", "diff_attention_generic"]


def install(monkeypatch) -> None:
    import kairyu_b200.kernels as kernels

    tapasun_torch_kernels.install(monkeypatch)
    for name in _NAMES:
        monkeypatch.setattr(kernels, name, globals()[name])
