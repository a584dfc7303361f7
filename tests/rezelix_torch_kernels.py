"""Plain torch statements of the kernels that Rezelix's parts call beyond those of the other ``*_torch_kernels`` modules, with
the signatures of ``kairyu_b200.kernels``, for CPU runs of the cache manager, the step function, the scheduler and the
command line (32-bit only).  ``install`` puts them all in place of the kernels for one test.  They are test code: the
package has no implementation but its kernels."""

from __future__ import annotations

import torch

import koravik_torch_kernels
from koravik_torch_kernels import embedding_norm
from mapalorn_torch_kernels import diff_attention_generic


def rglru_gates(x, taps, conv_bias, rings, weights_t, gate_bias, rate, a, into, *, row_ids, qo_indptr, positions, state_slots, flag=None):
    tokens, width = x.shape
    parts, n = weights_t.shape[1], weights_t.shape[2]
    for t in range(tokens):
        row, position = int(row_ids[t]), int(positions[t])
        first = int(qo_indptr[row])
        u = conv_bias.clone()
        for back in range(taps.shape[0]):
            if position - back < 0:
                continue
            earlier = x[t - back].float() if t - back >= first else rings[int(state_slots[row]), (position - back) % taps.shape[0]]
            u += taps[taps.shape[0] - 1 - back] * earlier
        sums = torch.einsum("pi,gpio->gpo", u.view(parts, n), weights_t.float()).reshape(2, width) + gate_bias
        r, i = torch.sigmoid(sums[0]), torch.sigmoid(sums[1])
        a[t] = torch.exp(rate * r)
        into[t] = torch.sqrt(-torch.expm1(2.0 * rate * r)) * i * u


def rglru_scan(a, into, x, y, states, rings, n_taps, out, *, qo_indptr, positions, state_slots, segments=None):
    for row in range(qo_indptr.numel() - 1):
        slot = int(state_slots[row])
        for t in range(int(qo_indptr[row]), int(qo_indptr[row + 1])):
            states[slot] = a[t] * states[slot] + into[t]
            out[t] = (states[slot] * torch.nn.functional.gelu(y[t].float(), approximate="tanh")).to(out.dtype)
            if rings is not None:
                rings[slot, int(positions[t]) % n_taps] = x[t].float()


_NAMES = ["embedding_norm", "diff_attention_generic", "rglru_gates", "rglru_scan"]


def install(monkeypatch) -> None:
    import kairyu_b200.kernels as kernels

    koravik_torch_kernels.install(monkeypatch)
    for name in _NAMES:
        monkeypatch.setattr(kernels, name, globals()[name])
