"""Koravik on the GPU against the plain implementation in ``koravik_plain.py``: every mechanism alone, whole prompts against
token-by-token decoding, portions down to two tokens, unequal requests in one batch over a pool so small that pages are used
again, keys made to stand out far away, at page borders, just inside and outside a window and among the first tokens it keeps,
long decoding, and greedy generation through ``LLM.generate``."""

import types

import numpy as np
import pytest
import torch

import koravik_plain as plain
import traces
from koravik_cases import CASES, attention, config, layer, make_weights, moe, relative_error, write_model

pytestmark = pytest.mark.gpu

# rms of the logits' error over rms of the logits, per position
FP32_BOUND = 1e-4
BF16_BOUND = 5e-2
LENGTHS = [70, 45, 101, 38, 64, 83, 9, 55, 2, 1]


def make_runner(folder, dtype, *, page_size, num_pages, max_requests=4, decode_mode="eager", max_model_len=1024):
    from kairyu_b200.cache import CacheLayout, CacheManager, CacheStorage
    from kairyu_b200.engine.engine import load_model
    from kairyu_b200.engine.runner import ModelRunner

    model, _ = load_model(folder, dtype=dtype, device="cuda")
    layout = CacheLayout.from_slot_specs(model.cache_slot_specs())
    cache = CacheManager(layout, num_pages=num_pages, page_size=page_size, max_requests=max_requests)
    storage = CacheStorage(layout, num_pages=num_pages, page_size=page_size, max_requests=max_requests, dtype=model.dtype, device="cuda")
    return ModelRunner(model, cache, storage, max_model_len=max_model_len, decode_mode=decode_mode, max_graph_batch=max_requests,
                       check_tables=True, debug_poison=True)


def judge(result, expected, dtype, what=""):
    """float32: every position within the bound.  bfloat16: the weights make the softmax pick single keys and the routers choose
    among close scores, so that faults show; rounding to bfloat16 then costs a few per cent at a typical position and much
    more where a close call turns.  A fault moves the median position beyond the bound or many positions far beyond it
    (test_koravik_cpu.py: test_the_bounds_see_each_fault), so the median is held to BF16_BOUND and few positions may be far off."""
    errors = np.array([relative_error(row, expected[name][position]) for (name, position), row in result.items()])
    if str(dtype).endswith("float32"):
        print(f"[koravik] {what} float32: worst {errors.max():.3e} bound {FP32_BOUND:.1e}")
        assert errors.max() < FP32_BOUND, (what, errors.max())
    else:
        far = float((errors >= 3 * BF16_BOUND).mean())
        print(f"[koravik] {what} bfloat16: median {np.median(errors):.3e} worst {errors.max():.3e} far off {far:.3f} bound {BF16_BOUND:.1e}")
        assert np.median(errors) < BF16_BOUND and far <= 0.10, (what, np.median(errors), far)


@pytest.fixture(scope="module", params=list(CASES))
def case(request, tmp_path_factory):
    cfg, seed, page_size = CASES[request.param]
    weights = make_weights(cfg, seed)
    folder = write_model(cfg, weights, tmp_path_factory.mktemp(request.param))
    requests = traces.make_requests(cfg["vocab"], LENGTHS, seed=seed + 100)
    expected = {name: plain.forward(cfg, weights, tokens).numpy() for name, tokens in requests.items()}
    return dict(name=request.param, cfg=cfg, page_size=page_size, weights=weights, folder=folder, requests=requests, expected=expected)


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("decode_mode", ["eager", "cuda_graph"])
def test_every_cut_matches_plain(case, dtype, decode_mode):
    """Whole prompts, tails decoded token by token, portions of changing size and mixed batches, one after the other on one engine
    whose pool holds far less than all requests (pages change hands; pages that went back are overwritten before the next step)."""
    requests = case["requests"]
    cuts = {
        "whole": traces.trace_whole(requests),
        "tail": traces.trace_decode_tail(requests, 32),
        "chunks": traces.trace_chunks(requests),
        "twos": traces.trace_chunks(requests, sizes=(2,)),
        "mixed": traces.trace_mixed(requests, seed=5),
    }
    pool = max(traces.peak_tokens(steps) for steps in cuts.values()) // case["page_size"] + 1
    total = sum(len(t) for t in requests.values())
    assert pool * case["page_size"] < total
    runner = make_runner(case["folder"], dtype, page_size=case["page_size"], num_pages=pool, decode_mode=decode_mode)
    results = {}
    for cut, steps in cuts.items():
        results[cut] = traces.run_in_process(runner, steps)
        assert len(results[cut]) == total
        judge(results[cut], case["expected"], dtype, f"{case['name']} {decode_mode} {cut}")
        assert runner.cache.live_requests == 0
    if decode_mode == "cuda_graph":
        assert runner.counters["graph_replays"] > 0
    if dtype == "float32":
        # no 32-bit sum depends on the batch or on where a prompt was cut
        for cut in ("tail", "chunks", "twos", "mixed"):
            different = [key for key, row in results["whole"].items() if not np.array_equal(row, results[cut][key])]
            assert not different, (cut, different[:12])


MIXERS = {
    "narrow": attention(2, 1, 16, 0.5, window=19, keep=2),
    "no_tensor_cores": attention(3, 3, 24, 0.4, rot=10, window=19, keep=5),
    "bands_by_tma": attention(4, 2, 32, 0.3, rot=16, window=50, keep=17),
    "widest": attention(16, 4, 128, 0.09, window=90, keep=4),
    "as_many_as_heads": attention(8, 8, 64, 0.12, window=40, keep=1),
    "sixteen_a_group": attention(16, 1, 48, 0.15, rot=20, window=33, keep=8),
    "three_a_group": attention(24, 8, 16, 0.25, window=70, keep=3),
    "too_many_heads": attention(40, 8, 16, 0.25, window=70, keep=3),       # the 32-bit-arithmetic kernel
    "too_wide_a_row": attention(10, 10, 64, 0.12, window=60, keep=2),      # the same
    "window_of_one": attention(2, 1, 32, 0.3, window=1),
    "keeps_more_than_the_window": attention(2, 2, 16, 0.3, window=5, keep=70),
    "long_window": attention(4, 4, 64, 0.12, window=131, keep=40),
    "sees_everything": attention(6, 2, 80, 0.1, rot=30),
}


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("kind", list(MIXERS))
def test_one_mixer_alone(kind, dtype, tmp_path):
    """A model of one layer without feed-forward, so that the mixer is all that mixes: a prompt of several windows' length in
    one step, then decoding over more than a window."""
    cfg = config(40, 53, [layer(MIXERS[kind], None)])
    weights = make_weights(cfg, 7)
    folder = write_model(cfg, weights, tmp_path / kind)
    tokens = traces.make_requests(53, [230], seed=3)["r0"]
    expected = {"r0": plain.forward(cfg, weights, tokens).numpy()}
    for page_size in (16, 6):  # pages of no power of two: no TMA copies
        runner = make_runner(folder, dtype, page_size=page_size, num_pages=320 // page_size, decode_mode="cuda_graph")
        result = traces.run_in_process(runner, traces.trace_decode_tail({"r0": tokens}, 90))
        judge(result, expected, dtype, f"{kind} alone, pages of {page_size}")


def _attention_reference(q, k, v, talk, scale, window, keep, positions):
    """[len(positions), heads * dim] by the plain pieces, from whole-sequence q [L, H, D], k and v [L, G, D]."""
    L, H, group = q.shape[0], q.shape[1], q.shape[1] // k.shape[1]
    at = torch.tensor(positions)
    scores = torch.stack([q[at, h] @ k[:, h // group].T for h in range(H)]) * scale
    scores = torch.einsum("hg,gij->hij", talk, scores)
    scores = scores.masked_fill(~plain.visible(L, window or L, keep)[at], float("-inf"))
    p = torch.softmax(scores, dim=-1)
    return torch.cat([p[h] @ v[:, h // group] for h in range(H)], dim=-1)


@pytest.mark.parametrize("variant", ["float32 generic", "bfloat16 generic", "bfloat16 tensor cores"])
@pytest.mark.parametrize("window, keep", [(40, 3), (41, 17), (700, 5), (64, 0), (None, 0)])
@pytest.mark.parametrize("sizes", [(4, 2, 32, 16), (12, 4, 128, 64), (3, 3, 48, 24), (16, 1, 64, 8), (32, 8, 64, 16)])
def test_keys_that_stand_out(variant, window, keep, sizes):
    """The attention kernels alone, from packed rows on, over a 900-token sequence whose pages are shuffled: the queries' mix, the
    page write and the attention.  Among keys whose scores are near zero, one key a query is given a score of 18 in one head
    (which the mix spreads to others): at distances 0 and 1, at a page's last and first place, just inside and just outside the
    window, hundreds of tokens away, and at the first tokens a window keeps and the next ones.  The same queries run as one
    prompt, as a portion that starts in the middle of a page beside single tokens of other lengths, and as single tokens."""
    from kairyu_b200 import kernels
    from kairyu_b200.engine.workspace import Workspace

    dtype = torch.float32 if variant.startswith("float32") else torch.bfloat16
    H, G, D, page = sizes
    L, scale = 900, 0.5
    gen = torch.Generator().manual_seed(11)
    q = torch.randn(L, H, D, generator=gen) * 0.1
    k = torch.randn(L, G, D, generator=gen) * 0.1
    talk = torch.eye(H) + torch.randn(H, H, generator=gen) * 0.3 * H ** -0.5
    edge = window if window is not None else 512
    targets = [("back", d) for d in (0, 1, page - 1, page, page + 1, edge - 1, edge, edge + 1, 600)]
    targets += [("at", p) for p in (0, max(keep - 1, 0), keep, keep + 1)]
    wanted = []
    for index, (kind, amount) in enumerate(targets):
        at = 899 - 9 * index  # the last token first: what lies behind it has never been written
        key = at - amount if kind == "back" else amount
        if key < 0:
            continue
        u = torch.nn.functional.normalize(torch.randn(D, generator=gen), dim=0) * 6.0
        head = index % H
        q[at, head] = u
        k[key, head // (H // G)] = u
        wanted.append(at)
    packed = torch.cat([q.reshape(L, H * D), k.reshape(L, G * D), torch.randn(L, 8, generator=gen)], dim=1).to(dtype)  # other columns behind
    q, k = packed[:, : H * D].double().view(L, H, D), packed[:, H * D : (H + G) * D].double().view(L, G, D)  # what the kernels are given, exactly
    want = _attention_reference(q, k, k, talk.double(), scale, window, keep, wanted)
    if window is not None:  # the stand-out keys matter: a window one shorter or longer, one kept token fewer or more
        for wrong in ((window - 1, keep), (window + 1, keep), (window, keep + 1)) + (((window, keep - 1),) if keep else ()):
            assert (_attention_reference(q, k, k, talk.double(), scale, wrong[0], wrong[1], wanted) - want).abs().max() > 0.2

    pages = torch.randperm(L // page + 1, generator=gen) + 1
    k_cache = torch.full((len(pages) + 1, page, G, D), 3e4, dtype=dtype, device="cuda")  # what no token has written is far off
    v_cache = torch.full((len(pages) + 1, page, G, D), float("nan"), dtype=dtype, device="cuda")
    k_cache[0] = v_cache[0] = 0.0  # the reserved page
    i32 = dict(dtype=torch.int32, device="cuda")
    table = pages.to(torch.int32).cuda()[None, :].contiguous()
    packed = packed.cuda()
    mixed = torch.empty(L, H * G * D, dtype=dtype, device="cuda")
    kernels.talking_prepare(packed, talk.cuda(), mixed, num_q_heads=H, num_kv_heads=G, head_dim=D, k_offset=H * D, v_offset=H * D,
                            positions=torch.arange(L, **i32), row_ids=torch.zeros(L, **i32), block_table=table, write_from=torch.zeros(1, **i32),
                            k_cache=k_cache, v_cache=v_cache)
    bound = 2e-5 if dtype == torch.float32 else 3e-2
    tile = kernels.talking_attention_tile(H, G)
    flag = torch.zeros(1, **i32)
    constants = dict(num_q_heads=H, scale=scale, window=window or 0, keep_first=keep, flag=flag)

    def run(q_rows, positions, row_ids, tables, seq_lens, qo_indptr):
        out = torch.zeros(q_rows.shape[0], H * D, dtype=dtype, device="cuda")
        if variant.endswith("generic"):
            kernels.diff_attention_generic(q_rows, out, k_cache.view(len(pages) + 1, page, 1, G * D), v_cache, positions=positions, row_ids=row_ids,
                                           block_table=tables, maps=1, **constants)
            return out
        rows = len(seq_lens)
        counts = [qo_indptr[r + 1] - qo_indptr[r] for r in range(rows)]
        tile_rows = [r for r in range(rows) if counts[r] > 1 for _ in range(0, counts[r], tile)]
        tile_starts = [s for r in range(rows) if counts[r] > 1 for s in range(0, counts[r], tile)]
        single = [r for r in range(rows) if counts[r] == 1]
        ctx = types.SimpleNamespace(
            qo_indptr=torch.tensor(qo_indptr, **i32), seq_lens=torch.tensor(seq_lens, **i32),
            tiles={tile: (len(tile_rows), torch.tensor(tile_rows or [0], **i32), torch.tensor(tile_starts or [0], **i32))},
            num_decode_rows=len(single), decode_rows=torch.tensor(single or [0], **i32),
            decode_tokens=torch.tensor([qo_indptr[r] for r in single] or [0], **i32), workspace=Workspace("cuda"), max_seq_len=max(seq_lens),
        )
        kernels.talking_attention(q_rows, out, k_cache, v_cache, ctx=ctx, block_table=tables, **constants)
        assert int(flag) == 0
        return out

    def off(got, places):
        return (got.double().cpu() - want[places]).abs().max()

    everyone = list(range(len(wanted)))
    got = run(mixed, torch.arange(L, **i32), torch.zeros(L, **i32), table, [L], [0, L])
    assert off(got[wanted], everyone) < bound
    # a portion that starts in the middle of a page, of a window and of a tile, beside single tokens of other lengths; pages
    # that no query of theirs can see are gone from their tables
    start = 813
    rows_q = torch.cat([mixed[start:], mixed[wanted]])
    positions = torch.tensor(list(range(start, L)) + wanted, **i32)
    row_ids = torch.tensor([0] * (L - start) + list(range(1, len(wanted) + 1)), **i32)
    tables = table.repeat(len(wanted) + 1, 1).contiguous()
    for r, oldest in enumerate([start] + wanted):
        if window is not None:
            tables[r, -(-keep // page) : max(oldest - window + 1, 0) // page] = -1
    indptr = [0, L - start] + [L - start + n + 1 for n in range(len(wanted))]
    got = run(rows_q, positions, row_ids, tables, [L] + [at + 1 for at in wanted], indptr)
    inside = [n for n, at in enumerate(wanted) if at >= start]
    assert off(got[[wanted[n] - start for n in inside]], inside) < bound
    assert off(got[L - start :], everyone) < bound
    # every token of a short sequence on its own: few keys, the kept tokens before the window has passed them
    few = list(range(0, min(70, L)))
    want_few = _attention_reference(q[:70], k[:70], k[:70], talk.double(), scale, window, keep, few)
    got = run(mixed[:70], torch.tensor(few, **i32), torch.tensor(few, **i32), table.repeat(70, 1).contiguous(), [at + 1 for at in few], list(range(71)))
    assert (got.double().cpu() - want_few).abs().max() < bound


def _step_context(tokens, dtype):
    from kairyu_b200.engine.workspace import Workspace
    from kairyu_b200.parts import StepContext

    return StepContext(num_tokens=tokens, num_rows=1, dtype=dtype, token_ids=None, positions=None, row_ids=None, qo_indptr=None, seq_lens=None,
                       write_from=None, state_slots=None, block_tables={}, host_qo_indptr=(), host_seq_lens=(), workspace=Workspace("cuda"))


@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("sizes", [
    # width, experts, top, ff, shared ff (None: no shared expert), tokens
    (40, 5, 3, 24, 16, 33), (64, 6, 1, 16, 64, 3), (72, 4, 4, 40, None, 16), (136, 3, 2, 200, 8, 11), (24, 1, 1, 70, 70, 130),
    (96, 16, 1, 96, 96, 700), (50, 2, 2, 18, 10, 300), (200, 40, 5, 72, 24, 8),
])
def test_mixture_alone(sizes, dtype):
    """The mixture by itself against the plain one, on every product path (few pairs an expert, the library's grouped product,
    the package's grouped kernels): relu squared without a gate, weights divided by the chosen scores' sum, the shared expert;
    and the rows handed on before their sum."""
    from kairyu_b200.parts import FEED_FORWARDS, PartSpec

    width, experts, top, ff, shared, tokens = sizes
    mlp = moe(experts, top, ff, shared=shared)
    weights = make_weights(config(width, 11, [layer(attention(1, 1, 8, 1.0), mlp)]), 3)
    x = torch.randn(tokens, width, generator=torch.Generator().manual_seed(9)).to(torch.bfloat16).float()
    part = FEED_FORWARDS.build(PartSpec(
        "moe", prefix="l0.mlp", hidden_size=width, intermediate_size=ff, num_experts=experts, top=top, routing="scores", score_function="sigmoid",
        correction=False, renormalise=True, router_bias=False, activation="relu2",
        shared_expert=dict(intermediate_size=shared) if shared is not None else None), dtype=dtype, device="cuda")
    part.load({n: t.to(dtype).cuda() for n, t in weights.items() if n.startswith("l0.mlp")})
    w = plain.sub(weights, "l0.mlp", torch.float64)
    want = plain.expert_mixture(x.double(), w, mlp)
    rows = x.to(device="cuda", dtype=dtype)
    got = part.forward(rows, _step_context(tokens, dtype)).float().cpu().double()
    handed = part.forward(rows, _step_context(tokens, dtype), combine=False)
    parts = handed.rows.double() if handed.at is None else handed.rows.double()[handed.at.long()]
    summed = (parts.view(tokens, top, width) * handed.weights.double().unsqueeze(-1)).sum(1)
    assert (handed.extra is None) == (shared is None)
    summed = (summed + (handed.extra.double() if handed.extra is not None else 0.0)).cpu()
    assert (handed.weights.sum(1) - 1.0).abs().max() < 1e-5
    bound = 1e-5 if dtype == torch.float32 else 3e-2
    scores = torch.sigmoid(x.double() @ w["router"].T)
    clear = torch.ones(tokens, dtype=torch.bool)
    if dtype == torch.bfloat16 and top < experts:  # bfloat16 may turn a close call between two experts: those tokens aside
        ranked = scores.sort(dim=1, descending=True).values
        clear = (ranked[:, top - 1] - ranked[:, top]) > 0.02
        assert clear.float().mean() > 0.3
    assert (got - want)[clear].abs().max() < bound * want.abs().max()
    assert (summed - want)[clear].abs().max() < bound * want.abs().max()


def test_route_weights_are_shares_of_the_chosen_scores():
    """The router kernel: choices one by one, ties to the lower index, weights that sum to one also where every score is tiny."""
    from kairyu_b200 import kernels

    g = torch.Generator().manual_seed(2)
    logits = torch.randn(60, 13, generator=g) * 3
    logits[7] = 0.25          # all equal
    logits[8] = -60.0         # scores near 1e-26: the sum's guard weighs in
    logits[8, 4] = -59.0
    for top in (1, 2, 13):
        ids = torch.empty(60, top, dtype=torch.int32, device="cuda")
        weights = torch.empty(60, top, device="cuda")
        kernels.moe_route_scores(logits.cuda(), None, top, ids, weights, score="sigmoid", renormalise=True)
        scores = torch.sigmoid(logits.double())
        for t in range(60):
            chosen = sorted(range(13), key=lambda e: (-float(logits[t, e]), e))[:top]
            assert ids[t].tolist() == chosen
            share = scores[t, chosen] / (scores[t, chosen].sum() + 1e-20)
            assert (weights[t].double().cpu() - share).abs().max() < 1e-6


@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("width", [50, 72, 1024, 2056, 5000])
def test_gated_sum_and_norm(width, dtype):
    """The kernel behind every sub-layer: plain rows and a mixture's rows before their sum, with and without an always-on expert's,
    the gate a view into wider rows, bias of either type, all rows and listed ones, with a norm, without, and with the
    embedding output's rows behind."""
    from kairyu_b200 import kernels

    g = torch.Generator().manual_seed(4)
    tokens, top = 21, 3
    x = torch.randn(tokens, width, generator=g) * 3
    origin = torch.randn(tokens, width, generator=g)
    y = torch.randn(tokens, width, generator=g).to(dtype)
    gate_rows = (torch.randn(tokens, width + 24, generator=g) * 2).to(dtype)
    gate = gate_rows[:, 24:]
    bias = torch.randn(width, generator=g).to(torch.bfloat16)
    weight = (1 + 0.2 * torch.randn(width, generator=g)).to(torch.bfloat16)
    parts = torch.randn(tokens * top, width, generator=g)
    mix = torch.rand(tokens, top, generator=g)
    at = torch.randperm(tokens * top, generator=g).to(torch.int32)
    extra = torch.randn(tokens, width, generator=g).to(dtype)
    factor = 0.6 * torch.sigmoid(gate.double() + bias.double())
    tolerance = 2e-5 if dtype == torch.float32 else 0.05

    def values(kind):
        if kind == "plain":
            return y.cuda(), y.double()
        rows = parts.to(dtype) if kind == "mixture" else parts
        total = (rows.double()[at.long()].view(tokens, top, width) * mix.double().unsqueeze(-1)).sum(1)
        if kind == "mixture":
            return kernels.WeightedRows(rows.cuda(), mix.cuda(), at.cuda(), extra.cuda()), total + extra.double()
        unsorted = (rows.double().view(tokens, top, width) * mix.double().unsqueeze(-1)).sum(1)
        return kernels.WeightedRows(rows.cuda(), mix.cuda()), unsorted

    for kind in ("plain", "mixture", "mixture in order"):
        given, summed = values(kind)
        for held in (torch.float32, dtype):  # the bias and the weight in 32-bit, and in the activations' type
            pending = kernels.PendingGated(given, gate_rows.cuda()[:, 24:], bias.to(held).cuda(), 0.6)
            residual = x.clone().cuda()
            out = torch.empty(tokens, width, dtype=dtype, device="cuda")
            kernels.gated_residual_norm(residual, pending, weight.to(held).cuda(), 1e-5, out)
            total = x.double() + factor * summed
            assert (residual.cpu().double() - total).abs().max() < 2e-5  # the sums are kept in 32-bit
            assert (out.cpu().double() - plain.rms_norm(total, weight.double(), 1e-5)).abs().max() < tolerance
            rows = torch.tensor([5, 0, 20], dtype=torch.int32, device="cuda")
            few = torch.empty(3, width, dtype=dtype, device="cuda")
            untouched = x.clone().cuda()
            kernels.gated_residual_norm(untouched, pending, weight.to(held).cuda(), 1e-5, few, rows=rows)
            assert torch.equal(few, out[rows.long()]) and torch.equal(untouched.cpu(), x)
        both = torch.empty(tokens, 2 * width, dtype=dtype, device="cuda")
        residual = x.clone().cuda()
        kernels.gated_residual_norm(residual, pending, None, 0.0, both, origin=origin.cuda())
        assert torch.equal(both[:, width:].cpu(), origin.to(dtype))
        assert (both[:, :width].cpu().double() - total).abs().max() < tolerance * 3
    both = torch.empty(tokens, 2 * width, dtype=dtype, device="cuda")
    kernels.gated_residual_norm(x.cuda(), None, None, 0.0, both, origin=origin.cuda())  # nothing to add: the embedding's own pass
    assert torch.equal(both.cpu(), torch.cat([x, origin], dim=1).to(dtype))


@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
def test_embedding_norm_and_prepare(dtype):
    """The gather with its norm and second copy; the queries' turn and mix and the page write, in every access width, for rows that
    write all, some and none of their positions."""
    from kairyu_b200 import kernels

    g = torch.Generator().manual_seed(6)
    table = torch.randn(29, 44, generator=g).to(dtype)
    ids = torch.tensor([3, 28, 0, 3], dtype=torch.int32)
    weight = (1 + 0.2 * torch.randn(44, generator=g)).to(torch.bfloat16)
    out, origin = torch.empty(4, 44, device="cuda"), torch.empty(4, 44, device="cuda")
    kernels.embedding_norm(table.cuda(), ids.cuda(), out, weight=weight.to(dtype).cuda(), eps=1e-5, origin=origin)
    assert (out.cpu().double() - plain.rms_norm(table.double()[ids.long()], weight.double(), 1e-5)).abs().max() < 1e-5 and torch.equal(out, origin)
    kernels.embedding_norm(table.cuda(), ids.cuda(), out, origin=origin)
    assert torch.equal(out.cpu(), table.float()[ids.long()]) and torch.equal(out, origin)

    page, tokens = 8, 37
    block_table = torch.tensor([[3, 1, 7, 5, 2, -1], [4, 6, 8, -1, -1, -1]], dtype=torch.int32, device="cuda")
    row_ids = torch.tensor([0] * 30 + [1] * 7, dtype=torch.int32, device="cuda")
    where = torch.tensor(list(range(5, 35)) + list(range(11, 18)), dtype=torch.int32, device="cuda")
    write_from = torch.tensor([8, 0], dtype=torch.int32, device="cuda")  # row 0 only reads its first page
    for H, G, D, rot, spare, own_values in ((3, 1, 20, 8, 5, False), (4, 4, 16, 16, 8, False), (6, 3, 24, 16, 16, True), (20, 2, 32, 32, 0, False),
                                            (8, 2, 64, 32, 8, False), (8, 1, 40, 16, 24, True), (5, 5, 12, 2, 0, True)):
        k_off = H * D
        v_off = k_off + (G * D if own_values else 0)
        packed = torch.randn(tokens, v_off + G * D + spare, generator=g).to(dtype)
        talk = torch.randn(H, H, generator=g)
        rate = torch.tensor([100.0 ** (-2.0 * i / rot) for i in range(rot // 2)], dtype=torch.float64)
        angles = torch.arange(64, dtype=torch.float64)[:, None] * rate[None]
        k_cache = torch.zeros(9, page, G, D, dtype=dtype, device="cuda")
        v_cache = torch.zeros_like(k_cache)
        mixed = torch.empty(tokens, H * G * D, dtype=dtype, device="cuda")
        kernels.talking_prepare(packed.cuda(), talk.cuda(), mixed, num_q_heads=H, num_kv_heads=G, head_dim=D, k_offset=k_off, v_offset=v_off,
                                positions=where, row_ids=row_ids, cos=angles.cos().float().cuda(), sin=angles.sin().float().cuda(),
                                block_table=block_table, write_from=write_from, k_cache=k_cache, v_cache=v_cache)
        s = packed.double()
        q = plain.rotate_halves(s[:, :k_off].view(tokens, H, D), where.cpu(), rot, 100.0)
        k = plain.rotate_halves(s[:, k_off : k_off + G * D].view(tokens, G, D), where.cpu(), rot, 100.0)
        wide = torch.stack([torch.stack([sum(float(talk[h, a]) * q[:, a] for a in range(c * (H // G), (c + 1) * (H // G))) for c in range(G)], 1) for h in range(H)], 1)
        want = wide.reshape(tokens, -1)
        tolerance = 2e-5 if dtype == torch.float32 else 0.01
        assert (mixed.cpu().double() - want).abs().max() < tolerance * max(1.0, float(want.abs().max()))
        for t in range(tokens):
            position, row = int(where[t]), int(row_ids[t])
            slot = (int(block_table[row, position // page]), position % page)
            if position >= int(write_from[row]):
                assert (k_cache[slot].cpu().double() - k[t]).abs().max() < (2e-5 if dtype == torch.float32 else 0.03)
                assert torch.equal(v_cache[slot].flatten().cpu(), packed[t, v_off : v_off + G * D])
            else:
                assert not k_cache[slot].any() and not v_cache[slot].any()


def test_long_decoding(tmp_path):
    """Six hundred tokens decoded one by one through graphs, windows passing over decoded tokens and pages changing hands, beside a
    second request that starts and ends meanwhile, in both modes."""
    cfg = config(40, 53, [layer(attention(4, 2, 32, 0.3, rot=16, window=90, keep=5), moe(4, 2, 16, shared=8)),
                          layer(attention(4, 1, 16, 0.3, window=200, keep=21), None)], loop=(0, 2, 2))
    weights = make_weights(cfg, 8)
    folder = write_model(cfg, weights, tmp_path / "m")
    tokens = traces.make_requests(53, [640, 50], seed=6)
    expected = {name: plain.forward(cfg, weights, t).numpy() for name, t in tokens.items()}
    long, short = tokens["r0"], tokens["r1"]
    steps = [{"step": 0, "entries": [{"id": "r0", "tokens": long[:40], "want": list(range(40))}], "end": []}]
    for n in range(40, 640):
        entries = [{"id": "r0", "tokens": [long[n]], "want": [0]}]
        if n == 300:
            entries.append({"id": "r1", "tokens": short[:20], "want": list(range(20))})
        if 300 < n <= 330:
            entries.append({"id": "r1", "tokens": [short[19 + n - 300]], "want": [0]})
        steps.append({"step": len(steps), "entries": entries, "end": ["r1"] if n == 330 else (["r0"] if n == 639 else [])})
    for dtype in ("float32", "bfloat16"):
        runner = make_runner(folder, dtype, page_size=16, num_pages=48, decode_mode="cuda_graph", max_requests=2)
        judge(traces.run_in_process(runner, steps), expected, dtype, "long decoding")
        runner.cache.check()


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_greedy_generation_through_the_engine(case, dtype):
    """``LLM.generate`` with a token budget that cuts the prompts into portions and batches them with decoding requests; greedy
    tokens against the plain model's own greedy continuation."""
    from kairyu_b200.entrypoints.llm import LLM
    from kairyu_b200.entrypoints.prompt import TokensPrompt
    from kairyu_b200.sampling.params import SamplingParams

    cfg, weights = case["cfg"], case["weights"]
    prompts = [tokens for tokens in list(case["requests"].values())[:6]]
    new = 12
    llm = LLM(model=str(case["folder"]), dtype=dtype, num_pages=64 * 16 // case["page_size"], page_size=case["page_size"], max_num_batched_tokens=24,
              max_num_seqs=4, max_model_len=256)
    outputs = llm.generate([TokensPrompt(prompt_token_ids=tokens) for tokens in prompts],
                           SamplingParams(temperature=0.0, max_tokens=new, ignore_eos=True), use_tqdm=False)
    for tokens, output in zip(prompts, outputs):
        got = list(output.outputs[0].token_ids)
        assert len(got) == new
        # teacher-forced: at every step the engine's choice is (nearly) the plain model's best given the engine's own history
        logits = plain.forward(cfg, weights, list(tokens) + got).numpy()
        close = []
        for step, token in enumerate(got):
            row = logits[len(tokens) - 1 + step]
            close.append((row.max() - row[token]) / row.std())
        if dtype == "float32":
            assert max(close) <= 1e-4, close
        else:  # bfloat16 may turn a close call: most steps agree
            assert np.mean(np.array(close) <= 0.15) >= 0.8, close


def test_trace_program(case, tmp_path):
    """The same through ``bin/trace_run``: a pool for the trace's peak."""
    steps = traces.trace_mixed(case["requests"], seed=9)
    result = traces.run_program(case["folder"], tmp_path / "out", steps, dtype="float32", max_tokens=traces.peak_tokens(steps), vocab=case["cfg"]["vocab"],
                                extra=["--page-size", str(case["page_size"])])
    worst = max(relative_error(row, case["expected"][name][position]) for (name, position), row in result.items())
    assert worst < FP32_BOUND
