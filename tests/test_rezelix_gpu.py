"""Rezelix on the GPU against the plain implementation in ``rezelix_plain.py``: every mechanism alone, whole prompts against
token-by-token decoding, portions down to two tokens, unequal requests in one batch over a pool and state slots so few that
they are used again, keys made to stand out far away and at page borders, long decoding, and greedy generation through
``LLM.generate``."""

import types

import numpy as np
import pytest
import torch

import rezelix_plain as plain
import traces
from rezelix_cases import CASES, attention, config, latent, layer, make_weights, relative_error, rglru, rot, write_model

pytestmark = pytest.mark.gpu

# rms of the logits' error over rms of the logits, per position
FP32_BOUND = 1e-4
BF16_BOUND = 4e-2
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
    """float32: every position within the bound.  bfloat16: the weights make the softmax pick single keys, so that faults show; rounding
    then costs a few per cent at a typical position and more where a close call turns.  A fault moves the median beyond the
    bound (test_rezelix_cpu.py: test_the_bounds_see_each_fault), so the median is held to it and few positions may be far off."""
    errors = np.array([relative_error(row, expected[name][position]) for (name, position), row in result.items()])
    if str(dtype).endswith("float32"):
        print(f"[rezelix] {what} float32: worst {errors.max():.3e} bound {FP32_BOUND:.1e}")
        assert errors.max() < FP32_BOUND, (what, errors.max())
    else:
        far = float((errors >= 3 * BF16_BOUND).mean())
        print(f"[rezelix] {what} bfloat16: median {np.median(errors):.3e} worst {errors.max():.3e} far off {far:.3f} bound {BF16_BOUND:.1e}")
        assert np.median(errors) < BF16_BOUND and far <= 0.05, (what, np.median(errors), far)


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
    whose pool holds far less than all requests (pages and state slots change hands; pages that went back are overwritten before
    the next step)."""
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


YARN = (6.0, 128, 16.0, 1.0)
MIXERS = {
    "attention heads of 16, cap by polynomial": attention(4, 2, 16, 0.6, rot(8, 500.0, YARN), softcap=25.0),
    "attention heads of 32, cap by exponential": attention(3, 1, 32, 0.45, rot(32), softcap=4.0),
    "attention heads of 64": attention(4, 4, 64, 0.3, rot(64, 3000.0, YARN), softcap=60.0),
    "attention heads of 64, a strong cap": attention(4, 1, 64, 0.4, rot(16), softcap=2.0),
    "attention heads of 128": attention(2, 1, 128, 0.22, rot(128, 1e5, (32.0, 64, 32.0, 1.0)), softcap=70.0),
    "attention heads of 128, a strong cap": attention(4, 2, 128, 0.22, rot(64), softcap=6.0),
    "attention heads of 96": attention(6, 3, 96, 0.25, rot(48, 700.0, YARN), softcap=20.0),
    "attention heads of 256": attention(2, 2, 256, 0.15, rot(64), softcap=9.0),
    "attention without a cap": attention(4, 2, 32, 0.45, rot(32, 500.0, YARN)),
    "attention without positions": attention(4, 2, 64, 0.3, None, softcap=8.0),
    "attention odd": attention(3, 3, 10, 0.7, rot(4, 60.0, YARN), softcap=3.0),
    "attention twenty heads over one": attention(20, 1, 16, 0.6, rot(16), softcap=5.0),
    "latent row of 32": latent(4, 16, 8, 16, 24, 0.5, 500.0, YARN),
    "latent row of 64": latent(3, 24, 16, 20, 48, 0.4, 1000.0),
    "latent row of 128": latent(2, 40, 32, 32, 96, 0.3, 1000.0, YARN),
    "latent row of 256": latent(2, 64, 64, 64, 192, 0.25, 1e4, (8.0, 96, 32.0, 1.0)),
    "latent row of 300": latent(2, 32, 44, 16, 256, 0.3),
    "latent odd": latent(5, 7, 2, 9, 11, 0.7, 40.0, YARN),
    "latent seventeen heads": latent(17, 16, 16, 8, 32, 0.4),
    "unit of one part of 16": rglru(16, 1, 4),
    "unit of eight parts of 8": rglru(64, 8, 3),
    "unit wider than the model": rglru(256, 2, 4),
    "unit of parts of 80": rglru(240, 3, 2),
    "unit of parts of 21": rglru(63, 3, 4),
    "unit of one part of 300": rglru(300, 1, 5),
    "unit with one tap": rglru(40, 5, 1),
}


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("kind", list(MIXERS))
def test_one_mixer_alone(kind, dtype, tmp_path):
    """A model of one layer without feed-forward, so that the mixer is all that mixes: a prompt of 230 tokens in one step, then 90
    tokens decoded one by one through a graph."""
    cfg = config(40, 53, [layer(MIXERS[kind], None)])
    weights = make_weights(cfg, 7)
    folder = write_model(cfg, weights, tmp_path / "m")
    tokens = traces.make_requests(53, [320], seed=3)["r0"]
    expected = {"r0": plain.forward(cfg, weights, tokens).numpy()}
    runner = make_runner(folder, dtype, page_size=16, num_pages=24, decode_mode="cuda_graph")
    result = traces.run_in_process(runner, traces.trace_decode_tail({"r0": tokens}, 90))
    judge(result, expected, dtype, f"{kind} alone")


def stand_out_model(kind, page):
    """(config, weights, tokens, wanted positions, the query of the pair 600 apart and its key's position).  Queries are made of the
    keys' weights behind a permutation of the input's coordinates: a query whose input is x scores far above the rest against
    the key whose input is x permuted."""
    mixer = {
        "attention": attention(4, 2, 32, 1.0, rot(8, 1e4, (4.0, 256, 32.0, 1.0)), softcap=60.0),
        "attention 64": attention(4, 1, 64, 0.4, rot(32, 1e4), softcap=80.0),
        "attention 128": attention(2, 2, 128, 0.25, rot(64, 1e4, (4.0, 256, 32.0, 1.0)), softcap=20.0),
        "attention odd": attention(3, 1, 20, 1.5, rot(4, 1e4), softcap=40.0),
        "latent": latent(3, 24, 8, 16, 24, 0.25, 1e4, (4.0, 256, 32.0, 1.0)),
        "latent 128": latent(2, 64, 32, 40, 96, 0.15, 1e4),
        "latent odd": latent(5, 14, 2, 10, 21, 0.5, 1e4),
    }[kind]
    vocab, width = 80, 48
    cfg = config(width, vocab, [layer(mixer, None)])
    weights = make_weights(cfg, 21)
    for name in ("embed.norm", "l0.norm1"):
        weights[name] = torch.ones(width)  # so that a permuted embedding stays one behind the norms
    gen = torch.Generator().manual_seed(5)
    perm = torch.randperm(width, generator=gen)
    m, p = mixer["mixer"], "l0.mix"
    if "kv_heads" in m:
        k = weights[f"{p}.k"].view(m["kv_heads"], m["dim"], width).repeat_interleave(m["heads"] // m["kv_heads"], dim=0).reshape(-1, width)
    else:
        rank = m["kv_rank"]
        down = weights[f"{p}.dkv"]
        plain_part = (weights[f"{p}.uk"] @ (weights[f"{p}.dkv.norm"][:, None] * down[:rank])).view(m["heads"], m["dim"], width)
        k = torch.cat([plain_part, down[rank:].expand(m["heads"], -1, -1)], dim=1).reshape(-1, width)
    q = torch.zeros_like(k)
    q[:, perm] = k
    weights[f"{p}.q"] = q.to(torch.bfloat16).float()
    # rare tokens come in pairs: token 8 + i is token i seen through the permutation (its embedding is token i's, permuted)
    weights["embed"][8:16] = weights["embed"][0:8][:, perm]
    L = 700
    tokens = torch.randint(16, vocab, (L,), generator=gen).tolist()
    wanted = []
    for index, distance in enumerate([0, 1, page - 1, page, page + 1, 600, None, None]):
        at = 680 - 9 * index
        key = at - distance if distance is not None else index - 6
        if distance != 0:
            tokens[at], tokens[key] = index, 8 + index
        wanted.append(at)
    wanted += [0, 1, 2, page - 1, page]
    return cfg, weights, tokens, wanted, 680 - 9 * 5, 680 - 9 * 5 - 600


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("kind", ["attention", "attention 64", "attention 128", "attention odd", "latent", "latent 128", "latent odd"])
def test_keys_that_stand_out(kind, dtype, tmp_path):
    """A 700-token prompt in which rare tokens come in pairs: a query whose partner stands at distance 1, page - 1, page, page + 1 or 600, or
    at the sequence's first two places, scores far above the hundreds of other keys, so a key that is lost, read from a wrong page
    or turned by a wrong angle moves the logits by far more than rounding.  Whole, cut in the middle of a page with the tail decoded,
    and in small portions, on pages that earlier requests have shuffled."""
    page = 16
    cfg, weights, tokens, wanted, far_query, far_key = stand_out_model(kind, page)
    L, vocab = len(tokens), cfg["vocab"]
    logits = plain.forward(cfg, weights, tokens).numpy()
    folder = write_model(cfg, weights, tmp_path / "m")
    runner = make_runner(folder, dtype, page_size=page, num_pages=2 * (L // page + 2), decode_mode="cuda_graph")
    warm = traces.make_requests(vocab, [150, 90], seed=8)
    traces.run_in_process(runner, [
        {"step": 0, "entries": [{"id": "r0", "tokens": warm["r0"], "want": []}, {"id": "r1", "tokens": warm["r1"][:50], "want": []}], "end": ["r0"]},
        {"step": 1, "entries": [{"id": "r1", "tokens": warm["r1"][50:], "want": []}], "end": ["r1"]},
    ])
    start = 613  # the middle of a page
    cuts = {
        "whole": [{"step": 0, "entries": [{"id": "far", "tokens": tokens, "want": wanted}], "end": ["far"]}],
        "tail": [{"step": 0, "entries": [{"id": "far", "tokens": tokens[:start], "want": [w for w in wanted if w < start]}], "end": []}]
                + [{"step": 1 + n, "entries": [{"id": "far", "tokens": [tokens[start + n]], "want": [0] if start + n in wanted else []}],
                    "end": ["far"] if start + n == L - 1 else []} for n in range(L - start)],
    }
    steps, at, turn = [], 0, 0
    while at < L:
        size = min((37, 2, 64, 5, 129)[turn % 5], L - at)
        steps.append({"step": len(steps), "entries": [{"id": "far", "tokens": tokens[at : at + size], "want": [w - at for w in wanted if at <= w < at + size]}],
                      "end": ["far"] if at + size == L else []})
        at, turn = at + size, turn + 1
    cuts["portions"] = steps
    for cut, steps in cuts.items():
        result = traces.run_in_process(runner, steps)
        assert sorted(position for _, position in result) == sorted(wanted)
        judge(result, {"far": logits}, dtype, f"{kind} stand-out {cut}")
    # the pairs do stand out: without the far key the logits at its query differ by far more than the bounds
    lost = list(tokens)
    lost[far_key] = 17
    assert relative_error(plain.forward(cfg, weights, lost).numpy()[far_query], logits[far_query]) > 3 * BF16_BOUND


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_state_does_not_leak_between_requests(dtype, tmp_path):
    """Two state slots, six requests one after the other in pairs: a slot's memory and kept inputs are zeroed when it changes hands."""
    cfg, seed, page_size = CASES["small_pages"]
    weights = make_weights(cfg, seed)
    folder = write_model(cfg, weights, tmp_path / "m")
    requests = traces.make_requests(cfg["vocab"], [40, 33, 25, 47, 18, 29], seed=12)
    expected = {name: plain.forward(cfg, weights, tokens).numpy() for name, tokens in requests.items()}
    runner = make_runner(folder, dtype, page_size=page_size, num_pages=40, max_requests=2)
    judge(traces.run_in_process(runner, traces.trace_mixed(requests, seed=2, max_live=2)), expected, dtype, "two state slots")


# ---------------------------------------------------------------------------- kernels


def _unit_inputs(parts, n, taps, counts, starts, seed=0):
    """Rows of `counts` tokens that start at positions `starts`, in shuffled state slots, with earlier inputs in their rings."""
    g = torch.Generator().manual_seed(seed)
    W, T, R = parts * n, sum(counts), len(counts)

    def normal(*shape):
        return torch.randn(*shape, generator=g)

    d = types.SimpleNamespace(parts=parts, n=n, W=W, T=T, n_taps=taps, counts=counts, starts=starts)
    d.packed = normal(T, 2 * W + 8).to(torch.bfloat16)
    d.gates = (normal(2, parts, n, n) * 1.5 * n ** -0.5).to(torch.bfloat16)  # [gate, part, out, in]
    d.taps, d.conv_bias, d.gate_bias, d.lam = normal(taps, W) * 0.6, normal(W) * 0.3, normal(2, W), normal(W) * 2 - 2
    d.slots = torch.randperm(R + 3, generator=g)[:R].tolist()
    d.states, d.rings = normal(R + 3, W), normal(R + 3, taps, W)
    d.indptr = [0] + np.cumsum(counts).tolist()
    d.rows = [row for row, count in enumerate(counts) for _ in range(count)]
    d.positions = [start + t for start, count in zip(starts, counts) for t in range(count)]
    return d


def _unit_reference(d):
    """(out, states, rings) in 64-bit, row by row through the plain pieces, the ring's inputs ahead of a row's tokens."""
    out = torch.zeros(d.T, d.W, dtype=torch.float64)
    states, rings = d.states.double().clone(), d.rings.double().clone()
    y, x = d.packed[:, : d.W].double(), d.packed[:, d.W : 2 * d.W].double()
    for row, (count, start) in enumerate(zip(d.counts, d.starts)):
        t0, slot = d.indptr[row], d.slots[row]
        earlier = [rings[slot, p % d.n_taps] for p in range(max(start - d.n_taps + 1, 0), start)]
        inputs = torch.cat([torch.stack(earlier), x[t0 : t0 + count]]) if earlier else x[t0 : t0 + count]
        u = plain.short_convolution(inputs, d.taps.double().T, d.conv_bias.double())[len(earlier):]
        r, i = (torch.sigmoid(plain.block_diagonal(u, d.gates[k].double(), d.gate_bias[k].double().view(d.parts, d.n))) for k in (0, 1))
        a = torch.exp(-8.0 * r * plain.softplus(d.lam.double()))
        into = torch.sqrt(1.0 - a * a) * i * u
        for t in range(count):
            states[slot] = a[t] * states[slot] + into[t]
            out[t0 + t] = states[slot] * plain.gelu_tanh(y[t0 + t])
            rings[slot, (start + t) % d.n_taps] = x[t0 + t]
    return out, states, rings


def _unit_run(d, how, dtype, segments=None):
    from kairyu_b200 import kernels

    i32 = dict(dtype=torch.int32, device="cuda")
    packed = d.packed.to(dtype).cuda()
    y, x = packed[:, : d.W], packed[:, d.W : 2 * d.W]
    states, rings = d.states.cuda(), d.rings.cuda() if d.n_taps > 1 else None
    taps, conv_bias, gate_bias = d.taps.cuda(), d.conv_bias.cuda(), d.gate_bias.cuda()
    rate = (-8.0 * plain.softplus(d.lam.double())).float().cuda()
    where = dict(row_ids=torch.tensor(d.rows, **i32), qo_indptr=torch.tensor(d.indptr, **i32), positions=torch.tensor(d.positions, **i32),
                 state_slots=torch.tensor(d.slots, **i32))
    flag = torch.zeros(1, **i32)
    out = torch.full((d.T, d.W), float("nan"), dtype=dtype, device="cuda")
    a, into = torch.empty(d.T, d.W, device="cuda"), torch.empty(d.T, d.W, device="cuda")
    padded = kernels.rglru_padded(d.n)
    if how == "fma":
        kernels.rglru_gates(x, taps, conv_bias, rings, d.gates.to(dtype).transpose(2, 3).contiguous().cuda(), gate_bias, rate, a, into, flag=flag, **where)
    else:
        weights = torch.zeros(2, d.parts, padded, padded, dtype=dtype)
        weights[:, :, : d.n, : d.n] = d.gates
        weights = weights.cuda()
        hi, lo = (torch.full((d.T, d.parts * padded), float("nan"), dtype=dtype, device="cuda") for _ in range(2))
        kernels.rglru_convolve(x, taps, conv_bias, rings, hi, lo, d.parts, update_rings=how == "step", flag=flag, **where)
        if how == "step":
            kernels.rglru_step(hi, lo, y, states, weights, gate_bias, rate, out, row_ids=where["row_ids"], state_slots=where["state_slots"], flag=flag)
        else:
            kernels.rglru_gates_tc5(hi, lo, weights, gate_bias, rate, a, into, flag=flag)
    if how != "step":
        kernels.rglru_scan(a, into, x, y, states, rings, d.n_taps, out, qo_indptr=where["qo_indptr"], positions=where["positions"],
                           state_slots=where["state_slots"], segments=segments)
    assert int(flag) == 0
    return out.double().cpu(), states.double().cpu(), rings.double().cpu() if rings is not None else d.rings.double()


UNITS = [(1, 16, 4), (2, 72, 3), (3, 24, 4), (2, 256, 4), (1, 136, 2), (4, 8, 1), (2, 200, 5), (3, 10, 4), (2, 21, 3), (1, 300, 7)]


@pytest.mark.parametrize("parts, n, taps", UNITS)
def test_unit_kernels_on_portions(parts, n, taps):
    """Convolution, gates and walk on unequal rows (one begins a sequence, others go on from their rings, two of one token), on FMAs in
    32-bit and on tensor cores, the walk in one piece and cut into segments of every kind; the states and rings they leave."""
    d = _unit_inputs(parts, n, taps, [130, 1, 3, 77, 1, 260], [0, 5, 1, 2, 0, 40])
    want = _unit_reference(d)
    scale = max(1.0, float(want[1].abs().max()))
    for how, dtype, segments, tolerance in (("fma", torch.float32, (1, 1), 1e-5), ("fma", torch.float32, (16, 4), 1e-5), ("tc5", torch.bfloat16, None, 2e-4),
                                            ("tc5", torch.bfloat16, (1, 1), 2e-4), ("tc5", torch.bfloat16, (3, 2), 2e-4), ("tc5", torch.bfloat16, (16, 8), 2e-4)):
        out, states, rings = _unit_run(d, how, dtype, segments)
        assert (states - want[1]).abs().max() < tolerance * scale, (how, segments)
        rounding = 0.0 if dtype == torch.float32 else 2.0 ** -8
        assert ((out - want[0]).abs() <= tolerance * scale * 4 + rounding * want[0].abs()).all(), (how, segments)
        for row, slot in enumerate(d.slots):
            if taps > 1:
                assert torch.equal(rings[slot], want[2][slot]), (how, row)
        untouched = [slot for slot in range(len(d.counts) + 3) if slot not in d.slots]
        assert torch.equal(states[untouched], d.states.double()[untouched]) and torch.equal(rings[untouched], d.rings.double()[untouched])


@pytest.mark.parametrize("rows", [1, 8, 13, 70])
@pytest.mark.parametrize("parts, n, taps", UNITS)
def test_unit_kernels_on_single_tokens(parts, n, taps, rows):
    """A step of single tokens at positions 0, 1, 2, ... and far on, through the kernel made for it."""
    d = _unit_inputs(parts, n, taps, [1] * rows, [(7 * row) % 90 if row % 3 else row // 3 for row in range(rows)], seed=rows)
    want = _unit_reference(d)
    out, states, rings = _unit_run(d, "step", torch.bfloat16)
    scale = max(1.0, float(want[1].abs().max()))
    assert (states - want[1]).abs().max() < 1e-4 * scale
    assert ((out - want[0]).abs() <= 4e-4 * scale + 2.0 ** -8 * want[0].abs()).all()
    if taps > 1:
        assert torch.equal(rings[d.slots], want[2][d.slots])


def test_unit_decays_close_to_one():
    """Decays so close to one that the distance from one is lost in 32-bit unless it is formed from the logarithm, and that a rounding which leans
    one way adds up over 3,000 tokens of one sign; every path."""
    d = _unit_inputs(2, 24, 4, [3000], [0], seed=4)
    d.lam = d.lam * 0.0 - 9.0
    d.conv_bias = d.conv_bias.abs() + 3.0
    want = _unit_reference(d)
    for how, dtype, tolerance in (("fma", torch.float32, 2e-5), ("tc5", torch.bfloat16, 1e-4)):
        _, states, _ = _unit_run(d, how, dtype)
        error = (states - want[1])[d.slots].abs().max() / want[1][d.slots].abs().max()
        assert error < tolerance, (how, error)


@pytest.mark.parametrize("D", [16, 48, 64, 96, 128, 256])
def test_the_cap_in_every_attention_kernel(D):
    """The tensor-core kernels with the cap in both forms, and without, against sums in 64-bit: a prompt's portion (also with its keys split over
    blocks and two tiles a block where the kernel has that), single tokens in one split and several."""
    from kairyu_b200 import kernels
    from kairyu_b200.engine.workspace import Workspace

    H, G, L, page = 4, 2, 500, 16
    gen = torch.Generator().manual_seed(D)
    i32 = dict(dtype=torch.int32, device="cuda")
    k, v = torch.randn(2, L, G, D, generator=gen).to(torch.bfloat16)
    q = torch.randn(L, H, D, generator=gen).to(torch.bfloat16)
    pages = torch.randperm(L // page + 1, generator=gen) + 1
    both = torch.zeros(2, len(pages) + 1, page, G, D, dtype=torch.bfloat16)
    for j in range(L):
        both[0, pages[j // page], j % page], both[1, pages[j // page], j % page] = k[j], v[j]
    k_cache, v_cache = both.cuda()
    table = pages.to(torch.int32).cuda()[None].contiguous()
    scale = 2.5 * D ** -0.5
    longest = float(q.double().norm(dim=-1).max() * k.double().norm(dim=-1).max())
    near_cap = scale * longest / 0.44
    tile = kernels.attention_prefill_tile_rows(D)
    wide = kernels.attention_prefill_wide_tile_rows(D)
    for cap, softcap in ((None, None), (near_cap, kernels.SoftCap.make(scale, near_cap, longest)), (3.0, kernels.SoftCap.make(scale, 3.0)),
                         (near_cap, kernels.SoftCap.make(scale, near_cap))):
        if softcap is not None:
            assert softcap.mode == (1 if cap == near_cap and softcap.c[0] else 2)
        want = torch.cat([plain.softmax_of_the_past(plain.cap(q[:, h].double() @ k[:, h // 2].double().T * scale, cap)) @ v[:, h // 2].double() for h in range(H)], dim=-1)
        rows = q.reshape(L, H * D).cuda()
        flag = torch.zeros(1, **i32)
        for start in (0, 311):
            count = L - start
            starts = list(range(0, count, tile))
            shape = dict(qo_indptr=torch.tensor([0, count], **i32), seq_lens=torch.tensor([L], **i32), block_table=table, tile_rows=torch.zeros(len(starts), **i32),
                         tile_starts=torch.tensor(starts, **i32), num_tiles=len(starts), num_q_heads=H, scale=scale, flag=flag, max_seq_len=L, workspace=Workspace("cuda"))
            variants = [dict(num_splits=1), dict(num_splits=3)]
            if wide:
                wides = list(range(0, count, wide))
                variants.append(dict(num_splits=1, two_tiles=True, wide_tiles=(len(wides), torch.zeros(len(wides), **i32), torch.tensor(wides, **i32))))
            for variant in variants:
                out = torch.zeros(count, H * D, dtype=torch.bfloat16, device="cuda")
                kernels.attention_prefill_mma(rows[start:], out, k_cache, v_cache, softcap=softcap, **shape, **variant)
                assert int(flag) == 0
                assert (out.double().cpu() - want[start:]).abs().max() < 2e-2, (cap, start, variant)
        at = [0, 1, 15, 16, 200, 499]
        for splits in (None, 1, 2):
            out = torch.zeros(len(at), H * D, dtype=torch.bfloat16, device="cuda")
            kernels.attention_decode_mma(rows[at].contiguous(), out, k_cache, v_cache, seq_lens=torch.tensor([p + 1 for p in at], **i32), block_table=table.repeat(len(at), 1).contiguous(),
                                         decode_rows=torch.arange(len(at), **i32), decode_tokens=torch.arange(len(at), **i32), num_rows=len(at), max_seq_len=L,
                                         num_q_heads=H, scale=scale, workspace=Workspace("cuda"), flag=flag, num_splits=splits, softcap=softcap)
            assert int(flag) == 0
            assert (out.double().cpu() - want[at]).abs().max() < 2e-2, (cap, splits)


@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("sizes", [
    # query heads, key/value heads, head width, rotated columns, value width (None: a value is its key), other columns between
    (3, 1, 20, 8, None, 3), (4, 2, 32, 16, None, 8), (5, 5, 16, 16, None, 0), (8, 2, 64, 64, None, 16), (2, 1, 128, 32, None, 8), (9, 3, 96, 96, None, 8),
    (2, 2, 256, 64, None, 0), (1, 1, 264, 16, None, 8), (6, 2, 48, 0, None, 8), (4, 2, 32, 16, 24, 8), (3, 1, 10, 2, 14, 1),
])
def test_heads_of_unit_mean_square(sizes, dtype):
    """Rotation, then every head of q and k divided by its own root mean square, and the page write, with values that are the keys as projected and
    with values of their own; for rows that write all, some and none of their positions."""
    from kairyu_b200 import kernels

    H, G, D, turned, vdim, spare = sizes
    g = torch.Generator().manual_seed(6)
    page, tokens = 8, 37
    block_table = torch.tensor([[3, 1, 7, 5, 2, -1], [4, 6, 8, -1, -1, -1]], dtype=torch.int32, device="cuda")
    row_ids = torch.tensor([0] * 30 + [1] * 7, dtype=torch.int32, device="cuda")
    where = torch.tensor(list(range(5, 35)) + list(range(11, 18)), dtype=torch.int32, device="cuda")
    write_from = torch.tensor([8, 0], dtype=torch.int32, device="cuda")  # row 0 only reads its first page
    k_off = H * D
    DV = D if vdim is None else vdim
    v_off = k_off if vdim is None else k_off + G * D + spare
    source = (torch.randn(tokens, max(v_off + G * DV, k_off + G * D) + spare, generator=g) * 0.05).to(dtype)  # small: eps weighs in
    table = rot(turned, 100.0, (4.0, 32, 4.0, 1.0)) if turned else None
    tables = {}
    if turned:
        f, amplitude = plain.yarn(table)
        angles = torch.arange(64, dtype=torch.float64)[:, None] * torch.tensor(f, dtype=torch.float64)
        tables = dict(cos=(angles.cos() * amplitude).float().cuda(), sin=(angles.sin() * amplitude).float().cuda())
    k_cache = torch.zeros(9, page, G, D, dtype=dtype, device="cuda")
    v_cache = torch.zeros(9, page, G, DV, dtype=dtype, device="cuda")
    packed = source.clone().cuda()
    flag = torch.zeros(1, dtype=torch.int32, device="cuda")
    kernels.projection_norm_rope_write(packed, num_q_heads=H, num_kv_heads=G, head_dim=D, value_dim=DV, k_offset=k_off, v_offset=v_off, positions=where,
                                       row_ids=row_ids, eps=1e-3, block_table=block_table, write_from=write_from, k_cache=k_cache, v_cache=v_cache, flag=flag,
                                       unit_heads=True, **tables)
    assert int(flag) == 0
    s = source.double()
    q, k = (plain.unit_rms(plain.rotate_halves(part.view(tokens, -1, D), where.cpu(), table), 1e-3) for part in (s[:, :k_off], s[:, k_off : k_off + G * D]))
    tolerance = 2e-6 if dtype == torch.float32 else 1.0 / 128
    assert ((packed[:, :k_off].double().cpu() - q.reshape(tokens, -1)).abs() <= tolerance * q.abs().max()).all()
    assert torch.equal(packed[:, k_off:].cpu(), source[:, k_off:])
    for t in range(tokens):
        position, row = int(where[t]), int(row_ids[t])
        slot = (int(block_table[row, position // page]), position % page)
        if position >= int(write_from[row]):
            assert (k_cache[slot].cpu().double() - k[t]).abs().max() <= tolerance * k.abs().max()
            assert torch.equal(v_cache[slot].flatten().cpu(), source[t, v_off : v_off + G * DV])
        else:
            assert not k_cache[slot].any() and not v_cache[slot].any()


@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("width", [50, 72, 1024, 2056])
def test_scaled_sum_and_norm(width, dtype):
    """The norm's kernel with a pending sum that is scaled column by column: all rows (the residual takes the sum in 32-bit) and listed rows (it does not)."""
    from kairyu_b200 import kernels

    g = torch.Generator().manual_seed(4)
    tokens = 21
    x = torch.randn(tokens, width, generator=g) * 3
    y = torch.randn(tokens, width, generator=g).to(dtype)
    scale, weight = torch.randn(width, generator=g), (1 + 0.2 * torch.randn(width, generator=g)).to(torch.bfloat16)
    residual, out = x.clone().cuda(), torch.empty(tokens, width, dtype=dtype, device="cuda")
    kernels.rmsnorm(residual, weight.to(dtype).cuda(), 1e-5, out, delta=y.cuda(), delta_scale=scale.cuda())
    total = x.double() + scale.double() * y.double()
    assert (residual.cpu().double() - total).abs().max() < 1e-5
    want = plain.rms_norm(total, weight.double(), 1e-5)
    assert (out.cpu().double() - want).abs().max() < (2e-5 if dtype == torch.float32 else 0.03)
    rows = torch.tensor([5, 0, 20], dtype=torch.int32, device="cuda")
    untouched, few = x.clone().cuda(), torch.empty(3, width, dtype=dtype, device="cuda")
    kernels.rmsnorm(untouched, weight.to(dtype).cuda(), 1e-5, few, delta=y.cuda(), delta_scale=scale.cuda(), rows=rows)
    assert torch.equal(few, out[rows.long()]) and torch.equal(untouched.cpu(), x)


@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("width", [50, 72, 1028, 5120, 16500])
def test_embedding_with_its_norm(width, dtype):
    """The gather with a norm of its own, in every access width; an id outside the table is flagged and gives zeros."""
    from kairyu_b200 import kernels

    g = torch.Generator().manual_seed(6)
    table = torch.randn(29, width, generator=g).to(dtype)
    ids = torch.tensor([3, 28, 0, 3, 29], dtype=torch.int32)
    weight = (1 + 0.2 * torch.randn(width, generator=g)).to(dtype)
    out, flag = torch.empty(5, width, device="cuda"), torch.zeros(1, dtype=torch.int32, device="cuda")
    kernels.embedding_norm(table.cuda(), ids.cuda(), out, weight=weight.cuda(), eps=1e-5, scale=1.5, flag=flag)
    want = plain.rms_norm(table.double()[ids[:4].long()] * 1.5, weight.double(), 1e-5)
    assert (out[:4].cpu().double() - want).abs().max() < 2e-5 and not out[4].any()
    assert int(flag) == kernels.FLAG_BAD_TOKEN


@pytest.mark.parametrize("tokens", [1, 5, 8, 16])
def test_folded_product_scales_what_it_adds(tokens):
    """A few rows: the product that adds its result to the residual scales it column by column on the way, and leaves the next norm half done."""
    from kairyu_b200 import kernels
    from kairyu_b200.engine.workspace import Workspace

    g = torch.Generator().manual_seed(tokens)
    width, inner = 208, 96
    ws = Workspace("cuda")
    x = torch.randn(tokens, inner, generator=g).to(torch.bfloat16)
    w = (torch.randn(width, inner, generator=g) * inner ** -0.5).to(torch.bfloat16)
    residual, scale = torch.randn(tokens, width, generator=g), torch.randn(width, generator=g)
    weight = (1 + 0.2 * torch.randn(width, generator=g)).to(torch.bfloat16)
    held = residual.clone().cuda()
    fold = kernels.ResidualNorm(held, weight.cuda(), 1e-5, ws.buffer("values", tokens, width, torch.bfloat16),
                                ws.flat("sumsq", 16 * kernels.skinny_blocks(tokens, width), torch.float32).view(-1, 16), scale.cuda())
    kernels.linear(x.cuda(), w.cuda(), None, None, fold=fold)
    total = residual.double() + scale.double() * (x.double() @ w.double().T)
    assert (held.cpu().double() - total).abs().max() < 1e-4
    half = fold.result()
    assert (half.values.cpu().double() - total * weight.double()).abs().max() < 0.05
    assert torch.allclose(half.sumsq[:, :tokens].sum(0).cpu().double(), (total * total).sum(-1), rtol=1e-4)


@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
def test_gated_head_products(dtype):
    """The product a head whose result is gated by columns of wider rows."""
    from kairyu_b200 import kernels

    g = torch.Generator().manual_seed(3)
    for tokens, heads, rank, vdim, before in ((1, 3, 24, 12, 8), (9, 5, 32, 16, 64), (40, 2, 48, 9, 3), (130, 4, 16, 40, 0)):
        x = torch.randn(tokens, heads, rank + 8, generator=g).to(dtype)
        w = (torch.randn(heads, vdim, rank, generator=g) * rank ** -0.5).to(dtype)
        rows = torch.randn(tokens, before + heads * vdim, generator=g).to(dtype) * 2
        out = torch.empty(tokens, heads, vdim, dtype=dtype, device="cuda")
        kernels.heads_linear(x.cuda()[:, :, :rank], w.cuda(), out, gate=rows.cuda()[:, before:])
        want = torch.einsum("thk,hnk->thn", x[:, :, :rank].double(), w.double()) * torch.sigmoid(rows[:, before:].double()).view(tokens, heads, vdim)
        assert (out.cpu().double() - want).abs().max() < (1e-5 if dtype == torch.float32 else 0.04)


# ---------------------------------------------------------------------------- the engine


def test_long_decoding(tmp_path):
    """Six hundred tokens decoded one by one through graphs, beside a second request that starts and ends meanwhile, in both modes."""
    cfg = config(40, 53, [layer(rglru(32, 2, 4), None), layer(attention(4, 2, 32, 0.45, rot(16, 1e4, (4.0, 128, 16.0, 1.0)), softcap=6.0), 24),
                          layer(latent(3, 16, 16, 12, 32, 0.4), None), layer(rglru(48, 3, 2), 16)])
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
