"""Rezelix without a GPU: the config reader, the spec it builds, model folders written and read back, the rotation tables, the cap's
polynomial, what the GPU tests' bounds can see, the plain implementation's own pieces, and, with the kernels replaced by their
torch statements, every cut through the step function and greedy generation through the scheduler and the command line."""

import json
import math

import numpy as np
import pytest
import torch

import rezelix_plain as plain
import traces
from rezelix_cases import CASES, YARN, attention, config, latent, layer, make_weights, relative_error, rglru, rot, write_model

from kairyu_b200.cache import CacheLayout, CacheManager
from kairyu_b200.config.model_config import ConfigError
from kairyu_b200.engine.engine import build_model
from kairyu_b200.parts import PagedKVSpec, StateSpec
from kairyu_b200.registry import architecture_of, supported_architectures
from kairyu_b200.weights.loading import WeightError, load_into


def test_registered_by_its_config_key():
    assert "Rezelix" in supported_architectures()
    assert architecture_of({"architecture": "Rezelix"}).name == "Rezelix"


@pytest.mark.parametrize("name", list(CASES))
def test_spec_and_cache_needs(name):
    cfg, _, _ = CASES[name]
    model, parsed = build_model(cfg, dtype="float32", device="meta")
    entries = cfg["layers"]
    assert len(model.blocks) == len(entries) == len(model.schedule)
    assert [(call.layer, call.cache_slot) for call in model.schedule] == [(i, i) for i in range(len(entries))]
    needs = model.cache_slot_specs()
    for index, entry in enumerate(entries):
        m = entry["mixer"]
        if entry["type"] == "attention":
            assert needs[index] == (PagedKVSpec(m["kv_heads"], m["dim"], None, v_head_dim=m["dim"]),)
        elif entry["type"] == "latent_attention":
            assert needs[index] == (PagedKVSpec(1, m["kv_rank"] + m["rot_dim"], None, v_head_dim=0),)
        else:
            ring = (StateSpec((m["conv"], m["width"]), "float32"),) if m["conv"] > 1 else ()
            assert needs[index] == (StateSpec((m["width"],), "float32"),) + ring
        assert (model.blocks[index].ffn is None) == (entry["mlp"] is None)
    assert {spec.name: tuple(spec.shape) for spec in model.tensor_specs()} == {n: tuple(t.shape) for n, t in make_weights(cfg, 0).items()}
    assert parsed.vocab_size == cfg["vocab"] and parsed.hidden_size == cfg["width"]
    assert model.graph_safe()


@pytest.mark.parametrize("damage, message", [
    (lambda c: c.pop("vocab"), "vocab"),
    (lambda c: c.pop("width"), "width"),
    (lambda c: c.update(layers=[]), "layers"),
    (lambda c: c["norm"].pop("eps"), "eps"),
    (lambda c: c["layers"][1]["mixer"].pop("scale"), "scale"),
    (lambda c: c["layers"][1]["mixer"].update(scale=-0.5), "scale"),
    (lambda c: c["layers"][1]["mixer"].update(softcap=0.0), "softcap"),
    (lambda c: c["layers"][1]["mixer"].update(vdim=8), "vdim"),
    (lambda c: c["layers"][1]["mixer"].update(kv_heads=3), "multiple"),
    (lambda c: c["layers"][1]["mixer"]["rot"].update(dims=7), "even"),
    (lambda c: c["layers"][1]["mixer"]["rot"].update(dims=64), "at most 32"),
    (lambda c: c["layers"][1]["mixer"]["rot"]["scaling"].pop("original"), "original"),
    (lambda c: c["layers"][1]["mixer"]["rot"]["scaling"].update(factor=0), "factor"),
    (lambda c: c["layers"][2]["mixer"].pop("kv_rank"), "kv_rank"),
    (lambda c: c["layers"][2]["mixer"]["rot"].update(dims=6), "rot_dim"),
    (lambda c: c["layers"][2]["mixer"].pop("rot"), "rot"),
    (lambda c: c["layers"][0]["mixer"].update(blocks=5), "equal parts"),
    (lambda c: c["layers"][0]["mixer"].pop("conv"), "conv"),
    (lambda c: c["layers"][0].update(type="conv"), "unknown layer type"),
    (lambda c: c["layers"][0]["mlp"].update(kind="moe"), "unknown feed-forward"),
    (lambda c: c["layers"][0]["mlp"].pop("ff"), "ff"),
])
def test_config_errors_name_the_key(damage, message):
    cfg = json.loads(json.dumps(CASES["mixed"][0]))
    damage(cfg)
    with pytest.raises(ConfigError, match=message):
        build_model(cfg, dtype="float32", device="meta")


def test_model_folder_round_trip(tmp_path):
    cfg, seed, _ = CASES["mixed"]
    weights = make_weights(cfg, seed)
    folder = write_model(cfg, weights, tmp_path / "m")
    model, _ = build_model(cfg, dtype="float32", device="cpu")
    load_into(model, folder, strict_unexpected=True)
    recurrent, attending, latent_mixer = (model.blocks[i].mixer for i in range(3))
    assert torch.equal(recurrent.w_in[:64], weights["l0.mix.y"]) and torch.equal(recurrent.w_in[64:], weights["l0.mix.x"])
    assert torch.equal(recurrent.taps, weights["l0.mix.conv"].T) and torch.equal(recurrent.gates_t[1, 3], weights["l0.mix.ri"][3].T)
    assert torch.allclose(recurrent.rate, (-8.0 * torch.log1p(torch.exp(weights["l0.mix.lam"].double()))).float())
    assert attending.v_offset == attending.k_offset == 128 and attending.w_in.shape[0] == 128 + 64
    assert torch.equal(latent_mixer.w_in[-36:], weights["l2.mix.g"])  # the gate rides in the input product
    assert torch.equal(model.blocks[1]._scales[1], weights["l1.ls2"]) and model.blocks[2]._scales[1] is None
    broken = dict(weights)
    del broken["l2.mix.g"]
    broken["l0.mix.ra"] = torch.zeros(3, 16, 16)
    with pytest.raises(WeightError) as error:
        load_into(build_model(cfg, dtype="float32", device="cpu")[0], write_model(cfg, broken, tmp_path / "b"))
    assert error.value.missing == ["l2.mix.g"] and error.value.wrong_shape[0][0] == "l0.mix.ra"
    # bfloat16 holds the gates' matrices padded to whole 16 columns
    model, _ = build_model(CASES["odd"][0], dtype="bfloat16", device="cpu")
    load_into(model, write_model(CASES["odd"][0], make_weights(CASES["odd"][0], 1), tmp_path / "o"))
    gates = model.blocks[1].mixer.gates
    assert gates.shape == (2, 2, 32, 32) and not gates[:, :, 21:].any() and not gates[:, :, :, 21:].any() and gates[1, 1, :21, :21].any()


def test_random_weights_through_the_registry(tmp_path):
    from kairyu_b200.weights import write_random_model

    cfg, _, _ = CASES["small_pages"]
    folder = write_random_model(cfg, tmp_path / "r", seed=4, dtype="bfloat16")
    model, _ = build_model(json.loads((folder / "config.json").read_text()), dtype="float32", device="cpu")
    load_into(model, folder, strict_unexpected=True)


@pytest.mark.parametrize("table", [rot(16, 500.0, YARN), rot(8, 300.0, (3.0, 48, 6.0, 1.0)), rot(64, 1e6, (32.0, 4096, 32.0, 1.0)), rot(2, 50.0, (2.0, 32, 4.0, 0.25)),
                                   rot(6, 100.0, (7.0, 3, 20.0, 2.0)), rot(10, 30.0, (0.5, 64, 1.0, 16.0)), rot(12, 77.0)])
def test_rotation_tables_are_correctly_rounded(table):
    """Every entry of the engine's table is the 64-bit cosine or sine, times the amplitude, rounded once; also where the ramp's ends meet or
    cross and where the factor is below one."""
    from kairyu_b200.models.rezelix import _parse_rot, _rope
    from kairyu_b200.parts import POSITION_ENCODINGS

    spec = _rope(_parse_rot(table, table["dims"], "rot"), 5000)
    cos, sin = POSITION_ENCODINGS.build(spec, device="cpu", dtype=torch.float32).rotary_tables()
    f, amplitude = plain.yarn(table)
    angles = torch.arange(5000, dtype=torch.float64)[:, None] * torch.tensor(f, dtype=torch.float64)
    assert torch.equal(cos, (angles.cos() * amplitude).float()) and torch.equal(sin, (angles.sin() * amplitude).float())


@pytest.mark.parametrize("scale, cap, largest", [(0.125, 30.0, 64.6), (0.09, 26.0, 129.0), (1.0, 40.0, 16.2), (0.5, 3.0, 10.0), (0.1, 50.0, None)])
def test_the_cap_as_the_kernels_take_it(scale, cap, largest):
    """The numbers the host hands to the tensor-core kernels: both forms against tanh, over the whole range of scores."""
    from kairyu_b200.kernels import SoftCap

    held = SoftCap.make(scale, cap, largest)
    near = largest is not None and scale / cap * largest <= 0.45
    assert held.mode == (1 if near else 2)
    reach = largest if largest is not None else 40.0 * cap / scale
    for raw in np.linspace(-reach, reach, 801):
        want = cap * math.tanh(scale * raw / cap) * math.log2(math.e)
        full = held.b - 2.0 * held.b / (1.0 + 2.0 ** min(held.a * raw, 1000.0))
        assert abs(full - want) < 1e-5 * cap
        if near:
            got = raw * sum(held.c[j] * (raw * raw) ** j for j in range(4))
            assert abs(got - want) <= 4e-7 * abs(want)
    for wrong in ((0.0, 1.0), (1.0, 0.0), (-1.0, 2.0)):
        with pytest.raises(ValueError):
            SoftCap.make(*wrong)


def _faults():
    """Ways to get one mechanism wrong, each a (name, patch) where ``patch(mp)`` replaces one piece of the plain model."""
    p = plain
    right = {name: getattr(p, name) for name in ("yarn", "rotate_halves", "unit_rms", "short_convolution", "latent_attention", "rms_norm")}

    def attention_with(order="turn then norm", values="projected"):
        def run(h, w, m, eps):
            n, H, G, d = h.shape[0], m["heads"], m["kv_heads"], m["dim"]
            positions = torch.arange(n)
            raw = (h @ w["k"].T).view(n, G, d)
            prepare = {
                "turn then norm": lambda x: p.unit_rms(p.rotate_halves(x, positions, m.get("rot")), eps),
                "norm then turn": lambda x: p.rotate_halves(p.unit_rms(x, eps), positions, m.get("rot")),
                "turn": lambda x: p.rotate_halves(x, positions, m.get("rot")),
            }[order]
            q, k = prepare((h @ w["q"].T).view(n, H, d)), prepare(raw)
            v = {"projected": raw, "turned": p.rotate_halves(raw, positions, m.get("rot")), "normed": p.unit_rms(raw, eps)}[values]
            own = [head // (H // G) for head in range(H)]
            out = [p.softmax_of_the_past(p.cap((q[:, a] @ k[:, own[a]].T) * m["scale"], m.get("softcap"))) @ v[:, own[a]] for a in range(H)]
            return torch.cat(out, dim=-1) @ w["o"].T
        return run

    def latent_without(what):
        def run(h, w, m, eps):
            w = dict(w)
            if what == "gate":
                w["g"] = w["g"] * 0.0  # sigmoid(0): a half everywhere
            elif what == "scale of the query's width":
                m = dict(m, scale=(m["dim"] + m["rot_dim"]) ** -0.5)
            elif what == "latent norm's weight":
                w["dkv.norm"] = torch.ones_like(w["dkv.norm"])
            return right["latent_attention"](h, w, m, eps)
        return run

    def recurrence(scale=8.0, root=True, first=False, swap=False):
        def run(u, r, i, lam):
            if swap:
                r, i = i, r
            log_a = -scale * r * p.softplus(lam)
            a = torch.exp(log_a)
            into = (torch.sqrt(-torch.expm1(2.0 * log_a)) if root else 1.0 - a) * i * u
            if first:
                into[0] = (i * u)[0]
            S, out = torch.zeros_like(u[0]), []
            for t in range(u.shape[0]):
                S = a[t] * S + into[t]
                out.append(S)
            return torch.stack(out)
        return run

    def every(mp, **names):
        for name, function in names.items():
            mp.setattr(p, name, function)

    return [
        ("no cap", lambda mp: every(mp, cap=lambda s, c: s)),
        ("values turned", lambda mp: every(mp, attention=attention_with(values="turned"))),
        ("values of unit mean square", lambda mp: every(mp, attention=attention_with(values="normed"))),
        ("queries and keys not normed", lambda mp: every(mp, attention=attention_with("turn"))),
        ("normed before the turn", lambda mp: every(mp, attention=attention_with("norm then turn"))),
        ("no frequency scaling", lambda mp: every(mp, yarn=lambda t: (right["yarn"](dict(t, scaling=None))[0], right["yarn"](t)[1]))),
        ("no amplitude", lambda mp: every(mp, yarn=lambda t: (right["yarn"](t)[0], 1.0))),
        ("positions doubled", lambda mp: every(mp, rotate_halves=lambda x, positions, t: right["rotate_halves"](x, positions * 2, t))),
        ("the output gate shut halfway", lambda mp: every(mp, latent_attention=latent_without("gate"))),
        ("the scale from the width", lambda mp: every(mp, latent_attention=latent_without("scale of the query's width"))),
        ("the latent norm's weight left out", lambda mp: every(mp, latent_attention=latent_without("latent norm's weight"))),
        ("the convolution a token late", lambda mp: every(mp, short_convolution=lambda x, taps, bias: right["short_convolution"](x, taps.roll(1, dims=1), bias))),
        ("the convolution's bias left out", lambda mp: every(mp, short_convolution=lambda x, taps, bias: right["short_convolution"](x, taps, bias * 0.0))),
        ("gelu left out", lambda mp: every(mp, gelu_tanh=lambda z: z)),
        ("the decay's factor", lambda mp: every(mp, gated_linear_recurrence=recurrence(scale=1.0))),
        ("the input not under a root", lambda mp: every(mp, gated_linear_recurrence=recurrence(root=False))),
        ("the two gates swapped", lambda mp: every(mp, gated_linear_recurrence=recurrence(swap=True))),
        ("the gates' matrices transposed", lambda mp: every(mp, block_diagonal=lambda u, mats, bias: (
            torch.einsum("tbi,bio->tbo", u.view(u.shape[0], mats.shape[0], -1), mats) + bias).reshape(u.shape))),
        ("the first token's input whole", lambda mp: every(mp, gated_linear_recurrence=recurrence(first=True))),
    ]


# what these do is small in bfloat16 at most positions of some configurations; the 32-bit bound sees them
SMALL = ("no amplitude", "no frequency scaling", "normed before the turn", "the first token's input whole", "values of unit mean square",
         "the convolution's bias left out", "no cap", "the latent norm's weight left out", "the scale from the width")


@pytest.mark.parametrize("name", list(CASES))
def test_the_bounds_see_each_fault(name):
    """What the GPU tests' bounds are for: the plain model with one mechanism wrong is beyond the 32-bit bound at many positions, and,
    but for small faults, beyond the bfloat16 bound at the median position.  (A fault in a part that a configuration does not
    have changes nothing there and is skipped.)"""
    cfg, seed, _ = CASES[name]
    weights = make_weights(cfg, seed)
    tokens = traces.make_requests(cfg["vocab"], [90], seed=1)["r0"]
    correct = plain.forward(cfg, weights, tokens).numpy()
    seen = 0
    for what, patch in _faults():
        with pytest.MonkeyPatch.context() as mp:
            patch(mp)
            off = plain.forward(cfg, weights, tokens).numpy()
        errors = np.array([relative_error(off[i], correct[i]) for i in range(len(tokens))])
        if errors.max() < 1e-12:
            continue
        seen += 1
        if what == "the first token's input whole":
            assert errors[0] > 1e-2, (what, errors[0])
            continue
        assert np.mean(errors > 1e-4) > 0.3, (what, float(np.mean(errors > 1e-4)))
        if what not in SMALL:
            assert np.median(errors) > 4e-2, (what, float(np.median(errors)))
    assert seen >= 16, seen


def test_plain_model_pieces():
    """The oracle's own pieces against sums written out by hand."""
    g = torch.Generator().manual_seed(1)
    x = torch.randn(4, 2, 10, generator=g, dtype=torch.float64)
    positions = torch.tensor([0, 1, 7, 4095])
    a = plain.rotate_halves(x, positions, {"dims": 8, "base": 100.0})
    assert torch.equal(a[0], x[0]) and torch.equal(a[..., 8:], x[..., 8:])
    angle = 7 * 100.0 ** (-2.0 * 1 / 8)
    u, v = x[2, 1, 1], x[2, 1, 5]
    assert torch.allclose(a[2, 1, 1], u * np.cos(angle) - v * np.sin(angle)) and torch.allclose(a[2, 1, 5], v * np.cos(angle) + u * np.sin(angle))
    # the ramp by hand: 16 dimensions of base 100, 64 positions: pair i turns 64 * 100^(-i/8) / 2 pi times
    f, amplitude = plain.yarn(rot(16, 100.0, (4.0, 64, 6.0, 1.0)))
    turns = [64.0 * 100.0 ** (-i / 8) / (2 * math.pi) for i in range(8)]
    lo, hi = max(i for i in range(8) if turns[i] >= 6.0), min(i for i in range(8) if turns[i] <= 1.0)
    for i in range(8):
        share = min(max((i - lo) / (hi - lo), 0.0), 1.0)
        assert f[i] == pytest.approx(100.0 ** (-i / 8) * (1.0 - share + share / 4.0))
    assert amplitude == pytest.approx(1.0 + 0.1 * math.log(4.0)) and 0 <= lo < hi < 7
    # attention by hand: one layer, three tokens
    m = attention(4, 2, 6, 0.9, rot(2, 10.0, (2.0, 16, 4.0, 1.0)), softcap=2.0)["mixer"]
    w = {"q": torch.randn(24, 8, generator=g, dtype=torch.float64), "k": torch.randn(12, 8, generator=g, dtype=torch.float64),
         "o": torch.randn(8, 24, generator=g, dtype=torch.float64)}
    h = torch.randn(3, 8, generator=g, dtype=torch.float64)
    rate, amp = plain.yarn(m["rot"])

    def prepared(vector, position):
        c, s = math.cos(position * rate[0]) * amp, math.sin(position * rate[0]) * amp
        turned = [vector[0] * c - vector[1] * s, vector[1] * c + vector[0] * s] + list(vector[2:])
        length = math.sqrt(sum(float(e) ** 2 for e in turned) / 6 + 1e-5)
        return [float(e) / length for e in turned]

    rows = []
    for i in range(3):
        heads = []
        for a in range(4):
            q = prepared((w["q"] @ h[i])[a * 6 : a * 6 + 6], i)
            e = []
            for j in range(i + 1):
                k = prepared((w["k"] @ h[j])[(a // 2) * 6 : (a // 2) * 6 + 6], j)
                e.append(math.exp(2.0 * math.tanh(sum(x * y for x, y in zip(q, k)) * 0.9 / 2.0)))
            heads.append(sum(e[j] * (w["k"] @ h[j])[(a // 2) * 6 : (a // 2) * 6 + 6] for j in range(i + 1)) / sum(e))
        rows.append(w["o"] @ torch.cat(heads))
    assert torch.allclose(plain.attention(h, w, m, 1e-5), torch.stack(rows), atol=1e-9)
    # the recurrence by hand, two channels
    u = torch.tensor([[1.0, -2.0], [0.5, 3.0]], dtype=torch.float64)
    r, i = torch.tensor([[0.3, 0.9], [0.6, 0.1]], dtype=torch.float64), torch.tensor([[0.5, 0.25], [1.0, 0.75]], dtype=torch.float64)
    lam = torch.tensor([-3.0, 0.5], dtype=torch.float64)
    S = [0.0, 0.0]
    want = []
    for t in range(2):
        for c in range(2):
            decay = math.exp(-8.0 * float(r[t, c]) * math.log(1.0 + math.exp(float(lam[c]))))
            S[c] = decay * S[c] + math.sqrt(1.0 - decay ** 2) * float(i[t, c]) * float(u[t, c])
        want.append(list(S))
    assert torch.allclose(plain.gated_linear_recurrence(u, r, i, lam), torch.tensor(want, dtype=torch.float64))
    taps = torch.tensor([[1.0, 10.0, 100.0]], dtype=torch.float64)
    conv = plain.short_convolution(torch.tensor([[1.0], [2.0], [3.0], [4.0]], dtype=torch.float64), taps, torch.tensor([0.5], dtype=torch.float64))
    assert conv.flatten().tolist() == [100.5, 210.5, 321.5, 432.5]
    # a prefix of a sequence gives the whole sequence's rows
    cfg = config(24, 19, [layer(attention(2, 1, 8, 0.8, rot(4, 20.0), softcap=4.0), 10), layer(rglru(16, 2, 3), None), layer(latent(2, 6, 4, 6, 10, 0.6), None)])
    weights = make_weights(cfg, 5)
    tokens = traces.make_requests(19, [20], seed=2)["r0"]
    whole = plain.forward(cfg, weights, tokens)
    for cut in (1, 7, 19):
        assert torch.allclose(plain.forward(cfg, weights, tokens[:cut]), whole[:cut], atol=1e-9)


# ---------------------------------------------------------------------------- the engine on the CPU
# The kernels replaced by their torch statements (rezelix_torch_kernels.py): the cache manager's pages and states, the step function,
# the scheduler and the command line as this design drives them, in 32-bit.  The same workloads run on the GPU with the kernels.

SHORT = [33, 12, 40, 9, 2, 1, 27]


def cpu_runner(folder, *, page_size, num_pages, max_requests=4):
    from kairyu_b200.cache import CacheStorage
    from kairyu_b200.engine.engine import load_model
    from kairyu_b200.engine.runner import ModelRunner

    model, _ = load_model(folder, dtype="float32", device="cpu")
    layout = CacheLayout.from_slot_specs(model.cache_slot_specs())
    cache = CacheManager(layout, num_pages=num_pages, page_size=page_size, max_requests=max_requests)
    storage = CacheStorage(layout, num_pages=num_pages, page_size=page_size, max_requests=max_requests, dtype=model.dtype, device="cpu")
    return ModelRunner(model, cache, storage, max_model_len=512, decode_mode="eager", check_tables=True, debug_poison=True)


@pytest.mark.parametrize("name", ["mixed", "odd", "small_pages"])
def test_every_cut_on_the_cpu(name, tmp_path, monkeypatch):
    import rezelix_torch_kernels

    rezelix_torch_kernels.install(monkeypatch)
    cfg, seed, page_size = CASES[name]
    weights = make_weights(cfg, seed)
    folder = write_model(cfg, weights, tmp_path / "m")
    requests = traces.make_requests(cfg["vocab"], SHORT, seed=3)
    expected = {n: plain.forward(cfg, weights, t).numpy() for n, t in requests.items()}
    cuts = {
        "whole": traces.trace_whole(requests),
        "tail": traces.trace_decode_tail(requests, 9),
        "chunks": traces.trace_chunks(requests, sizes=(5, 2, 11, 3)),
        "mixed": traces.trace_mixed(requests, seed=4, max_live=3),
    }
    pool = max(traces.peak_tokens(steps, round_to=page_size) for steps in cuts.values()) // page_size + 1
    runner = cpu_runner(folder, page_size=page_size, num_pages=pool, max_requests=3)
    for cut, steps in cuts.items():
        result = traces.run_in_process(runner, steps)
        assert len(result) == sum(SHORT)
        worst = max(relative_error(row, expected[n][p]) for (n, p), row in result.items())
        assert worst < 1e-4, (cut, worst)
        assert runner.cache.live_requests == 0
        runner.cache.check()


def test_generation_and_the_command_line_on_the_cpu(tmp_path, capsys, monkeypatch):
    """make-random, validate, generate: greedy tokens through the scheduler (a token budget that cuts the prompts) equal the
    plain model's own continuation."""
    import rezelix_torch_kernels
    from safetensors.torch import load_file

    from kairyu_b200.entrypoints import cli

    rezelix_torch_kernels.install(monkeypatch)
    cfg = CASES["mixed"][0]
    (tmp_path / "config.json").write_text(json.dumps(cfg))
    folder = tmp_path / "model"
    cli.main(["make-random", str(tmp_path / "config.json"), str(folder), "--seed", "5", "--dtype", "float32"])
    cli.main(["validate", str(folder)])
    assert "valid: Rezelix, 6 layers" in capsys.readouterr().out
    prompts = [[5, 17, 3, 9], [1], list(range(20, 60))]
    cli.main(["generate", str(folder), "--dtype", "float32", "--device", "cpu", "--temperature", "0", "--max-tokens", "6", "--num-pages", "24",
              "--page-size", "8", "--max-num-seqs", "2", "--max-num-batched-tokens", "16"]
             + [arg for p in prompts for arg in ("--prompt-token-ids", ",".join(map(str, p)))])
    lines = [json.loads(line) for line in capsys.readouterr().out.splitlines() if line.startswith("{")]
    weights = {n: t.float() for n, t in load_file(str(folder / "model.safetensors")).items()}
    for prompt, line in zip(prompts, lines):
        tokens = list(prompt)
        for _ in range(6):
            tokens.append(int(plain.forward(cfg, weights, tokens)[-1].argmax()))
        assert line["outputs"][0]["token_ids"] == tokens[len(prompt):]


def test_bench_configurations_build():
    """bench.py --design rezelix: the three models build and have about the same bytes."""
    import bench_rezelix

    for size in bench_rezelix.SIZES.values():
        models = [build_model(make(size), dtype="bfloat16", device="meta")[0]
                  for make in (bench_rezelix.rezelix_config, bench_rezelix.tapasun_config, bench_rezelix.dense_config)]
        assert all(len(model.schedule) == bench_rezelix.LAYERS for model in models)
        counts = [sum(math.prod(spec.shape) for spec in model.tensor_specs()) for model in models]
        assert all(0.85 < counts[0] / other < 1.18 for other in counts[1:]), counts
