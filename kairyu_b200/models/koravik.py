"""Koravik: a decoder of pre-norm layers whose sub-layers' results are gated element by element, a run of which loops over
the same weights and is fed the embedding output anew on every pass.

``x0 = N(embed[token])`` and ``x = x0`` (N: an RMS norm).  A layer is ``h = norm1(x); x += m * sigmoid(R1 h + b1) * mixer(h)``,
then the same with ``norm2``, ``R2``, ``b2`` and the feed-forward (``kairyu_b200/parts/block.py``: ``gated_residual``), ``m`` one
constant of the model.  ``loop: {start, stop, times}``: layers start .. stop - 1 run ``times`` times in a row, and right before
the first layer of every pass ``x <- W_in [x; x0]`` (``kairyu_b200/parts/stream_map.py``); every pass has a cache of its own,
which in the spec is one ``LayerSpec`` named by several ``LayerCall`` entries with different cache slots.

The mixer is grouped-query attention with rotary positions on the leading ``rot.dims`` columns of queries and keys, values that
are the keys before their turn, scores mixed over the heads by a matrix before the softmax, and a sliding window that always
keeps the sequence's first tokens (``kairyu_b200/parts/talking_attention.py``).  The feed-forward is a mixture of ungated
relu-squared experts chosen by the largest sigmoid scores, weighted by the chosen scores divided by their sum, beside an
optional shared expert (``kairyu_b200/parts/moe.py``), or absent.  The logits are the embedding table's products with the
normed stream, times a constant.

config.json keys::

    architecture: "Koravik"    vocab, width    norm: {eps}    residual_mult    logit_scale    loop?: {start, stop, times}
    layers: [ {type: "attention", mixer: {...}, mlp: {...} | null}, ... ]
      mixer: heads, kv_heads, dim, vdim (= dim: a value is a key), scale, rot?: {base, dims}, mask?: {size, keep_first?}
      mlp:   kind: "moe", expert: {ff}, router: {experts, top}, shared?: {ff}

Tensors: ``embed``, ``embed.norm``, ``loop.in``, ``l<i>.norm1``, ``l<i>.mix.{q,k,talk,o}``, ``l<i>.rg1`` (+ ``.b``), and with a
feed-forward ``l<i>.norm2``, ``l<i>.mlp.{router,e<n>.{up,down},shared.{up,down}}``, ``l<i>.rg2`` (+ ``.b``), ``final.norm``
(matrices stored [out, in]).  The file names no length limit; the engine needs one to size its rotary tables and takes
``max_positions`` if the file gives it, else ``DEFAULT_MAX_POSITIONS``.
"""

from __future__ import annotations

from dataclasses import dataclass, field
from typing import Any, Mapping, Optional

from kairyu_b200.config.model_config import ConfigError
from kairyu_b200.parts.base import LayerCall, LayerSpec, ModelSpec, PartSpec

DEFAULT_MAX_POSITIONS = 131072


@dataclass(frozen=True)
class KoravikLayer:
    mixer: Mapping[str, Any]
    mlp: Optional[Mapping[str, Any]]


@dataclass(frozen=True)
class KoravikConfig:
    architecture: str
    vocab_size: int
    hidden_size: int
    norm_eps: float
    residual_mult: float
    logit_scale: float
    layers: tuple[KoravikLayer, ...]
    loop: Optional[tuple[int, int, int]]  # (start, stop, times)
    max_position_embeddings: int
    eos_token_ids: tuple[int, ...] = ()
    raw: Mapping[str, Any] = field(default_factory=dict, compare=False, repr=False)

    def run_order(self) -> list[tuple[int, bool]]:
        """(layer index, whether a pass of the loop begins with it) in the order the layers run."""
        count = len(self.layers)
        if self.loop is None:
            return [(index, False) for index in range(count)]
        start, stop, times = self.loop
        one_pass = [(index, index == start) for index in range(start, stop)]
        return [(index, False) for index in range(start)] + one_pass * times + [(index, False) for index in range(stop, count)]


def _get(table: Any, key: str, where: str) -> Any:
    if not isinstance(table, Mapping) or key not in table or table[key] is None:
        raise ConfigError(f"config.json: {where} is missing {key!r}")
    return table[key]


def _size(table: Any, key: str, where: str) -> int:
    value = _get(table, key, where)
    if type(value) is not int or value < 1:
        raise ConfigError(f"config.json: {where}.{key} must be an integer >= 1, got {value!r}")
    return value


def _real(table: Any, key: str, where: str) -> float:
    value = _get(table, key, where)
    if isinstance(value, bool) or not isinstance(value, (int, float)):
        raise ConfigError(f"config.json: {where}.{key} must be a number, got {value!r}")
    return float(value)


def _parse_rot(rot: Any, dim: int, where: str) -> Optional[tuple[float, int]]:
    if rot is None:
        return None
    dims = _size(rot, "dims", where)
    if dims % 2:
        raise ConfigError(f"config.json: {where}.dims must be even, got {dims}")
    if dims > dim:
        raise ConfigError(f"config.json: {where}.dims={dims} of dim={dim} columns a head")
    base = _real(rot, "base", where)
    if base <= 0.0:
        raise ConfigError(f"config.json: {where}.base must be positive, got {base!r}")
    return base, dims


def _parse_mask(mask: Any, where: str) -> tuple[Optional[int], int]:
    """(window, kept first tokens); no mask: every key stays in sight."""
    if mask is None:
        return None, 0
    keep = mask.get("keep_first", 0) if isinstance(mask, Mapping) else 0
    if keep is None:
        keep = 0
    if type(keep) is not int or keep < 0:
        raise ConfigError(f"config.json: {where}.keep_first must be an integer >= 0, got {keep!r}")
    return _size(mask, "size", where), keep


def _parse_mixer(kind: Any, mixer: Any, where: str) -> dict[str, Any]:
    if kind != "attention":
        raise ConfigError(f"config.json: {where}: unknown layer type {kind!r} (attention)")
    heads, kv_heads, dim = _size(mixer, "heads", where), _size(mixer, "kv_heads", where), _size(mixer, "dim", where)
    if heads % kv_heads:
        raise ConfigError(f"config.json: {where}: heads={heads} is not a multiple of kv_heads={kv_heads}")
    if mixer.get("vdim") is not None and _size(mixer, "vdim", where) != dim:
        raise ConfigError(f"config.json: {where}: vdim={mixer['vdim']} differs from dim={dim}, but a value is the key as projected")
    window, keep_first = _parse_mask(mixer.get("mask"), f"{where}.mask")
    return dict(heads=heads, kv_heads=kv_heads, dim=dim, scale=_real(mixer, "scale", where), rot=_parse_rot(mixer.get("rot"), dim, f"{where}.rot"),
                window=window, keep_first=keep_first)


def _parse_mlp(mlp: Any, where: str) -> Optional[dict[str, Any]]:
    if mlp is None:
        return None
    kind = _get(mlp, "kind", where)
    if kind != "moe":
        raise ConfigError(f"config.json: {where}: unknown feed-forward kind {kind!r} (moe)")
    router = _get(mlp, "router", where)
    shared = mlp.get("shared")
    parsed = dict(experts=_size(router, "experts", f"{where}.router"), top=_size(router, "top", f"{where}.router"),
                  ff=_size(_get(mlp, "expert", where), "ff", f"{where}.expert"),
                  shared_ff=_size(shared, "ff", f"{where}.shared") if shared is not None else None)
    if parsed["top"] > parsed["experts"]:
        raise ConfigError(f"config.json: {where}: top={parsed['top']} of {parsed['experts']} experts")
    return parsed


def _parse_loop(loop: Any, count: int) -> Optional[tuple[int, int, int]]:
    if loop is None:
        return None
    values = []
    for key in ("start", "stop", "times"):
        value = _get(loop, key, "loop")
        if type(value) is not int or value < 0:
            raise ConfigError(f"config.json: loop.{key} must be an integer >= 0, got {value!r}")
        values.append(value)
    start, stop, times = values
    if not start <= stop <= count:
        raise ConfigError(f"config.json: loop runs layers {start} .. {stop - 1} of {count}")
    if times < 1 and start != stop:
        raise ConfigError(f"config.json: loop.times must be >= 1, got {times}")
    return (start, stop, times) if start != stop else None


def parse_koravik(config: Mapping[str, Any]) -> KoravikConfig:
    entries = _get(config, "layers", "the file")
    if not isinstance(entries, list) or not entries:
        raise ConfigError("config.json: layers must be a non-empty list")
    layers = []
    for index, entry in enumerate(entries):
        where = f"layers[{index}]"
        mixer = _get(entry, "mixer", where)
        layers.append(KoravikLayer(_parse_mixer(_get(entry, "type", where), mixer, f"{where}.mixer"), _parse_mlp(entry.get("mlp"), f"{where}.mlp")))
    limit = config.get("max_positions", DEFAULT_MAX_POSITIONS)
    if type(limit) is not int or limit < 1:
        raise ConfigError(f"config.json: max_positions must be an integer >= 1, got {limit!r}")
    eos = config.get("eos_token_id")
    return KoravikConfig(
        architecture="Koravik",
        vocab_size=_size(config, "vocab", "the file"),
        hidden_size=_size(config, "width", "the file"),
        norm_eps=_real(_get(config, "norm", "the file"), "eps", "norm"),
        residual_mult=_real(config, "residual_mult", "the file"),
        logit_scale=_real(config, "logit_scale", "the file"),
        layers=tuple(layers),
        loop=_parse_loop(config.get("loop"), len(layers)),
        max_position_embeddings=limit,
        eos_token_ids=(eos,) if type(eos) is int else tuple(eos) if isinstance(eos, list) else (),
        raw=dict(config),
    )


def _layer_spec(index: int, layer: KoravikLayer, config: KoravikConfig) -> LayerSpec:
    prefix = f"l{index}"
    width, eps = config.hidden_size, config.norm_eps
    m = layer.mixer
    position = None
    if m["rot"] is not None:
        base, dims = m["rot"]
        # angles are formed in 64-bit and rounded once: every table entry is the correctly rounded cosine or sine
        position = PartSpec("rope", rotary_dim=dims, theta=base, scaling=None, max_positions=config.max_position_embeddings, wide_angles=True)
    mixer = PartSpec(
        "talking_attention", prefix=f"{prefix}.mix", hidden_size=width, num_heads=m["heads"], num_kv_heads=m["kv_heads"], head_dim=m["dim"],
        scale=m["scale"], position=position, window=m["window"], keep_first=m["keep_first"], values="keys",
    )
    ffn = None
    if layer.mlp is not None:
        f = layer.mlp
        ffn = PartSpec(
            "moe", prefix=f"{prefix}.mlp", hidden_size=width, intermediate_size=f["ff"], num_experts=f["experts"], top=f["top"], routing="scores",
            score_function="sigmoid", correction=False, renormalise=True, router_bias=False, activation="relu2",
            shared_expert=dict(intermediate_size=f["shared_ff"]) if f["shared_ff"] is not None else None,
        )
    return LayerSpec(
        prefix=prefix, block="gated_residual", mixer=mixer, ffn=ffn,
        mixer_norm=PartSpec("rmsnorm", name=f"{prefix}.norm1", size=width, eps=eps),
        ffn_norm=PartSpec("rmsnorm", name=f"{prefix}.norm2", size=width, eps=eps) if ffn is not None else None,
        options={"gate_names": (f"{prefix}.rg1", f"{prefix}.rg2"), "residual_mult": config.residual_mult},
    )


def koravik_spec(config: KoravikConfig) -> ModelSpec:
    specs = tuple(_layer_spec(index, layer, config) for index, layer in enumerate(config.layers))
    # every run of a layer, a looped one each time, is a call with a cache slot of its own
    schedule = tuple(LayerCall(layer=index, cache_slot=slot, remaps_stream=begins) for slot, (index, begins) in enumerate(config.run_order()))
    width, eps = config.hidden_size, config.norm_eps
    looped = config.loop is not None
    return ModelSpec(
        embedding=PartSpec("token_embedding", name="embed", vocab_size=config.vocab_size, hidden_size=width,
                           norm=PartSpec("rmsnorm", name="embed.norm", size=width, eps=eps), keep_origin=looped),
        layers=specs,
        schedule=schedule,
        stream_map=PartSpec("origin_concat", name="loop.in", hidden_size=width) if looped else None,
        # the factor on the logits rides on the last norm's weight: logits = embed . (N(x) * logit_scale)
        final_norm=PartSpec("rmsnorm", name="final.norm", size=width, eps=eps, gain=config.logit_scale),
        head=PartSpec("linear_head", name="head", vocab_size=config.vocab_size, hidden_size=width, tied_to="embed"),
        vocab_size=config.vocab_size,
        hidden_size=width,
        max_position_embeddings=config.max_position_embeddings,
    )
