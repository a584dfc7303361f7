"""Rezelix: a pre-norm decoder whose layers are listed one by one in ``config.json`` and whose sub-layers' results are scaled
column by column as they join the stream.

``x = N(embed[token])`` (N: an RMS norm).  A layer is ``x += s1 * mixer(norm1(x))``, then, unless its ``mlp`` is null,
``x += s2 * ff(norm2(x))``, s1 and s2 a factor a column (``kairyu_b200/parts/block.py``: ``pre_norm`` with ``scale_names``).
The mixer of a layer is

* ``attention``: grouped-query attention with rotary positions on the leading ``rot.dims`` columns of every head (pairs
  (i, i + dims/2)), queries and keys divided by their root mean square behind the rotation, values that are the keys as
  projected, and a soft cap on the scores (``kairyu_b200/parts/gated_attention.py``);
* ``latent_attention``: attention over one cached latent row a token plus one rotated key part that all heads share, with a
  sigmoid output gate (``kairyu_b200/parts/latent_attention.py``);
* ``rglru``: a recurrent block around a real-gated linear recurrent unit (``kairyu_b200/parts/rglru.py``).

The feed-forward is ``down(silu(gate h) * (up h))`` or absent.  ``logits = head N(x)``.

config.json keys::

    architecture: "Rezelix"    vocab, width    norm: {eps}
    layers: [ {type, mixer: {...}, mlp: {kind: "dense", ff} | null}, ... ]
      attention mixer:        heads, kv_heads, dim, vdim (= dim: a value is a key), scale, softcap?, rot?: {base, dims, scaling?}
      latent_attention mixer: heads, dim, rot_dim, vdim, kv_rank, scale, rot: {base, dims, scaling?}     (dims = rot_dim)
      rglru mixer:            width, blocks, conv
      rot.scaling:            {factor, original, fast, slow}: pairs that turn more than ``fast`` times within ``original`` positions
                              keep their frequency, those that turn less than ``slow`` times are slowed ``factor`` times, the
                              pairs between are blended; cosine and sine grow by 0.1 ln(factor) + 1

Tensors: ``embed``, ``embed.norm``, ``l<i>.norm1``, ``l<i>.ls1``, ``l<i>.mix.{q,k,o}``, ``l<i>.mix.{q,dkv,dkv.norm,uk,uv,g,o}`` or
``l<i>.mix.{y,y.b,x,x.b,conv,conv.b,ra,ra.b,ri,ri.b,lam,o}``, with a feed-forward ``l<i>.norm2``, ``l<i>.ls2``,
``l<i>.mlp.{gate,up,down}``, ``final.norm``, ``head`` (matrices stored [out, in]).  The file names no length limit; the engine
needs one to size its rotary tables and takes ``max_positions`` if the file gives it, else ``DEFAULT_MAX_POSITIONS``.
"""

from __future__ import annotations

import math
from dataclasses import dataclass, field
from typing import Any, Mapping, Optional

from kairyu_b200.config.model_config import ConfigError, RopeScaling
from kairyu_b200.parts.base import LayerCall, LayerSpec, ModelSpec, PartSpec

DEFAULT_MAX_POSITIONS = 131072


@dataclass(frozen=True)
class RezelixLayer:
    kind: str  # "attention" | "latent_attention" | "rglru"
    mixer: Mapping[str, Any]
    mlp: Optional[Mapping[str, Any]]


@dataclass(frozen=True)
class RezelixConfig:
    architecture: str
    vocab_size: int
    hidden_size: int
    norm_eps: float
    layers: tuple[RezelixLayer, ...]
    max_position_embeddings: int
    eos_token_ids: tuple[int, ...] = ()
    raw: Mapping[str, Any] = field(default_factory=dict, compare=False, repr=False)


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


def _positive(table: Any, key: str, where: str) -> float:
    value = _real(table, key, where)
    if value <= 0.0:
        raise ConfigError(f"config.json: {where}.{key} must be positive, got {value!r}")
    return value


def _parse_rot(rot: Any, columns: int, where: str) -> dict[str, Any]:
    dims = _size(rot, "dims", where)
    if dims % 2 or dims > columns:
        raise ConfigError(f"config.json: {where}.dims must be even and at most {columns}, got {dims}")
    base = _positive(rot, "base", where)
    scaling = rot.get("scaling")
    if scaling is not None:
        place = f"{where}.scaling"
        if base == 1.0:
            raise ConfigError(f"config.json: {where}.base must not be 1 where frequencies are scaled")
        scaling = dict(factor=_positive(scaling, "factor", place), original=_positive(scaling, "original", place),
                       fast=_positive(scaling, "fast", place), slow=_positive(scaling, "slow", place))
    return dict(base=base, dims=dims, scaling=scaling)


def _parse_mixer(kind: Any, mixer: Any, where: str) -> dict[str, Any]:
    if kind == "attention":
        heads, kv_heads, dim = _size(mixer, "heads", where), _size(mixer, "kv_heads", where), _size(mixer, "dim", where)
        if heads % kv_heads:
            raise ConfigError(f"config.json: {where}: heads={heads} is not a multiple of kv_heads={kv_heads}")
        if mixer.get("vdim") is not None and _size(mixer, "vdim", where) != dim:
            raise ConfigError(f"config.json: {where}: vdim={mixer['vdim']} differs from dim={dim}, but a value is the key as projected")
        return dict(heads=heads, kv_heads=kv_heads, dim=dim, scale=_positive(mixer, "scale", where),
                    softcap=_positive(mixer, "softcap", where) if mixer.get("softcap") is not None else None,
                    rot=_parse_rot(mixer["rot"], dim, f"{where}.rot") if mixer.get("rot") is not None else None)
    if kind == "latent_attention":
        rot_dim = _size(mixer, "rot_dim", where)
        rot = _parse_rot(_get(mixer, "rot", where), rot_dim, f"{where}.rot")
        if rot["dims"] != rot_dim:
            raise ConfigError(f"config.json: {where}.rot.dims={rot['dims']} differs from rot_dim={rot_dim}: the rotated part turns as a whole")
        return dict(heads=_size(mixer, "heads", where), dim=_size(mixer, "dim", where), rot_dim=rot_dim, vdim=_size(mixer, "vdim", where),
                    kv_rank=_size(mixer, "kv_rank", where), scale=_positive(mixer, "scale", where), rot=rot)
    if kind == "rglru":
        width, blocks = _size(mixer, "width", where), _size(mixer, "blocks", where)
        if width % blocks:
            raise ConfigError(f"config.json: {where}: width={width} does not split into blocks={blocks} equal parts")
        return dict(width=width, blocks=blocks, conv=_size(mixer, "conv", where))
    raise ConfigError(f"config.json: {where}: unknown layer type {kind!r} (attention, latent_attention, rglru)")


def _parse_mlp(mlp: Any, where: str) -> Optional[dict[str, Any]]:
    if mlp is None:
        return None
    kind = _get(mlp, "kind", where)
    if kind != "dense":
        raise ConfigError(f"config.json: {where}: unknown feed-forward kind {kind!r} (dense)")
    return dict(ff=_size(mlp, "ff", where))


def parse_rezelix(config: Mapping[str, Any]) -> RezelixConfig:
    entries = _get(config, "layers", "the file")
    if not isinstance(entries, list) or not entries:
        raise ConfigError("config.json: layers must be a non-empty list")
    layers = []
    for index, entry in enumerate(entries):
        where = f"layers[{index}]"
        kind = _get(entry, "type", where)
        layers.append(RezelixLayer(kind, _parse_mixer(kind, _get(entry, "mixer", where), f"{where}.mixer"), _parse_mlp(entry.get("mlp"), f"{where}.mlp")))
    limit = config.get("max_positions", DEFAULT_MAX_POSITIONS)
    if type(limit) is not int or limit < 1:
        raise ConfigError(f"config.json: max_positions must be an integer >= 1, got {limit!r}")
    eos = config.get("eos_token_id")
    return RezelixConfig(
        architecture="Rezelix",
        vocab_size=_size(config, "vocab", "the file"),
        hidden_size=_size(config, "width", "the file"),
        norm_eps=_real(_get(config, "norm", "the file"), "eps", "norm"),
        layers=tuple(layers),
        max_position_embeddings=limit,
        eos_token_ids=(eos,) if type(eos) is int else tuple(eos) if isinstance(eos, list) else (),
        raw=dict(config),
    )


def _rope(rot: Optional[Mapping[str, Any]], limit: int) -> Optional[PartSpec]:
    if rot is None:
        return None
    scaling = None
    if rot["scaling"] is not None:
        s = rot["scaling"]
        scaling = RopeScaling(kind="yarn", factor=s["factor"], original_max_position_embeddings=s["original"], beta_fast=s["fast"],
                              beta_slow=s["slow"], amplitude=0.1 * math.log(s["factor"]) + 1.0)
    # angles are formed in 64-bit and rounded once: every table entry is the correctly rounded cosine or sine
    return PartSpec("rope", rotary_dim=rot["dims"], theta=rot["base"], scaling=scaling, max_positions=limit, wide_angles=True)


def _layer_spec(index: int, layer: RezelixLayer, config: RezelixConfig) -> LayerSpec:
    prefix = f"l{index}"
    width, eps = config.hidden_size, config.norm_eps
    m = layer.mixer
    if layer.kind == "attention":
        mixer = PartSpec(
            "gated_attention", prefix=f"{prefix}.mix", hidden_size=width, num_heads=m["heads"], num_kv_heads=m["kv_heads"], head_dim=m["dim"],
            value_dim=m["dim"], scale=m["scale"], norm_eps=eps, qk_norm="turned", position=_rope(m["rot"], config.max_position_embeddings),
            rotary_interleaved=False, sink=None, gate=False, window=None, values="keys", softcap=m["softcap"],
        )
    elif layer.kind == "latent_attention":
        mixer = PartSpec(
            "latent_attention", prefix=f"{prefix}.mix", hidden_size=width, num_heads=m["heads"], head_dim=m["dim"], value_dim=m["vdim"],
            kv_rank=m["kv_rank"], scale=m["scale"], window=None, norm_eps=eps, rot_dim=m["rot_dim"],
            position=_rope(m["rot"], config.max_position_embeddings), rotary_interleaved=False, sink=False, gate=True,
        )
    else:
        mixer = PartSpec("rglru", prefix=f"{prefix}.mix", hidden_size=width, width=m["width"], parts=m["blocks"], conv_taps=m["conv"])
    ffn = None
    if layer.mlp is not None:
        ffn = PartSpec("swiglu", prefix=f"{prefix}.mlp", hidden_size=width, intermediate_size=layer.mlp["ff"], activation="silu",
                       names=("gate", "up", "down"))
    return LayerSpec(
        prefix=prefix, block="pre_norm", mixer=mixer, ffn=ffn,
        mixer_norm=PartSpec("rmsnorm", name=f"{prefix}.norm1", size=width, eps=eps),
        ffn_norm=PartSpec("rmsnorm", name=f"{prefix}.norm2", size=width, eps=eps) if ffn is not None else None,
        options={"scale_names": (f"{prefix}.ls1", f"{prefix}.ls2")},
    )


def rezelix_spec(config: RezelixConfig) -> ModelSpec:
    width, eps = config.hidden_size, config.norm_eps
    return ModelSpec(
        embedding=PartSpec("token_embedding", name="embed", vocab_size=config.vocab_size, hidden_size=width,
                           norm=PartSpec("rmsnorm", name="embed.norm", size=width, eps=eps)),
        layers=tuple(_layer_spec(index, layer, config) for index, layer in enumerate(config.layers)),
        schedule=tuple(LayerCall(layer=index, cache_slot=index) for index in range(len(config.layers))),
        final_norm=PartSpec("rmsnorm", name="final.norm", size=width, eps=eps),
        head=PartSpec("linear_head", name="head", vocab_size=config.vocab_size, hidden_size=width, tied_to=None),
        vocab_size=config.vocab_size,
        hidden_size=width,
        max_position_embeddings=config.max_position_embeddings,
    )
