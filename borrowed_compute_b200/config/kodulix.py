"""Typed configuration of the Kodulix decoder, read from its config.json.

The file gives the model's sizes (``vocab``, ``width``), ``norm.eps``, ``residual_mult`` (what every sublayer's normed result is
multiplied by), ``logit_scale``, ``embedding.bigram`` (a second embedding named by two tokens) and a list ``layers`` whose entries
may differ: ``type`` ``attention`` (grouped-query attention without rotation: a bias by distance, a query temperature), the mixer's
sizes in ``mixer``, and the feed-forward in ``mlp`` (``kind`` ``moe`` with ``router``, ``expert`` and ``shared``, or null for none).
The one size the file does not give, the rows of a layer's table of distance biases, is the shape of a tensor and is filled in from
the model folder (``complete_from_shapes``); a configuration written by hand states it as ``mixer.bias_rows``.
"""

from __future__ import annotations

import copy
from dataclasses import dataclass
from typing import Any, Dict, Mapping, Optional, Tuple

from .errors import ConfigError
from .fegidra import _num

MIXER_TYPES = ("attention",)


@dataclass(frozen=True)
class BigramConfig:
    buckets: int
    mul_prev: int
    mul_cur: int


@dataclass(frozen=True)
class QueryTemperatureConfig:
    coef: float
    every: int


@dataclass(frozen=True)
class BiasedMixerConfig:
    heads: int
    kv_heads: int
    dim: int              # query/key dimensions a head
    vdim: int
    scale: float
    bias_rows: int        # buckets of distances
    bias_max: int         # the distance from which on everything falls into the last bucket
    q_temp: Optional[QueryTemperatureConfig]


@dataclass(frozen=True)
class GroupedExpertsConfig:
    experts: int
    top: int
    groups: int           # groups of neighbours among experts and identity experts together (1: none)
    keep: int
    identity: int
    ff: int
    limit: float
    shared_ff: int        # 0: no shared expert
    shared_limit: float


@dataclass(frozen=True)
class KodulixLayerConfig:
    type: str
    mixer: BiasedMixerConfig
    mlp: Optional[GroupedExpertsConfig]


def _bigram(d: Any) -> Optional[BigramConfig]:
    if d is None:
        return None
    where = "embedding.bigram"
    out = BigramConfig(buckets=_num(d, "buckets", where), mul_prev=_num(d, "mul_prev", where, positive=False), mul_cur=_num(d, "mul_cur", where, positive=False))
    for key, value in (("mul_prev", out.mul_prev), ("mul_cur", out.mul_cur)):
        if not 0 <= value < 1 << 31:
            raise ConfigError(f"config.json: '{where}.{key}' must lie within 0 .. 2^31 - 1, got {value}")
    return out


def _attention(m: Mapping[str, Any], where: str) -> BiasedMixerConfig:
    heads = _num(m, "heads", where)
    kv_heads = _num(m, "kv_heads", where, default=heads)
    if heads % kv_heads:
        raise ConfigError(f"config.json: '{where}.heads' ({heads}) must be a multiple of kv_heads ({kv_heads})")
    dim = _num(m, "dim", where)
    temp = m.get("q_temp")
    out = BiasedMixerConfig(
        heads=heads, kv_heads=kv_heads, dim=dim, vdim=_num(m, "vdim", where, default=dim), scale=_num(m, "scale", where, float, default=1.0 / float(dim) ** 0.5),
        bias_rows=_num(m, "bias_rows", where), bias_max=int(_num(m, "bias_max", where, float)),
        q_temp=None if temp is None else QueryTemperatureConfig(coef=_num(temp, "coef", where + ".q_temp", float, positive=False),
                                                                every=int(_num(temp, "every", where + ".q_temp", float))))
    if out.bias_rows < 2 or out.bias_rows % 2:
        raise ConfigError(f"config.json: '{where}': a table of distance biases has an even number of rows, at least 2, got {out.bias_rows}")
    if out.bias_max <= out.bias_rows // 2:
        raise ConfigError(f"config.json: '{where}.bias_max' ({out.bias_max}) must be more than half of the table's {out.bias_rows} rows")
    return out


def _experts(mlp: Any, where: str) -> Optional[GroupedExpertsConfig]:
    if mlp is None:
        return None
    kind = mlp.get("kind") if isinstance(mlp, Mapping) else mlp
    if kind != "moe":
        raise ConfigError(f"config.json: '{where}.kind' {kind!r} is not supported (only 'moe')")
    r, e, shared = mlp.get("router"), mlp.get("expert"), mlp.get("shared")
    experts, top = _num(r, "experts", where + ".router"), _num(r, "top", where + ".router")
    identity = _num(r, "identity", where + ".router", default=0, positive=False)
    groups, keep = 1, 1
    if r.get("groups") is not None:
        groups, keep = _num(r["groups"], "count", where + ".router.groups"), _num(r["groups"], "keep", where + ".router.groups")
    if identity < 0:
        raise ConfigError(f"config.json: '{where}.router.identity' must not be negative, got {identity}")
    if (experts + identity) % groups or keep > groups:
        raise ConfigError(f"config.json: '{where}.router.groups': {experts + identity} experts do not form {groups} equal groups of which {keep} are kept")
    if top > (experts + identity) // groups * keep or top > 16:
        raise ConfigError(f"config.json: '{where}.router.top' ({top}) is more than the {(experts + identity) // groups * keep} experts of the kept groups, or than 16")
    return GroupedExpertsConfig(
        experts=experts, top=top, groups=groups, keep=keep, identity=identity, ff=_num(e, "ff", where + ".expert"), limit=_num(e, "limit", where + ".expert", float),
        shared_ff=0 if shared is None else _num(shared, "ff", where + ".shared"),
        shared_limit=0.0 if shared is None else _num(shared, "limit", where + ".shared", float))


@dataclass(frozen=True)
class KodulixConfig:
    vocab: int
    width: int
    norm_eps: float
    residual_mult: float
    logit_scale: float
    bigram: Optional[BigramConfig]
    layers: Tuple[KodulixLayerConfig, ...]

    @staticmethod
    def from_dict(d: Mapping[str, Any]) -> "KodulixConfig":
        top = "config.json"
        vocab, width = _num(d, "vocab", top), _num(d, "width", top)
        if d.get("norm") is None:
            raise ConfigError("config.json: required key 'norm.eps' is missing")
        embedding = d.get("embedding")
        if embedding is not None and not isinstance(embedding, Mapping):
            raise ConfigError("config.json: 'embedding' must be an object")
        raw = d.get("layers")
        if not isinstance(raw, (list, tuple)) or not raw:
            raise ConfigError("config.json: 'layers' must be a non-empty list")
        layers = []
        for i, entry in enumerate(raw):
            where = f"layers[{i}]"
            if not isinstance(entry, Mapping) or entry.get("type") not in MIXER_TYPES:
                raise ConfigError(f"config.json: '{where}.type' must be one of {list(MIXER_TYPES)}, got "
                                  f"{entry.get('type') if isinstance(entry, Mapping) else entry!r}")
            if not isinstance(entry.get("mixer"), Mapping):
                raise ConfigError(f"config.json: '{where}.mixer' must be an object")
            layers.append(KodulixLayerConfig(entry["type"], _attention(entry["mixer"], where + ".mixer"), _experts(entry.get("mlp"), where + ".mlp")))
        return KodulixConfig(
            vocab=vocab, width=width, norm_eps=_num(d["norm"], "eps", "norm", float), residual_mult=_num(d, "residual_mult", top, float, default=1.0, positive=False),
            logit_scale=_num(d, "logit_scale", top, float, default=1.0, positive=False), bigram=_bigram((embedding or {}).get("bigram")), layers=tuple(layers))


def complete_from_shapes(config: Mapping[str, Any], shapes: Mapping[str, Tuple[int, ...]]) -> Dict[str, Any]:
    """config.json with the sizes that only tensor shapes give filled in: a mixer's ``bias_rows`` are the rows of ``l<i>.mix.rel``."""
    out = copy.deepcopy(dict(config))
    layers = out.get("layers")
    if not isinstance(layers, list):
        return out
    for i, entry in enumerate(layers):
        if isinstance(entry, dict) and isinstance(entry.get("mixer"), dict):
            shape = shapes.get(f"l{i}.mix.rel")
            if "bias_rows" not in entry["mixer"] and shape is not None and len(shape) == 2:
                entry["mixer"]["bias_rows"] = int(shape[0])
    return out
