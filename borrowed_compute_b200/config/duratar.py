"""Typed configuration of the Duratar decoder, read from its config.json.

The file gives the model's sizes (``vocab``, ``width``, ``streams``: the copies of the residual stream a row carries), ``norm.eps``
and a list ``layers`` whose entries differ: each names its mixer by ``type`` (``attention``: differential attention with a sliding
window that keeps a sequence's first positions, or, with ``kv_from``, the same over an earlier layer's keys and values;
``lightning``: linear attention with a constant decay a head; ``channel_delta``: the gated delta rule with a decay a key channel),
the mixer's sizes in ``mixer`` and its feed-forward in ``mlp`` (``kind`` ``dense``, or null for none).  The sizes the file does not
give, the inner widths of a ``channel_delta`` mixer's two low-rank projections, are shapes of tensors and are filled in from the
model folder (``complete_from_shapes``); a configuration written by hand states them as ``mixer.decay_rank`` and
``mixer.gate_rank``.
"""

from __future__ import annotations

import copy
from dataclasses import dataclass
from typing import Any, Dict, Mapping, Optional, Tuple

from .errors import ConfigError
from .fegidra import _num

MIXER_TYPES = ("attention", "lightning", "channel_delta")


@dataclass(frozen=True)
class FrequencyScalingConfig:
    factor: float
    low: float
    high: float
    original: int


@dataclass(frozen=True)
class DifferentialMixerConfig:
    heads: int
    kv_heads: int
    dim: int              # query/key dimensions of one map
    vdim: int
    scale: float
    diff: float
    window: int           # 0: every earlier position
    keep_first: int       # positions at a sequence's start that stay visible behind the window
    rot_dims: int         # rotated dimensions of a map (0: none)
    rot_base: float
    rot_scaling: Optional[FrequencyScalingConfig]
    kv_from: Optional[int]    # the layer whose keys and values this one reads; None: its own


@dataclass(frozen=True)
class LightningMixerConfig:
    heads: int
    dim: int
    vdim: int
    decay: Tuple[float, ...]  # one a head


@dataclass(frozen=True)
class ChannelDeltaMixerConfig:
    heads: int
    kv_heads: int
    dim: int
    vdim: int
    taps: int
    decay_rank: int
    gate_rank: int


@dataclass(frozen=True)
class DuratarLayerConfig:
    type: str
    mixer: Any            # DifferentialMixerConfig, LightningMixerConfig or ChannelDeltaMixerConfig
    ff: int               # 0: no feed-forward


def _heads(m: Mapping[str, Any], where: str) -> Tuple[int, int]:
    heads = _num(m, "heads", where)
    kv_heads = _num(m, "kv_heads", where, default=heads)
    if heads % kv_heads:
        raise ConfigError(f"config.json: '{where}.heads' ({heads}) must be a multiple of kv_heads ({kv_heads})")
    return heads, kv_heads


def _scaling(rot: Mapping[str, Any], where: str) -> Optional[FrequencyScalingConfig]:
    sc = rot.get("scaling")
    if sc is None:
        return None
    out = FrequencyScalingConfig(factor=_num(sc, "factor", where, float), low=_num(sc, "low", where, float), high=_num(sc, "high", where, float),
                                 original=int(_num(sc, "original", where, float)))
    if out.high <= out.low:
        raise ConfigError(f"config.json: '{where}.high' ({out.high}) must be more than low ({out.low})")
    return out


def _attention(m: Mapping[str, Any], where: str) -> DifferentialMixerConfig:
    heads, kv_heads = _heads(m, where)
    dim, rot, mask = _num(m, "dim", where), m.get("rot"), m.get("mask")
    rot_dims = 0 if rot is None else _num(rot, "dims", where + ".rot", positive=False)
    if rot_dims < 0 or rot_dims % 2 or rot_dims > dim:
        raise ConfigError(f"config.json: '{where}.rot.dims' ({rot_dims}) must be even, not negative and at most dim ({dim})")
    window = keep = 0
    if mask is not None:
        window = _num(mask, "size", where + ".mask")
        keep = _num(mask, "keep_first", where + ".mask", default=0, positive=False)
        if keep < 0:
            raise ConfigError(f"config.json: '{where}.mask.keep_first' must not be negative, got {keep}")
    kv_from = m.get("kv_from")
    if kv_from is not None and (isinstance(kv_from, bool) or not isinstance(kv_from, int)):
        raise ConfigError(f"config.json: '{where}.kv_from' must be the number of a layer, got {kv_from!r}")
    return DifferentialMixerConfig(
        heads=heads, kv_heads=kv_heads, dim=dim, vdim=_num(m, "vdim", where, default=dim),
        scale=_num(m, "scale", where, float, default=1.0 / float(dim) ** 0.5), diff=_num(m, "diff", where, float, positive=False),
        window=window, keep_first=keep, rot_dims=rot_dims,
        rot_base=10000.0 if rot is None else _num(rot, "base", where + ".rot", float),
        rot_scaling=None if rot is None else _scaling(rot, where + ".rot.scaling"), kv_from=kv_from)


def _lightning(m: Mapping[str, Any], where: str) -> LightningMixerConfig:
    heads, dim, decay = _num(m, "heads", where), _num(m, "dim", where), m.get("decay")
    if not isinstance(decay, (list, tuple)) or len(decay) != heads or any(isinstance(d, bool) or not isinstance(d, (int, float)) for d in decay):
        raise ConfigError(f"config.json: '{where}.decay' must be a list of {heads} numbers, one a head")
    return LightningMixerConfig(heads=heads, dim=dim, vdim=_num(m, "vdim", where, default=dim), decay=tuple(float(d) for d in decay))


def _channel_delta(m: Mapping[str, Any], where: str) -> ChannelDeltaMixerConfig:
    heads, kv_heads = _heads(m, where)
    dim = _num(m, "dim", where)
    return ChannelDeltaMixerConfig(heads=heads, kv_heads=kv_heads, dim=dim, vdim=_num(m, "vdim", where, default=dim), taps=_num(m, "conv", where),
                                   decay_rank=_num(m, "decay_rank", where), gate_rank=_num(m, "gate_rank", where))


_MIXERS = {"attention": _attention, "lightning": _lightning, "channel_delta": _channel_delta}


def _feed_forward(mlp: Any, where: str) -> int:
    if mlp is None:
        return 0
    if not isinstance(mlp, Mapping) or mlp.get("kind") != "dense":
        raise ConfigError(f"config.json: '{where}.kind' {mlp.get('kind') if isinstance(mlp, Mapping) else mlp!r} is not supported (only 'dense')")
    return _num(mlp, "ff", where)


@dataclass(frozen=True)
class DuratarConfig:
    vocab: int
    width: int
    streams: int
    norm_eps: float
    layers: Tuple[DuratarLayerConfig, ...]

    @staticmethod
    def from_dict(d: Mapping[str, Any]) -> "DuratarConfig":
        top = "config.json"
        vocab, width, streams = _num(d, "vocab", top), _num(d, "width", top), _num(d, "streams", top)
        if d.get("norm") is None:
            raise ConfigError("config.json: required key 'norm.eps' is missing")
        eps = _num(d["norm"], "eps", "norm", float)
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
            mixer = _MIXERS[entry["type"]](entry["mixer"], where + ".mixer")
            if entry["type"] == "attention" and mixer.kv_from is not None:
                j = mixer.kv_from
                owner = layers[j].mixer if 0 <= j < i else None
                if not isinstance(owner, DifferentialMixerConfig) or owner.kv_from is not None:
                    raise ConfigError(f"config.json: '{where}.mixer.kv_from' ({j}) must name an earlier attention layer with keys and values of its own")
                if (owner.kv_heads, owner.dim, owner.vdim) != (mixer.kv_heads, mixer.dim, mixer.vdim):
                    raise ConfigError(f"config.json: '{where}.mixer.kv_from' ({j}): that layer keeps {owner.kv_heads} heads of {owner.dim} and {owner.vdim}, "
                                      f"this one reads {mixer.kv_heads} of {mixer.dim} and {mixer.vdim}")
            layers.append(DuratarLayerConfig(entry["type"], mixer, _feed_forward(entry.get("mlp"), where + ".mlp")))
        return DuratarConfig(vocab=vocab, width=width, streams=streams, norm_eps=eps, layers=tuple(layers))


def complete_from_shapes(config: Mapping[str, Any], shapes: Mapping[str, Tuple[int, ...]]) -> Dict[str, Any]:
    """config.json with the sizes that only tensor shapes give filled in: a ``channel_delta`` mixer's ``decay_rank`` and ``gate_rank`` are
    the rows of its inner projections ``l<i>.mix.a1`` and ``l<i>.mix.g1``."""
    out = copy.deepcopy(dict(config))
    layers = out.get("layers")
    if not isinstance(layers, list):
        return out
    for i, entry in enumerate(layers):
        if isinstance(entry, dict) and entry.get("type") == "channel_delta" and isinstance(entry.get("mixer"), dict):
            for key, name in (("decay_rank", "a1"), ("gate_rank", "g1")):
                shape = shapes.get(f"l{i}.mix.{name}")
                if key not in entry["mixer"] and shape is not None and len(shape) == 2:
                    entry["mixer"][key] = int(shape[0])
    return out
