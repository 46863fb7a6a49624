"""Typed configuration of the Sapanex decoder, read from config.json.

The file is nested: `architecture` (the name), `vocab`, `width`, `norm.eps`, `embedding.scale` (absent: one),
`postln_alpha` (what the stream is multiplied by before a sublayer's output joins it), and `layers`, one object
per layer: `type` = "attention" or "general_delta", `mixer` with that mixer's sizes and constants, `mlp` (`kind`
"dense", `ff`) or null.

  attention        heads, kv_heads, dim, vdim, scale; rot (base, dims, and optionally scaling: factor, original,
                   fast, slow); mask (size: tokens a position sees, pool: tokens of a pooled block before them)
  general_delta    heads, dim

Every size and constant comes from the file (the inner size of the recurrence's decay map from the stored tensor);
a key that is absent means the mechanism is absent.
"""
from __future__ import annotations

from dataclasses import asdict, dataclass
from typing import Any, Mapping, Optional, Tuple, Union

from .errors import ConfigError, UnsupportedConfig
from .sufolix import DEFAULT_MAX_POSITIONS, MAX_LAYERS, _int, _num, _obj


@dataclass(frozen=True)
class RampScaling:
    factor: float
    original: float
    fast: float
    slow: float


@dataclass(frozen=True)
class Rotation:
    base: float
    dims: int
    scaling: Optional[RampScaling]


@dataclass(frozen=True)
class PooledWindow:
    size: int
    pool: int


@dataclass(frozen=True)
class AttentionMixer:
    heads: int
    kv_heads: int
    dim: int                 # head size of queries and keys
    vdim: int                # head size of values
    scale: float             # multiplier of q.k
    rot: Optional[Rotation]
    mask: Optional[PooledWindow]

    @classmethod
    def from_dict(cls, d: Any, what: str) -> "AttentionMixer":
        d = _obj(d, what)
        heads, kv = _int(d, "heads", what), _int(d, "kv_heads", what)
        dim, vdim = _int(d, "dim", what), _int(d, "vdim", what)
        if heads % kv:
            raise ConfigError(f"config.json: {what}: {heads} heads are not a multiple of {kv} kv_heads")
        if max(dim, vdim) > 512:
            raise UnsupportedConfig(f"config.json: {what}: head sizes beyond 512 are not served")
        rot = None
        if d.get("rot") is not None:
            r = _obj(d["rot"], what + ".rot")
            dims, base = _int(r, "dims", what + ".rot"), _num(r, "base", what + ".rot")
            if dims % 2 or dims > dim:
                raise ConfigError(f"config.json: {what}.rot.dims must be even and at most dim, found {dims}")
            if vdim % 2:
                raise ConfigError(f"config.json: {what}.vdim must be even where values are rotated, found {vdim}")
            if base <= 0:
                raise ConfigError(f"config.json: {what}.rot.base must be positive")
            scaling = None
            if r.get("scaling") is not None:
                s = _obj(r["scaling"], what + ".rot.scaling")
                scaling = RampScaling(*(_num(s, k, what + ".rot.scaling") for k in ("factor", "original", "fast", "slow")))
                if min(scaling.factor, scaling.original, scaling.fast, scaling.slow) <= 0 or base == 1.0:
                    raise ConfigError(f"config.json: {what}.rot.scaling: factor, original, fast and slow must be positive, and base not one")
            rot = Rotation(base, dims, scaling)
        mask = None
        if d.get("mask") is not None:
            m = _obj(d["mask"], what + ".mask")
            mask = PooledWindow(_int(m, "size", what + ".mask"), _int(m, "pool", what + ".mask"))
        return cls(heads, kv, dim, vdim, _num(d, "scale", what), rot, mask)


@dataclass(frozen=True)
class DeltaMixer:
    heads: int
    dim: int                 # rows and columns of a head's state

    @classmethod
    def from_dict(cls, d: Any, what: str) -> "DeltaMixer":
        d = _obj(d, what)
        out = cls(_int(d, "heads", what), _int(d, "dim", what))
        if out.dim > 256:
            raise UnsupportedConfig(f"config.json: {what}.dim: a state of more than 256 rows is not served")
        return out


@dataclass(frozen=True)
class SapanexLayer:
    type: str                # "attention" | "general_delta"
    mixer: Union[AttentionMixer, DeltaMixer]
    ff: int                  # 0: no feed-forward


@dataclass(frozen=True)
class SapanexConfig:
    vocab: int
    width: int
    eps: float
    embedding_scale: float
    alpha: float
    layers: Tuple[SapanexLayer, ...]
    max_positions: int = DEFAULT_MAX_POSITIONS

    def to_dict(self) -> dict:
        return asdict(self)

    @classmethod
    def from_dict(cls, raw: Mapping[str, Any]) -> "SapanexConfig":
        raw = _obj(raw, "the file")
        layers_raw = raw.get("layers")
        if not isinstance(layers_raw, (list, tuple)) or not layers_raw:
            raise ConfigError("config.json: layers must be a non-empty list")
        if len(layers_raw) > MAX_LAYERS:
            raise ConfigError("config.json: invalid layer count")
        layers = []
        for i, entry in enumerate(layers_raw):
            what = f"layers[{i}]"
            entry = _obj(entry, what)
            kind = entry.get("type")
            if kind == "attention":
                mixer = AttentionMixer.from_dict(entry.get("mixer"), what + ".mixer")
            elif kind == "general_delta":
                mixer = DeltaMixer.from_dict(entry.get("mixer"), what + ".mixer")
            else:
                raise UnsupportedConfig(f"config.json: {what}.type {kind!r} is not served (attention, general_delta)")
            ff = 0
            if entry.get("mlp") is not None:
                m = _obj(entry["mlp"], what + ".mlp")
                if m.get("kind") != "dense":
                    raise UnsupportedConfig(f"config.json: {what}.mlp.kind {m.get('kind')!r} is not served (dense)")
                ff = _int(m, "ff", what + ".mlp")
            layers.append(SapanexLayer(kind, mixer, ff))
        eps = _num(_obj(raw.get("norm"), "norm"), "eps", "norm")
        if eps <= 0:
            raise ConfigError("config.json: norm.eps must be positive")
        scale = _num(_obj(raw["embedding"], "embedding"), "scale", "embedding") if raw.get("embedding") is not None else 1.0
        max_positions = raw.get("max_positions", DEFAULT_MAX_POSITIONS)
        if isinstance(max_positions, bool) or not isinstance(max_positions, int) or max_positions <= 0:
            raise ConfigError("config.json: max_positions must be a positive integer")
        return cls(_int(raw, "vocab", "the file"), _int(raw, "width", "the file"), eps, scale, _num(raw, "postln_alpha", "the file"),
                   tuple(layers), max_positions)
