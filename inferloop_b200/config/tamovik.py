"""Typed configuration of the Tamovik decoder, read from config.json.

The file is nested: `architecture` (the name), `vocab`, `width`, `norm.eps`, `embedding.bigram` (`buckets`, `mul_prev`,
`mul_cur`: a second table chosen by the pair of the previous token and the token; absent: no such table), and `layers`,
one object per layer with `type`, `mixer` (its sizes and constants) and `mlp` (`kind` "dense" with `ff`, or "moe" with
`router` (`experts`, `top`, optional `groups` {`count`, `keep`}) and `expert` (`ff`, `limit`); or null).

  latent_attention   heads, dim (unrotated query/key size a head), rot_dim (rotated size), vdim, kv_rank, scale, rot.base,
                     rot.dims and optionally rot.scaling (factor, original, fast, slow)
  parallel           left: heads, kv_heads, dim, vdim (the same: the values are keys), conv (taps), scale and optionally
                     mask.size (aligned chunks); right: heads, dim, vdim, gate_cap

Every size and constant comes from the file; a key that is absent means the mechanism is absent.
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

    @classmethod
    def from_dict(cls, d: Any, size: int, what: str) -> "Rotation":
        d = _obj(d, what)
        dims, base = _int(d, "dims", what), _num(d, "base", what)
        if dims % 2 or dims > size:
            raise ConfigError(f"config.json: {what}.dims must be even and at most {size}, found {dims}")
        if base <= 0:
            raise ConfigError(f"config.json: {what}.base must be positive")
        scaling = None
        if d.get("scaling") is not None:
            s = _obj(d["scaling"], what + ".scaling")
            scaling = RampScaling(*(_num(s, k, what + ".scaling") for k in ("factor", "original", "fast", "slow")))
            if min(scaling.factor, scaling.original, scaling.fast, scaling.slow) <= 0 or base == 1.0:
                raise ConfigError(f"config.json: {what}.scaling: all four must be positive, and the base not one")
        return cls(base, dims, scaling)


@dataclass(frozen=True)
class LatentMixer:
    heads: int
    dim: int            # unrotated elements of a head's query and key
    rot_dim: int        # rotated elements: a head's query ends in them, the keys share one such part
    vdim: int
    kv_rank: int        # size of the cached latent
    scale: float
    rot: Optional[Rotation]

    @classmethod
    def from_dict(cls, d: Any, what: str) -> "LatentMixer":
        d = _obj(d, what)
        rot_dim = _int(d, "rot_dim", what)
        rot = None if d.get("rot") is None else Rotation.from_dict(d["rot"], rot_dim, what + ".rot")
        out = cls(_int(d, "heads", what), _int(d, "dim", what), rot_dim, _int(d, "vdim", what), _int(d, "kv_rank", what),
                  _num(d, "scale", what), rot)
        if out.kv_rank + out.rot_dim > 640 or max(out.dim, out.vdim) > 512:
            raise UnsupportedConfig(f"config.json: {what}: kv_rank + rot_dim beyond 640, or dim or vdim beyond 512, are not served")
        return out


@dataclass(frozen=True)
class ChunkedBranch:
    heads: int
    kv_heads: int
    dim: int
    conv: int                # taps of the convolution in front of the norms
    scale: float
    chunk: Optional[int]     # positions of an aligned chunk; None: every earlier key is seen

    @classmethod
    def from_dict(cls, d: Any, what: str) -> "ChunkedBranch":
        d = _obj(d, what)
        heads, kv, dim = _int(d, "heads", what), _int(d, "kv_heads", what), _int(d, "dim", what)
        if heads % kv:
            raise ConfigError(f"config.json: {what}: {heads} heads are not a multiple of {kv} kv_heads")
        if _int(d, "vdim", what) != dim:
            raise ConfigError(f"config.json: {what}: the values are keys, so vdim {d['vdim']} must be dim {dim}")
        chunk = None if d.get("mask") is None else _int(_obj(d["mask"], what + ".mask"), "size", what + ".mask")
        out = cls(heads, kv, dim, _int(d, "conv", what), _num(d, "scale", what), chunk)
        if dim > 512:
            raise UnsupportedConfig(f"config.json: {what}: head sizes beyond 512 are not served")
        if out.conv > 16:
            raise UnsupportedConfig(f"config.json: {what}.conv: more than 16 taps are not served")
        if (heads + kv) * dim > 51200:
            raise UnsupportedConfig(f"config.json: {what}: more than 51,200 channels of queries and keys are not served")
        return out


@dataclass(frozen=True)
class MatrixMemoryBranch:
    heads: int
    dim: int
    vdim: int
    gate_cap: float

    @classmethod
    def from_dict(cls, d: Any, what: str) -> "MatrixMemoryBranch":
        d = _obj(d, what)
        out = cls(_int(d, "heads", what), _int(d, "dim", what), _int(d, "vdim", what), _num(d, "gate_cap", what))
        if out.gate_cap <= 0:
            raise ConfigError(f"config.json: {what}.gate_cap must be positive")
        if out.dim > 256 or out.vdim > 8192:
            raise UnsupportedConfig(f"config.json: {what}: states of more than 256 x 8,192 are not served")
        return out


@dataclass(frozen=True)
class ParallelMixer:
    left: ChunkedBranch
    right: MatrixMemoryBranch

    @classmethod
    def from_dict(cls, d: Any, what: str) -> "ParallelMixer":
        d = _obj(d, what)
        return cls(ChunkedBranch.from_dict(d.get("left"), what + ".left"), MatrixMemoryBranch.from_dict(d.get("right"), what + ".right"))


@dataclass(frozen=True)
class DenseFeedForward:
    ff: int


@dataclass(frozen=True)
class ExpertsFeedForward:
    experts: int
    top: int
    groups: int          # 1: no groups
    keep: int
    ff: int
    limit: float


def _mlp(d: Any, what: str):
    d = _obj(d, what)
    kind = d.get("kind")
    if kind == "dense":
        return DenseFeedForward(_int(d, "ff", what))
    if kind != "moe":
        raise UnsupportedConfig(f"config.json: {what}.kind {kind!r} is not served (dense, moe)")
    r = _obj(d.get("router"), what + ".router")
    experts, top = _int(r, "experts", what + ".router"), _int(r, "top", what + ".router")
    groups, keep = 1, 1
    if r.get("groups") is not None:
        g = _obj(r["groups"], what + ".router.groups")
        groups, keep = _int(g, "count", what + ".router.groups"), _int(g, "keep", what + ".router.groups")
        if experts % groups or keep > groups:
            raise ConfigError(f"config.json: {what}.router.groups: {groups} groups (keeping {keep}) of {experts} experts")
        if groups > 32:
            raise UnsupportedConfig(f"config.json: {what}.router.groups: more than 32 groups are not served")
    if top > experts // groups * keep:
        raise ConfigError(f"config.json: {what}.router: top {top} exceeds the experts that can be chosen")
    if experts > 512 or top > 32:
        raise UnsupportedConfig(f"config.json: {what}.router: more than 512 experts or 32 a token are not served")
    e = _obj(d.get("expert"), what + ".expert")
    limit = _num(e, "limit", what + ".expert")
    if limit <= 0:
        raise ConfigError(f"config.json: {what}.expert.limit must be positive")
    return ExpertsFeedForward(experts, top, groups, keep, _int(e, "ff", what + ".expert"), limit)


@dataclass(frozen=True)
class PairTable:
    buckets: int
    mul_prev: int
    mul_cur: int


@dataclass(frozen=True)
class TamovikLayer:
    type: str            # "latent_attention" | "parallel"
    mixer: Union[LatentMixer, ParallelMixer]
    mlp: Union[DenseFeedForward, ExpertsFeedForward, None]


@dataclass(frozen=True)
class TamovikConfig:
    vocab: int
    width: int
    eps: float
    pairs: Optional[PairTable]
    layers: Tuple[TamovikLayer, ...]
    max_positions: int = DEFAULT_MAX_POSITIONS

    def to_dict(self) -> dict:
        return asdict(self)

    @classmethod
    def from_dict(cls, raw: Mapping[str, Any]) -> "TamovikConfig":
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
            if kind == "latent_attention":
                mixer = LatentMixer.from_dict(entry.get("mixer"), what + ".mixer")
            elif kind == "parallel":
                mixer = ParallelMixer.from_dict(entry.get("mixer"), what + ".mixer")
            else:
                raise UnsupportedConfig(f"config.json: {what}.type {kind!r} is not served (latent_attention, parallel)")
            mlp = entry.get("mlp")
            layers.append(TamovikLayer(kind, mixer, None if mlp is None else _mlp(mlp, what + ".mlp")))
        eps = _num(_obj(raw.get("norm"), "norm"), "eps", "norm")
        if eps <= 0:
            raise ConfigError("config.json: norm.eps must be positive")
        pairs = None
        embedding = raw.get("embedding")
        if embedding is not None and _obj(embedding, "embedding").get("bigram") is not None:
            b, what = _obj(embedding["bigram"], "embedding.bigram"), "embedding.bigram"
            muls = []
            for key in ("mul_prev", "mul_cur"):
                v = b.get(key)
                if isinstance(v, bool) or not isinstance(v, int) or not 0 <= v < 1 << 31:
                    raise ConfigError(f"config.json: {what}.{key} must be a 32-bit integer of at least zero, found {v!r}")
                muls.append(v)
            pairs = PairTable(_int(b, "buckets", what), *muls)
        max_positions = raw.get("max_positions", DEFAULT_MAX_POSITIONS)
        if isinstance(max_positions, bool) or not isinstance(max_positions, int) or max_positions <= 0:
            raise ConfigError("config.json: max_positions must be a positive integer")
        return cls(_int(raw, "vocab", "the file"), _int(raw, "width", "the file"), eps, pairs, tuple(layers), max_positions)
