"""Typed configuration of the Dubazen design, read from its own ``config.json``.

The file is nested like those of the other designs with layers of several types: ``layers`` lists the layers in order,
each with its ``type`` (which mixer: ``parallel``, ``gla`` or ``mamba1``), the mixer's sizes and constants under
``mixer`` (for ``parallel`` those of its two halves under ``left`` and ``right``) and its feed-forward under ``mlp``
(``kind`` ``moe``; null: none).  ``streams`` is the number of residual streams, ``embedding.scale`` multiplies the
embedding rows, ``norm.eps`` is the constant of every norm.  Every size and every constant that differs between models
of the design is read from the file, but for the inner width of a ``gla`` layer's decay, which the file may leave to the
shape of its tensor; nothing is assumed about how many layers of which type there are or in which order.  A key that is
not listed is ignored; a layer type, a feed-forward kind or a value that the engine does not implement is refused by name.
"""
from __future__ import annotations

from dataclasses import dataclass
from typing import Optional, Tuple

from .schema import ConfigError, Key, non_negative, positive, read_keys

ARCHITECTURE = "Dubazen"
DEFAULT_MAX_POSITIONS = 1 << 17   # the design has no position limit; the engine's block tables need one

_TOP = (
    Key("vocab", int, check=positive),
    Key("width", int, check=positive),
    Key("layers", list),
    Key("norm", object),
    Key("embedding", object, default=None, nullable=True),
    Key("streams", int, default=1, check=positive),
    Key("max_positions", int, default=DEFAULT_MAX_POSITIONS, check=positive),
)
_PARALLEL = (Key("left", object), Key("right", object), Key("left_scale", float, default=1.0),
             Key("right_scale", float, default=1.0))
_LEFT = (
    Key("heads", int, check=positive), Key("kv_heads", int, default=lambda v: v["heads"], check=positive),
    Key("dim", int, check=positive), Key("vdim", int, default=lambda v: v["dim"], check=positive), Key("scale", float),
    Key("rot", object),
)
_RIGHT = (
    Key("heads", int, check=positive), Key("dim", int, check=positive),
    Key("vdim", int, default=lambda v: v["dim"], check=positive), Key("decay", list),
)
_GLA = (
    Key("heads", int, check=positive), Key("dim", int, check=positive),
    Key("vdim", int, default=lambda v: v["dim"], check=positive), Key("tau", float, check=positive),
    Key("decay_rank", int, default=None, nullable=True, check=positive),
)
_MAMBA = (Key("inner", int, check=positive), Key("state", int, check=positive), Key("dt_rank", int, check=positive),
          Key("conv", int, check=positive))
_ROT = (Key("dims", int, check=non_negative), Key("base", float, check=positive))
_MLP = (Key("kind", str), Key("expert", object), Key("router", object), Key("shared", object, default=None, nullable=True))
_ROUTER = (Key("experts", int, check=positive), Key("top", int, check=positive))
_EXPERT = (Key("ff", int, check=positive), Key("limit", float, check=positive))


@dataclass(frozen=True)
class AttentionConfig:
    heads: int
    kv_heads: int
    dim: int
    vdim: int
    scale: float
    rot_dims: int          # 0: no rotation of queries and keys
    rot_base: float        # also the base of the values' rotation


@dataclass(frozen=True)
class LightningConfig:
    heads: int
    dim: int
    vdim: int
    decay: Tuple[float, ...]


@dataclass(frozen=True)
class ParallelConfig:
    left: AttentionConfig
    right: LightningConfig
    left_scale: float
    right_scale: float


@dataclass(frozen=True)
class GlaConfig:
    heads: int
    dim: int
    vdim: int
    tau: float
    decay_rank: Optional[int]    # None: the shape of the decay's first matrix says


@dataclass(frozen=True)
class MambaConfig:
    inner: int
    state: int
    dt_rank: int
    conv: int


@dataclass(frozen=True)
class MoeConfig:
    experts: int
    top: int
    ff: int
    limit: float
    shared_ff: int            # 0: no shared expert
    shared_limit: float


@dataclass(frozen=True)
class LayerConfig:
    type: str                 # parallel | gla | mamba1
    mixer: object
    mlp: Optional[MoeConfig]


@dataclass(frozen=True)
class DubazenConfig:
    vocab: int
    width: int
    norm_eps: float
    embedding_scale: float
    streams: int
    max_positions: int
    layers: Tuple[LayerConfig, ...]

    @classmethod
    def from_json(cls, obj: dict) -> "DubazenConfig":
        v = read_keys(obj, _TOP)
        eps = _object(v["norm"], (Key("eps", float, check=positive),), "config.json: norm")["eps"]
        scale = 1.0
        if v["embedding"] is not None:
            scale = _object(v["embedding"], (Key("scale", float, default=1.0),), "config.json: embedding")["scale"]
        layers = []
        for i, raw in enumerate(v["layers"]):
            where = f"config.json: layers[{i}]"
            lv = _object(raw, (Key("type", str), Key("mixer", object), Key("mlp", object, default=None, nullable=True)), where)
            reader = _MIXERS.get(lv["type"])
            if reader is None:
                raise ConfigError(f"{where}: layer type {lv['type']!r} is not implemented ({', '.join(_MIXERS)})")
            mlp = _mlp(lv["mlp"], where + ".mlp") if lv["mlp"] is not None else None
            layers.append(LayerConfig(lv["type"], reader(lv["mixer"], where + ".mixer"), mlp))
        if not layers:
            raise ConfigError("config.json: layers is empty")
        return cls(vocab=v["vocab"], width=v["width"], norm_eps=eps, embedding_scale=scale, streams=v["streams"],
                   max_positions=v["max_positions"], layers=tuple(layers))


def _object(raw, schema, where: str) -> dict:
    if not isinstance(raw, dict):
        raise ConfigError(f"{where}: must be an object")
    return read_keys(raw, schema, where=where)


def _left(raw, where: str) -> AttentionConfig:
    m = _object(raw, _LEFT, where)
    if m["heads"] % m["kv_heads"]:
        raise ConfigError(f"{where}: heads must be a multiple of kv_heads")
    if m["vdim"] % 2:
        raise ConfigError(f"{where}: vdim={m['vdim']}: values are rotated in pairs")
    r = _object(m["rot"], _ROT, where + ".rot")
    if r["dims"] % 2 or r["dims"] > m["dim"]:
        raise ConfigError(f"{where}.rot: dims must be even and at most {m['dim']}")
    return AttentionConfig(heads=m["heads"], kv_heads=m["kv_heads"], dim=m["dim"], vdim=m["vdim"], scale=m["scale"],
                           rot_dims=r["dims"], rot_base=r["base"])


def _right(raw, where: str) -> LightningConfig:
    m = _object(raw, _RIGHT, where)
    if len(m["decay"]) != m["heads"] or not all(isinstance(d, (int, float)) and not isinstance(d, bool) for d in m["decay"]):
        raise ConfigError(f"{where}: decay must list one number a head ({m['heads']})")
    return LightningConfig(heads=m["heads"], dim=m["dim"], vdim=m["vdim"], decay=tuple(float(d) for d in m["decay"]))


def _parallel(raw, where: str) -> ParallelConfig:
    m = _object(raw, _PARALLEL, where)
    return ParallelConfig(left=_left(m["left"], where + ".left"), right=_right(m["right"], where + ".right"),
                          left_scale=m["left_scale"], right_scale=m["right_scale"])


def _gla(raw, where: str) -> GlaConfig:
    return GlaConfig(**_object(raw, _GLA, where))


def _mamba(raw, where: str) -> MambaConfig:
    return MambaConfig(**_object(raw, _MAMBA, where))


_MIXERS = {"parallel": _parallel, "gla": _gla, "mamba1": _mamba}


def _mlp(raw, where: str) -> MoeConfig:
    kind = _object(raw, (Key("kind", str),), where)["kind"]
    if kind != "moe":
        raise ConfigError(f"{where}: kind {kind!r} is not implemented (moe)")
    m = _object(raw, _MLP, where)
    e, r = _object(m["expert"], _EXPERT, where + ".expert"), _object(m["router"], _ROUTER, where + ".router")
    if r["top"] > r["experts"]:
        raise ConfigError(f"{where}.router: top={r['top']} exceeds experts={r['experts']}")
    s = _object(m["shared"], _EXPERT, where + ".shared") if m["shared"] is not None else {"ff": 0, "limit": 0.0}
    return MoeConfig(experts=r["experts"], top=r["top"], ff=e["ff"], limit=e["limit"], shared_ff=s["ff"],
                     shared_limit=s["limit"])
