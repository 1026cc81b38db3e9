"""Typed configuration of the Balelorn design, read from its own ``config.json``.

The file is nested like Bobepel's: ``layers`` lists the layers in order, each with its ``type`` (``attention``), the
mixer's sizes and constants under ``mixer`` and its feed-forward under ``mlp`` (``kind``: ``dense`` or ``moe``; null:
none).  Every size and every constant that differs between models of the design is read from the file; nothing is
assumed about how many layers there are, in which order, which of them mix their values or carry experts.  A key that
is not listed is ignored; a layer type, a feed-forward kind or a value that the engine does not implement is refused
by name.
"""
from __future__ import annotations

from dataclasses import dataclass
from typing import Optional, Tuple

from .schema import ConfigError, Key, positive, read_keys

ARCHITECTURE = "Balelorn"
DEFAULT_MAX_POSITIONS = 1 << 17   # the design has no position limit; the engine's block tables need one

_TOP = (
    Key("vocab", int, check=positive),
    Key("width", int, check=positive),
    Key("layers", list),
    Key("norm", object),
    Key("max_positions", int, default=DEFAULT_MAX_POSITIONS, check=positive),
)
_ATTENTION = (
    Key("heads", int, check=positive), Key("kv_heads", int, default=lambda v: v["heads"], check=positive),
    Key("dim", int, check=positive), Key("vdim", int, default=lambda v: v["dim"], check=positive),
    Key("scale", float), Key("rot", object, default=None, nullable=True),
    Key("mask", object, default=None, nullable=True), Key("v_mix", bool, default=False),
)
_ROT = (Key("dims", int), Key("base", float, check=positive))
_MASK = (Key("size", int, check=positive),)


@dataclass(frozen=True)
class RotaryConfig:
    dims: int                 # the leading elements of a head that are rotated
    base: float


@dataclass(frozen=True)
class AttentionConfig:
    heads: int
    kv_heads: int
    dim: int
    vdim: int
    scale: float
    rot: Optional[RotaryConfig]
    chunk: Optional[int]      # positions of a chunk; None: every earlier position is visible
    v_mix: bool


@dataclass(frozen=True)
class DenseConfig:
    ff: int


@dataclass(frozen=True)
class MoeConfig:
    experts: int
    top: int
    ff: int
    limit: float


@dataclass(frozen=True)
class LayerConfig:
    type: str                 # attention
    mixer: AttentionConfig
    mlp: object               # DenseConfig | MoeConfig | None (the layer has no feed-forward)


@dataclass(frozen=True)
class BalelornConfig:
    vocab: int
    width: int
    norm_eps: float
    max_positions: int
    layers: Tuple[LayerConfig, ...]

    @classmethod
    def from_json(cls, obj: dict) -> "BalelornConfig":
        v = read_keys(obj, _TOP)
        eps = _object(v["norm"], (Key("eps", float, check=positive),), "config.json: norm")["eps"]
        layers = []
        for i, raw in enumerate(v["layers"]):
            where = f"config.json: layers[{i}]"
            lv = _object(raw, (Key("type", str), Key("mixer", object),
                               Key("mlp", object, default=None, nullable=True)), where)
            if lv["type"] != "attention":
                raise ConfigError(f"{where}: layer type {lv['type']!r} is not implemented (attention)")
            mixer = _attention(lv["mixer"], where + ".mixer")
            mlp = _mlp(lv["mlp"], where + ".mlp") if lv["mlp"] is not None else None
            layers.append(LayerConfig(lv["type"], mixer, mlp))
        if not layers:
            raise ConfigError("config.json: layers is empty")
        mixing = [(i, layer.mixer) for i, layer in enumerate(layers) if layer.mixer.v_mix]
        for i, m in mixing[1:]:
            first = mixing[0][1]
            if m.kv_heads * m.vdim != first.kv_heads * first.vdim:
                raise ConfigError(f"config.json: layers[{i}].mixer: its {m.kv_heads} x {m.vdim} values cannot be mixed "
                                  f"with the {first.kv_heads} x {first.vdim} of layer {mixing[0][0]}")
        return cls(vocab=v["vocab"], width=v["width"], norm_eps=eps, max_positions=v["max_positions"],
                   layers=tuple(layers))


def _object(raw, schema, where: str) -> dict:
    if not isinstance(raw, dict):
        raise ConfigError(f"{where}: must be an object")
    return read_keys(raw, schema, where=where)


def _attention(raw, where: str) -> AttentionConfig:
    m = _object(raw, _ATTENTION, where)
    if m["heads"] % m["kv_heads"]:
        raise ConfigError(f"{where}: heads must be a multiple of kv_heads")
    rot = None
    if m["rot"] is not None:
        r = _object(m["rot"], _ROT, where + ".rot")
        if r["dims"] % 2 or not 0 <= r["dims"] <= m["dim"]:
            raise ConfigError(f"{where}: rot.dims must be even and at most dim")
        rot = RotaryConfig(r["dims"], r["base"]) if r["dims"] else None
    chunk = _object(m["mask"], _MASK, where + ".mask")["size"] if m["mask"] is not None else None
    return AttentionConfig(heads=m["heads"], kv_heads=m["kv_heads"], dim=m["dim"], vdim=m["vdim"], scale=m["scale"],
                           rot=rot, chunk=chunk, v_mix=m["v_mix"])


def _mlp(raw, where: str):
    kind = _object(raw, (Key("kind", str),), where)["kind"]
    if kind == "dense":
        return DenseConfig(_object(raw, (Key("ff", int, check=positive),), where)["ff"])
    if kind != "moe":
        raise ConfigError(f"{where}: kind {kind!r} is not implemented (dense, moe)")
    m = _object(raw, (Key("expert", object), Key("router", object)), where)
    e = _object(m["expert"], (Key("ff", int, check=positive), Key("limit", float, check=positive)), where + ".expert")
    r = _object(m["router"], (Key("experts", int, check=positive), Key("top", int, check=positive)), where + ".router")
    if r["top"] > r["experts"]:
        raise ConfigError(f"{where}.router: top={r['top']} exceeds experts={r['experts']}")
    return MoeConfig(experts=r["experts"], top=r["top"], ff=e["ff"], limit=e["limit"])
