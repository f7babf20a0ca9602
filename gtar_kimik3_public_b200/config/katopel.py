"""Configuration of the Katopel decoder (config.json key ``"architecture": "Katopel"``).

The file is nested: ``vocab``, ``width``, ``norm.eps``, ``embedding.scale``, ``loop`` (``start``, ``stop``, ``times``: which layers
run several times in a row; absent: none), and a list ``layers`` whose entries give the layer's ``type`` (which mixer: ``delta``
or ``parallel``), the mixer's sizes under ``mixer`` (a ``parallel`` one has two of them, ``left`` and ``right``, with ``left_scale``
and ``right_scale``) and the feed-forward under ``mlp`` (null: none; ``kind`` ``dense`` with ``ff``, or ``moe`` with ``expert.ff``,
``router.experts``, ``router.top`` and optionally ``shared.ff``).  Every size and every constant that the file gives is read from
it; what the design fixes (the norms' form and places, SiLU, the pairing of rotated entries, the router's rule) is in the parts
and in the builder.
"""

from __future__ import annotations

import dataclasses
from typing import Any, ClassVar

from .base import ConfigError, ModelConfig

MIXERS = ("delta", "parallel")
FEED_FORWARDS = ("dense", "moe")
MAX_HEAD = 512  # entries of a head that the kernels' warps hold
MAX_TAPS = 16
_NAME = "KatopelConfig"


def _need(where: str, table: Any, keys: tuple[str, ...], optional: tuple[str, ...] = ()) -> dict:
    if not isinstance(table, dict):
        raise ConfigError(f"{_NAME}: {where} must be an object")
    missing = [k for k in keys if k not in table]
    unknown = [k for k in table if k not in keys and k not in optional]
    if missing or unknown:
        parts = ([f"missing keys {sorted(missing)}"] if missing else []) + ([f"unknown keys {sorted(unknown)}"] if unknown else [])
        raise ConfigError(f"{_NAME}: {where}: " + "; ".join(parts))
    return table


def _int(where: str, value: Any, least: int = 1, most: int | None = None) -> int:
    if isinstance(value, bool) or not isinstance(value, (int, float)) or int(value) != value or value < least:
        raise ConfigError(f"{_NAME}: {where} must be an integer of at least {least}, got {value!r}")
    if most is not None and value > most:
        raise ConfigError(f"{_NAME}: {where} must be at most {most}, got {value!r}")
    return int(value)


def _number(where: str, value: Any, positive: bool = True) -> float:
    if isinstance(value, bool) or not isinstance(value, (int, float)) or (positive and not value > 0):
        raise ConfigError(f"{_NAME}: {where} must be a {'positive ' if positive else ''}number, got {value!r}")
    return float(value)


def _check_heads(where: str, m: dict) -> None:
    _int(where + ".heads", m["heads"])
    _int(where + ".kv_heads", m["kv_heads"])
    _int(where + ".dim", m["dim"], most=MAX_HEAD)
    _int(where + ".vdim", m["vdim"], most=MAX_HEAD)
    if m["heads"] % m["kv_heads"]:
        raise ConfigError(f"{_NAME}: {where}.heads ({m['heads']}) must be a multiple of kv_heads ({m['kv_heads']})")


def _check_delta(where: str, mixer: Any) -> None:
    _check_heads(where, _need(where, mixer, ("heads", "kv_heads", "dim", "vdim", "conv")))
    _int(where + ".conv", mixer["conv"], most=MAX_TAPS)


def _check_attention(where: str, mixer: Any) -> None:
    m = _need(where, mixer, ("heads", "kv_heads", "dim", "vdim", "scale"), ("rot", "mask"))
    _check_heads(where, m)
    _number(where + ".scale", m["scale"])
    if m.get("rot") is not None:
        rot = _need(where + ".rot", m["rot"], ("base", "dims"))
        _number(where + ".rot.base", rot["base"])
        dims = _int(where + ".rot.dims", rot["dims"], least=0)
        if dims % 2 or dims > m["dim"]:
            raise ConfigError(f"{_NAME}: {where}.rot.dims ({dims}) must be even and at most dim ({m['dim']})")
    if m.get("mask") is not None:  # absent: every earlier key is seen
        _int(where + ".mask.size", _need(where + ".mask", m["mask"], ("size",))["size"])


@dataclasses.dataclass(frozen=True)
class KatopelConfig(ModelConfig):
    vocab: int
    width: int
    layers: list
    norm: dict
    loop: dict | None = None  # absent: every layer runs once
    embedding: dict | None = None  # absent: the table's rows enter the stream as they are
    initializer_range: float | None = None  # only read by the random-weights mode
    max_position_embeddings: int | None = None  # longest sequence a request may reach (optional)

    ARCH_NAMES: ClassVar[tuple[str, ...]] = ("Katopel",)
    IGNORED_KEYS: ClassVar[frozenset[str]] = frozenset({"architecture", "torch_dtype", "dtype"})

    @property
    def eps(self) -> float:
        return float(self.norm["eps"])

    @property
    def embedding_scale(self) -> float:
        return float(self.embedding["scale"]) if self.embedding else 1.0

    def to_dict(self) -> dict[str, Any]:
        out = {k: v for k, v in dataclasses.asdict(self).items() if v is not None}
        out["architecture"] = self.ARCH_NAMES[0]
        return out

    def validate(self) -> None:
        _int("vocab", self.vocab)
        _int("width", self.width)
        _number("norm.eps", _need("norm", self.norm, ("eps",))["eps"])
        if self.embedding is not None:
            _number("embedding.scale", _need("embedding", self.embedding, ("scale",))["scale"], positive=False)
        if not isinstance(self.layers, list) or not self.layers:
            raise ConfigError(f"{_NAME}: layers must be a list with at least one layer")
        if self.loop is not None:
            loop = _need("loop", self.loop, ("start", "stop", "times"))
            start, stop = _int("loop.start", loop["start"], least=0), _int("loop.stop", loop["stop"])
            _int("loop.times", loop["times"])
            if not start < stop <= len(self.layers):
                raise ConfigError(f"{_NAME}: loop: layers {start} .. {stop - 1} are not layers of this model ({len(self.layers)} layers)")
        for i, layer in enumerate(self.layers):
            where = f"layers[{i}]"
            _need(where, layer, ("type", "mixer"), ("mlp",))
            kind, m = layer["type"], layer["mixer"]
            if kind not in MIXERS:
                raise ConfigError(f"{_NAME}: {where}.type {kind!r} is not a mixer of this design (known: {list(MIXERS)})")
            if kind == "delta":
                _check_delta(where + ".mixer", m)
            else:
                _need(where + ".mixer", m, ("left", "right"), ("left_scale", "right_scale"))
                _check_attention(where + ".mixer.left", m["left"])
                _check_delta(where + ".mixer.right", m["right"])
                for key in ("left_scale", "right_scale"):
                    if m.get(key) is not None:
                        _number(f"{where}.mixer.{key}", m[key], positive=False)
            if layer.get("mlp") is not None:
                self._check_mlp(where + ".mlp", layer["mlp"])
        if self.max_position_embeddings is not None:
            _int("max_position_embeddings", self.max_position_embeddings)

    @staticmethod
    def _check_mlp(where: str, mlp: Any) -> None:
        if not isinstance(mlp, dict) or mlp.get("kind") not in FEED_FORWARDS:
            raise ConfigError(f"{_NAME}: {where}.kind must be one of {list(FEED_FORWARDS)}")
        if mlp["kind"] == "dense":
            _int(where + ".ff", _need(where, mlp, ("kind", "ff"))["ff"])
            return
        _need(where, mlp, ("kind", "expert", "router"), ("shared",))
        _int(where + ".expert.ff", _need(where + ".expert", mlp["expert"], ("ff",))["ff"])
        if mlp.get("shared") is not None:
            _int(where + ".shared.ff", _need(where + ".shared", mlp["shared"], ("ff",))["ff"])
        r = _need(where + ".router", mlp["router"], ("experts", "top"))
        experts, top = _int(where + ".router.experts", r["experts"]), _int(where + ".router.top", r["top"])
        if top > experts:
            raise ConfigError(f"{_NAME}: {where}.router: {top} experts cannot be chosen from {experts}")
