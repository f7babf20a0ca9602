"""Configuration of the Topezen decoder (config.json key ``"architecture": "Topezen"``).

The file is nested: ``vocab``, ``width``, ``norm.eps``, ``embedding.scale`` and a list ``layers`` whose entries give the
layer's ``type`` (which mixer: ``latent_attention``, ``mlstm`` or ``attention``), the mixer's sizes under ``mixer`` and the
feed-forward under ``mlp`` (null: none; ``kind`` ``dense`` with ``ff``, or ``moe`` with ``expert.ff``, ``router.experts``,
``router.top``, optionally ``router.groups`` with ``count`` and ``keep``, and optionally ``shared.ff``).  Every size and
every constant that the file gives is read from it; what the design fixes (both norms read the same stream and have one
number each, the gates on the branches, the forms of the activations, the pairing of rotated entries, the sinks) is in the
parts.
"""

from __future__ import annotations

import dataclasses
from typing import Any, ClassVar

from .base import ConfigError, ModelConfig

MIXERS = ("latent_attention", "mlstm", "attention")
FEED_FORWARDS = ("dense", "moe")


def _need(where: str, table: Any, keys: tuple[str, ...], optional: tuple[str, ...] = ()) -> dict:
    if not isinstance(table, dict):
        raise ConfigError(f"TopezenConfig: {where} must be an object")
    missing = [k for k in keys if k not in table]
    unknown = [k for k in table if k not in keys and k not in optional]
    if missing or unknown:
        parts = ([f"missing keys {sorted(missing)}"] if missing else []) + ([f"unknown keys {sorted(unknown)}"] if unknown else [])
        raise ConfigError(f"TopezenConfig: {where}: " + "; ".join(parts))
    return table


def _positive_int(where: str, value: Any) -> int:
    if isinstance(value, bool) or not isinstance(value, (int, float)) or int(value) != value or value <= 0:
        raise ConfigError(f"TopezenConfig: {where} must be a positive integer, got {value!r}")
    return int(value)


def _positive(where: str, value: Any) -> float:
    if isinstance(value, bool) or not isinstance(value, (int, float)) or not value > 0:
        raise ConfigError(f"TopezenConfig: {where} must be a positive number, got {value!r}")
    return float(value)


@dataclasses.dataclass(frozen=True)
class TopezenConfig(ModelConfig):
    vocab: int
    width: int
    layers: list
    norm: dict
    embedding: dict | None = None  # absent: the table's rows enter the stream as they are
    initializer_range: float | None = None  # only read by the random-weights mode
    max_position_embeddings: int | None = None  # longest sequence a request may reach (optional)

    ARCH_NAMES: ClassVar[tuple[str, ...]] = ("Topezen",)
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
        _positive_int("vocab", self.vocab)
        _positive_int("width", self.width)
        _positive("norm.eps", _need("norm", self.norm, ("eps",))["eps"])
        if self.embedding is not None:
            _positive("embedding.scale", _need("embedding", self.embedding, ("scale",))["scale"])
        if not isinstance(self.layers, list) or not self.layers:
            raise ConfigError("TopezenConfig: layers must be a list with at least one layer")
        for i, layer in enumerate(self.layers):
            where = f"layers[{i}]"
            _need(where, layer, ("type", "mixer"), ("mlp",))
            kind = layer["type"]
            if kind not in MIXERS:
                raise ConfigError(f"TopezenConfig: {where}.type {kind!r} is not a mixer of this design (known: {list(MIXERS)})")
            getattr(self, "_check_" + kind)(where + ".mixer", layer["mixer"])
            if layer.get("mlp") is not None:
                self._check_mlp(where + ".mlp", layer["mlp"])
        if self.max_position_embeddings is not None:
            _positive_int("max_position_embeddings", self.max_position_embeddings)

    @staticmethod
    def _check_latent_attention(where: str, mixer: Any) -> None:
        m = _need(where, mixer, ("heads", "dim", "rot_dim", "vdim", "q_rank", "kv_rank", "scale", "rot"))
        for key in ("heads", "dim", "rot_dim", "vdim", "q_rank", "kv_rank"):
            _positive_int(f"{where}.{key}", m[key])
        _positive(f"{where}.scale", m["scale"])
        rot = _need(where + ".rot", m["rot"], ("base", "dims"))
        _positive(f"{where}.rot.base", rot["base"])
        dims = _positive_int(f"{where}.rot.dims", rot["dims"])
        if dims != m["rot_dim"] or dims % 2:
            raise ConfigError(f"TopezenConfig: {where}.rot.dims ({dims}) must be even and equal rot_dim ({m['rot_dim']})")

    @staticmethod
    def _check_mlstm(where: str, mixer: Any) -> None:
        m = _need(where, mixer, ("heads", "dim", "vdim", "gate_cap"))
        for key in ("heads", "dim", "vdim"):
            _positive_int(f"{where}.{key}", m[key])
        _positive(f"{where}.gate_cap", m["gate_cap"])

    @staticmethod
    def _check_attention(where: str, mixer: Any) -> None:
        m = _need(where, mixer, ("heads", "kv_heads", "dim", "vdim", "scale"), ("softcap", "mask"))
        for key in ("heads", "kv_heads", "dim", "vdim"):
            _positive_int(f"{where}.{key}", m[key])
        _positive(f"{where}.scale", m["scale"])
        if m["heads"] % m["kv_heads"]:
            raise ConfigError(f"TopezenConfig: {where}.heads ({m['heads']}) must be a multiple of kv_heads ({m['kv_heads']})")
        if m.get("softcap") is not None:  # absent: the scores are not capped
            _positive(f"{where}.softcap", m["softcap"])
        if m.get("mask") is not None:  # absent: every earlier key is seen
            mask = _need(where + ".mask", m["mask"], ("size",), ("keep_first",))
            _positive_int(f"{where}.mask.size", mask["size"])
            kept = mask.get("keep_first")
            if kept is not None and (isinstance(kept, bool) or not isinstance(kept, int) or kept < 0):
                raise ConfigError(f"TopezenConfig: {where}.mask.keep_first must be a whole number that is not negative, got {kept!r}")

    @staticmethod
    def _check_mlp(where: str, mlp: Any) -> None:
        if not isinstance(mlp, dict) or mlp.get("kind") not in FEED_FORWARDS:
            raise ConfigError(f"TopezenConfig: {where}.kind must be one of {list(FEED_FORWARDS)}")
        if mlp["kind"] == "dense":
            _positive_int(f"{where}.ff", _need(where, mlp, ("kind", "ff"))["ff"])
            return
        _need(where, mlp, ("kind", "expert", "router"), ("shared",))
        _positive_int(f"{where}.expert.ff", _need(where + ".expert", mlp["expert"], ("ff",))["ff"])
        if mlp.get("shared") is not None:
            _positive_int(f"{where}.shared.ff", _need(where + ".shared", mlp["shared"], ("ff",))["ff"])
        r = _need(where + ".router", mlp["router"], ("experts", "top"), ("groups",))
        experts, top = _positive_int(f"{where}.router.experts", r["experts"]), _positive_int(f"{where}.router.top", r["top"])
        allowed = experts
        if r.get("groups") is not None:
            g = _need(where + ".router.groups", r["groups"], ("count", "keep"))
            count, keep = _positive_int(f"{where}.router.groups.count", g["count"]), _positive_int(f"{where}.router.groups.keep", g["keep"])
            if experts % count or keep > count:
                raise ConfigError(f"TopezenConfig: {where}.router: {experts} experts do not form {count} equal groups of which {keep} are kept")
            allowed = keep * (experts // count)
        if top > allowed:
            raise ConfigError(f"TopezenConfig: {where}.router: {top} experts cannot be chosen from {allowed}")
