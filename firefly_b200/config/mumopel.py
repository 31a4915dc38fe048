"""Typed configuration of the Mumopel design.

``config.json`` names the design under ``architecture`` and gives every size and constant:

    vocab, width, streams, logit_softcap (absent or null: none), norm.eps
    layers[i]: type ("attention"), mixer {...}, mlp {...} | null
        attention:       heads, kv_heads, dim, vdim, scale, mask {size} | absent (every earlier position is seen),
                         rot {base, dims} | absent
        mlp kind "dense": ff
        mlp kind "moe":   router {experts, top}, expert {ff, limit}, shared {ff, limit} | absent
    loop {start, stop, times} | absent: layers start .. stop-1 run ``times`` times in a row with the same weights

The nested objects are kept as they are and checked here, so that a wrong or missing key is told by name before
anything is built.
"""
from __future__ import annotations

from dataclasses import dataclass
from typing import Any, ClassVar, Dict, Mapping, Optional, Tuple

from .base import ConfigError, ModelConfig
from .kolorax import _need as _need_loop
from .pepolorn import _need

MIXERS = ("attention",)


def _check_mixer(mx, where: str) -> None:
    for key in ("heads", "kv_heads", "dim", "vdim"):
        _need(mx, key, int, where)
    _need(mx, "scale", float, where)
    if int(mx["heads"]) % int(mx["kv_heads"]):
        raise ConfigError(f"config.json: {where}.heads must be a multiple of kv_heads")
    if mx.get("mask") is not None:
        _need(mx["mask"], "size", int, where + ".mask")
    rot = mx.get("rot")
    if rot is not None:
        if not (_need(rot, "base", float, where + ".rot") > 0):
            raise ConfigError(f"config.json: {where}.rot.base must be positive")
        dims = rot.get("dims")
        if isinstance(dims, bool) or not isinstance(dims, int) or dims < 0 or dims % 2 or dims > int(mx["dim"]):
            raise ConfigError(f"config.json: {where}.rot.dims must be even and at most dim, got {dims!r}")


def _check_mlp(ml, where: str) -> None:
    kind = _need(ml, "kind", str, where)
    if kind == "dense":
        _need(ml, "ff", int, where)
    elif kind == "moe":
        r = _need(ml, "router", None, where)
        if _need(r, "top", int, where + ".router") > _need(r, "experts", int, where + ".router"):
            raise ConfigError(f"config.json: {where}.router.top is larger than the number of experts")
        for key in ("expert", "shared"):
            part = ml.get(key)
            if part is None and key == "shared":
                continue
            _need(_need(ml, key, None, where), "ff", int, f"{where}.{key}")
            if not (_need(part, "limit", float, f"{where}.{key}") > 0):
                raise ConfigError(f"config.json: {where}.{key}.limit must be positive")
    else:
        raise ConfigError(f"config.json: {where}.kind '{kind}' is not one of ('dense', 'moe')")


@dataclass(frozen=True)
class MumopelConfig(ModelConfig):
    architecture: ClassVar[str] = "Mumopel"

    vocab: int
    width: int
    streams: int
    norm_eps: float
    logit_softcap: Optional[float]
    layers: Tuple[Mapping[str, Any], ...]
    loop: Optional[Mapping[str, int]] = None

    @property
    def vocab_size(self) -> int:
        return self.vocab

    @classmethod
    def from_dict(cls, raw: Mapping[str, Any]) -> "MumopelConfig":
        layers = raw.get("layers")
        if not isinstance(layers, list) or not layers:
            raise ConfigError("config.json: 'layers' must be a non-empty list")
        loop = raw.get("loop")
        cfg = cls(
            vocab=cls._get(raw, "vocab", int), width=cls._get(raw, "width", int), streams=cls._get(raw, "streams", int),
            norm_eps=_need(raw.get("norm") or {}, "eps", float, "norm"), logit_softcap=cls._get(raw, "logit_softcap", float, None),
            layers=tuple(layers), loop=None if not loop else {k: _need_loop(loop, k, int, "loop") for k in ("start", "stop", "times")})
        cfg.validate()
        return cfg

    def to_dict(self) -> Dict[str, Any]:
        out = {"architecture": self.architecture, "vocab": self.vocab, "width": self.width, "streams": self.streams,
               "norm": {"eps": self.norm_eps}, "layers": [dict(L) for L in self.layers]}
        if self.logit_softcap is not None:
            out["logit_softcap"] = self.logit_softcap
        if self.loop:
            out["loop"] = dict(self.loop)
        return out

    def validate(self) -> None:
        if self.vocab <= 0 or self.width <= 0:
            raise ConfigError("config.json: 'vocab' and 'width' must be positive")
        if not (1 <= self.streams <= 32):
            raise ConfigError(f"config.json: 'streams' must be 1 to 32, got {self.streams}")
        if not (self.norm_eps > 0):
            raise ConfigError(f"config.json: norm.eps must be > 0, got {self.norm_eps}")
        if self.logit_softcap is not None and not (self.logit_softcap > 0):
            raise ConfigError(f"config.json: logit_softcap must be > 0, got {self.logit_softcap}")
        for i, L in enumerate(self.layers):
            where = f"layers[{i}]"
            kind = _need(L, "type", str, where)
            if kind not in MIXERS:
                raise ConfigError(f"config.json: {where}.type '{kind}' is not one of {MIXERS}")
            _check_mixer(_need(L, "mixer", None, where), where + ".mixer")
            if L.get("mlp") is not None:
                _check_mlp(L["mlp"], where + ".mlp")
        if self.loop:
            a, b, n = self.loop["start"], self.loop["stop"], self.loop["times"]
            if not (0 <= a < b <= len(self.layers)) or n < 1:
                raise ConfigError(f"config.json: loop {dict(self.loop)} does not fit {len(self.layers)} layers")
