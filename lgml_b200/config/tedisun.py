"""Configuration of the Tedisun decoder, from its own ``config.json`` keys.

``architecture`` names it; ``vocab``, ``width``, ``norm.eps``, ``streams`` (how many residual streams), ``embedding.scale`` (the
factor on the embedding's rows; absent: 1) and ``logit_softcap`` (absent: none) are the model's own numbers.  ``layers`` lists
the layers one by one: ``type`` (the mixer: ``delta`` or ``parallel``), ``mixer`` (its sizes and constants) and ``mlp`` (the
feed-forward, or null for a layer without one).

delta ``mixer``: ``heads``, ``kv_heads``, ``dim``, ``vdim``, ``conv`` (taps of the short convolutions).

parallel ``mixer``: ``left``, ``right``, ``left_scale``, ``right_scale``.  ``left``: ``heads``, ``kv_heads``, ``dim``, ``vdim``,
``scale``, ``rot.base`` / ``rot.dims`` / ``rot.scaling`` (``factor``, ``low``, ``high``, ``original``; absent: the plain
frequencies), ``mask.size`` / ``mask.keep_first`` (the window and the first tokens that stay visible; absent: all keys).
``right``: ``heads``, ``dim``, ``vdim``, ``gate_cap``.

``mlp``: ``kind`` ``moe`` with ``expert.ff`` and ``router.experts``, ``router.identity`` (absent: 0), ``router.top``.
"""
from __future__ import annotations

import copy
from dataclasses import dataclass, field
from typing import Any, Dict, List, Optional

from .base import ConfigError, ModelConfig
from .gotulorn import _number, _positive_int

MIXERS = ("delta", "parallel")
MLP_KINDS = ("moe",)
MAX_STREAMS = 8
MAX_TAPS = 8


def _object(where: str, d: Dict[str, Any], key: str) -> Dict[str, Any]:
    v = d.get(key)
    if not isinstance(v, dict):
        raise ConfigError(f"config.json: {where}.{key} must be an object")
    return v


def _count(where: str, d: Dict[str, Any], key: str, default: int) -> int:
    v = d.get(key, default)
    if isinstance(v, bool) or not isinstance(v, int) or v < 0:
        raise ConfigError(f"config.json: {where}.{key} must be a non-negative integer, not {v!r}")
    return v


@dataclass
class TedisunConfig(ModelConfig):
    architecture: str = "Tedisun"
    vocab: int = 0
    width: int = 0
    norm_eps: float = 0.0
    streams: int = 1
    embed_scale: float = 1.0
    logit_softcap: Optional[float] = None
    layers: List[Dict[str, Any]] = field(default_factory=list)
    torch_dtype: str = "bfloat16"

    # the names other parts of the engine ask a configuration for
    @property
    def vocab_size(self) -> int:
        return self.vocab

    @property
    def hidden_size(self) -> int:
        return self.width

    @property
    def num_hidden_layers(self) -> int:
        return len(self.layers)

    @classmethod
    def from_dict(cls, d: Dict[str, Any]) -> "TedisunConfig":
        for key in ("vocab", "width", "layers", "norm", "streams"):
            if key not in d or d[key] is None:
                raise ConfigError(f"config.json: '{key}' is missing")
        norm = d["norm"]
        if not isinstance(norm, dict) or "eps" not in norm:
            raise ConfigError("config.json: 'norm' must be an object with 'eps'")
        if not isinstance(d["layers"], list):
            raise ConfigError("config.json: 'layers' must be a list")
        emb, cap = d.get("embedding"), d.get("logit_softcap")
        if emb is not None and not isinstance(emb, dict):
            raise ConfigError("config.json: 'embedding' must be an object")
        if cap is not None and (isinstance(cap, bool) or not isinstance(cap, (int, float))):
            raise ConfigError(f"config.json: logit_softcap must be a number, not {cap!r}")
        sizes = {key: _positive_int("config", d, key) for key in ("vocab", "width", "streams")}
        return cls(norm_eps=float(norm["eps"]), embed_scale=float(_number("embedding", emb, "scale")) if emb and "scale" in emb else 1.0,
                   logit_softcap=float(cap) if cap else None, layers=copy.deepcopy(d["layers"]), torch_dtype=str(d.get("torch_dtype", "bfloat16")), **sizes)

    def validate(self) -> None:
        if not self.norm_eps > 0:
            raise ConfigError("config.json: norm.eps must be positive")
        if self.streams > MAX_STREAMS:
            raise ConfigError(f"config.json: streams must be at most {MAX_STREAMS}, not {self.streams}")
        if self.logit_softcap is not None and not self.logit_softcap > 0:
            raise ConfigError("config.json: logit_softcap must be positive")
        if not self.layers:
            raise ConfigError("config.json: 'layers' is empty")
        for i, layer in enumerate(self.layers):
            where = f"layers[{i}]"
            if not isinstance(layer, dict) or layer.get("type") not in MIXERS:
                raise ConfigError(f"config.json: {where}.type must be one of {MIXERS}, not {layer.get('type') if isinstance(layer, dict) else layer!r}")
            m = _object(where, layer, "mixer")
            if layer["type"] == "delta":
                self._check_heads(where + ".mixer", m)
                if _positive_int(where + ".mixer", m, "conv") > MAX_TAPS:
                    raise ConfigError(f"config.json: {where}.mixer.conv must be at most {MAX_TAPS}")
            else:
                self._check_parallel(where + ".mixer", m)
            mlp = layer.get("mlp")
            if mlp is not None:
                self._check_mlp(where + ".mlp", mlp)

    @staticmethod
    def _check_heads(where: str, m: Dict[str, Any]) -> None:
        for key in ("heads", "kv_heads", "dim", "vdim"):
            _positive_int(where, m, key)
        if m["heads"] % m["kv_heads"]:
            raise ConfigError(f"config.json: {where}.heads {m['heads']} is no multiple of kv_heads {m['kv_heads']}")

    @classmethod
    def _check_parallel(cls, where: str, m: Dict[str, Any]) -> None:
        for key in ("left_scale", "right_scale"):
            _number(where, m, key)
        lw, left = where + ".left", _object(where, m, "left")
        cls._check_heads(lw, left)
        _number(lw, left, "scale")
        rot = _object(lw, left, "rot")
        if not _number(lw + ".rot", rot, "base") > 0:
            raise ConfigError(f"config.json: {lw}.rot.base must be positive")
        dims = _positive_int(lw + ".rot", rot, "dims")
        if dims % 2 or dims > left["dim"]:
            raise ConfigError(f"config.json: {lw}.rot.dims {dims} must be even and at most dim {left['dim']}")
        if rot.get("scaling") is not None:
            sc = _object(lw + ".rot", rot, "scaling")
            for key in ("factor", "low", "high", "original"):
                if not _number(lw + ".rot.scaling", sc, key) > 0:
                    raise ConfigError(f"config.json: {lw}.rot.scaling.{key} must be positive")
            if sc["high"] <= sc["low"]:
                raise ConfigError(f"config.json: {lw}.rot.scaling.high must be above low")
        if left.get("mask") is not None:
            mask = _object(lw, left, "mask")
            _positive_int(lw + ".mask", mask, "size")
            _count(lw + ".mask", mask, "keep_first", 0)
        rw, right = where + ".right", _object(where, m, "right")
        for key in ("heads", "dim", "vdim"):
            _positive_int(rw, right, key)
        if right["dim"] > 1024:
            raise ConfigError(f"config.json: {rw}.dim must be at most 1024")
        if not _number(rw, right, "gate_cap") > 0:
            raise ConfigError(f"config.json: {rw}.gate_cap must be positive")

    @staticmethod
    def _check_mlp(where: str, mlp: Any) -> None:
        if not isinstance(mlp, dict) or mlp.get("kind") not in MLP_KINDS:
            raise ConfigError(f"config.json: {where}.kind must be one of {MLP_KINDS}")
        _positive_int(where + ".expert", _object(where, mlp, "expert"), "ff")
        router = _object(where, mlp, "router")
        experts, top = _positive_int(where + ".router", router, "experts"), _positive_int(where + ".router", router, "top")
        identity = _count(where + ".router", router, "identity", 0)
        if top > experts + identity:
            raise ConfigError(f"config.json: {where}.router.top {top} is more than the {experts} + {identity} experts")

    def to_dict(self) -> Dict[str, Any]:
        d = {"architecture": self.architecture, "vocab": self.vocab, "width": self.width, "norm": {"eps": self.norm_eps}, "streams": self.streams,
             "embedding": {"scale": self.embed_scale}, "layers": copy.deepcopy(self.layers)}
        if self.logit_softcap is not None:
            d["logit_softcap"] = self.logit_softcap
        return d
