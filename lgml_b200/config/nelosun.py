"""Configuration of the Nelosun decoder, from its own ``config.json`` keys.

``architecture`` names it; ``vocab``, ``width``, ``norm.eps`` and ``embedding.scale`` (the factor on the embedding's rows;
absent: 1) are the model's own numbers; ``layers`` lists the layers one by one: ``type`` (the mixer: ``attention``,
``latent_attention`` or ``rglru``), ``mixer`` (its sizes and constants) and ``mlp`` (the feed-forward, or null for a layer without
one).  ``loop`` (``start``, ``stop``, ``times``; absent: every layer runs once): layers start .. stop - 1 run ``times`` times in a
row with the same weights, and every pass begins with a product over the stream and the embedding's output.

attention ``mixer``: ``heads``, ``kv_heads``, ``dim``, ``vdim``, ``scale``, ``q_temp.coef`` / ``q_temp.every`` (absent: no temperature).

latent_attention ``mixer``: ``heads``, ``dim`` (unrotated per head), ``rot_dim`` (rotated, shared by the heads on the key side),
``vdim``, ``q_rank``, ``kv_rank``, ``scale``, ``rot.base`` / ``rot.dims``.

rglru ``mixer``: ``width`` (the recurrence's channels), ``blocks`` (equal parts with a gate matrix each), ``conv`` (taps).

``mlp``: ``kind`` ``moe`` with ``expert.ff``, ``expert.limit``, ``router.experts``, ``router.top``.
"""
from __future__ import annotations

import copy
from dataclasses import dataclass, field
from typing import Any, Dict, List, Optional, Tuple

from .base import ConfigError, ModelConfig
from .gotulorn import _number, _positive_int

MIXERS = ("attention", "latent_attention", "rglru")


@dataclass
class NelosunConfig(ModelConfig):
    architecture: str = "Nelosun"
    vocab: int = 0
    width: int = 0
    norm_eps: float = 0.0
    embed_scale: float = 1.0
    loop: Optional[Tuple[int, int, int]] = None      # (start, stop, times)
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

    def layer_runs(self) -> List[Tuple[int, Optional[int]]]:
        """The layers in the order in which they run, as (layer, the pass of the loop that begins before it or None)."""
        n = len(self.layers)
        if not self.loop:
            return [(i, None) for i in range(n)]
        a, b, times = self.loop
        runs: List[Tuple[int, Optional[int]]] = [(i, None) for i in range(a)]
        for r in range(times):
            runs += [(i, r if i == a else None) for i in range(a, b)]
        return runs + [(i, None) for i in range(b, n)]

    @classmethod
    def from_dict(cls, d: Dict[str, Any]) -> "NelosunConfig":
        for key in ("vocab", "width", "layers", "norm"):
            if key not in d or d[key] is None:
                raise ConfigError(f"config.json: '{key}' is missing")
        norm = d["norm"]
        if not isinstance(norm, dict) or "eps" not in norm:
            raise ConfigError("config.json: 'norm' must be an object with 'eps'")
        if not isinstance(d["layers"], list):
            raise ConfigError("config.json: 'layers' must be a list")
        emb = d.get("embedding")
        if emb is not None and not isinstance(emb, dict):
            raise ConfigError("config.json: 'embedding' must be an object with 'scale'")
        loop = d.get("loop")
        if loop is not None:
            if not isinstance(loop, dict):
                raise ConfigError("config.json: 'loop' must be an object with 'start', 'stop' and 'times'")
            for key in ("start", "stop", "times"):
                v = loop.get(key)
                if isinstance(v, bool) or not isinstance(v, int) or v < 0:
                    raise ConfigError(f"config.json: loop.{key} must be a non-negative integer, not {v!r}")
            loop = (loop["start"], loop["stop"], loop["times"])
        return cls(vocab=int(d["vocab"]), width=int(d["width"]), norm_eps=float(norm["eps"]),
                   embed_scale=_number("embedding", emb, "scale") if emb and emb.get("scale") is not None else 1.0,
                   loop=loop, layers=copy.deepcopy(d["layers"]), torch_dtype=str(d.get("torch_dtype", "bfloat16")))

    def validate(self) -> None:
        if self.vocab <= 0 or self.width <= 0:
            raise ConfigError("config.json: 'vocab' and 'width' must be positive")
        if not self.norm_eps > 0:
            raise ConfigError("config.json: norm.eps must be positive")
        if not self.layers:
            raise ConfigError("config.json: 'layers' is empty")
        if self.loop is not None:
            a, b, times = self.loop
            if not (0 <= a < b <= len(self.layers)) or times < 1:
                raise ConfigError(f"config.json: loop must name layers start < stop <= {len(self.layers)} and times >= 1, not {self.loop}")
        for i, layer in enumerate(self.layers):
            where = f"layers[{i}]"
            if not isinstance(layer, dict) or layer.get("type") not in MIXERS:
                raise ConfigError(f"config.json: {where}.type must be one of {MIXERS}, not {layer.get('type') if isinstance(layer, dict) else layer!r}")
            m = layer.get("mixer")
            if not isinstance(m, dict):
                raise ConfigError(f"config.json: {where}.mixer must be an object")
            mw = where + ".mixer"
            if layer["type"] == "attention":
                for key in ("heads", "kv_heads", "dim", "vdim"):
                    _positive_int(mw, m, key)
                if m["heads"] % m["kv_heads"]:
                    raise ConfigError(f"config.json: {mw}.heads {m['heads']} is no multiple of kv_heads {m['kv_heads']}")
                _number(mw, m, "scale")
                if m.get("q_temp") is not None:
                    _number(mw + ".q_temp", m["q_temp"], "coef")
                    _positive_int(mw + ".q_temp", m["q_temp"], "every")
            elif layer["type"] == "latent_attention":
                for key in ("heads", "dim", "vdim", "rot_dim", "q_rank", "kv_rank"):
                    _positive_int(mw, m, key)
                _number(mw, m, "scale")
                rot = m.get("rot")
                if not isinstance(rot, dict):
                    raise ConfigError(f"config.json: {mw}.rot must be an object with 'base' and 'dims'")
                _number(mw + ".rot", rot, "base")
                dims = _positive_int(mw + ".rot", rot, "dims")
                if dims % 2 or dims > m["rot_dim"]:
                    raise ConfigError(f"config.json: {mw}.rot.dims {dims} must be even and at most rot_dim {m['rot_dim']}")
            else:
                for key in ("width", "blocks", "conv"):
                    _positive_int(mw, m, key)
                if m["width"] % m["blocks"]:
                    raise ConfigError(f"config.json: {mw}.width {m['width']} is no multiple of its {m['blocks']} blocks")
            mlp = layer.get("mlp")
            if mlp is not None:
                fw = where + ".mlp"
                if not isinstance(mlp, dict) or mlp.get("kind") != "moe":
                    raise ConfigError(f"config.json: {fw}.kind must be 'moe'")
                _positive_int(fw + ".expert", mlp.get("expert"), "ff")
                if not _number(fw + ".expert", mlp["expert"], "limit") > 0:
                    raise ConfigError(f"config.json: {fw}.expert.limit must be positive")
                n = _positive_int(fw + ".router", mlp.get("router"), "experts")
                top = _positive_int(fw + ".router", mlp["router"], "top")
                if top > n:
                    raise ConfigError(f"config.json: {fw}.router.top {top} is more than its {n} experts")

    def to_dict(self) -> Dict[str, Any]:
        d = {"architecture": self.architecture, "vocab": self.vocab, "width": self.width, "norm": {"eps": self.norm_eps},
             "embedding": {"scale": self.embed_scale}, "layers": copy.deepcopy(self.layers)}
        if self.loop is not None:
            d["loop"] = {"start": self.loop[0], "stop": self.loop[1], "times": self.loop[2]}
        return d
