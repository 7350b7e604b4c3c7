"""Typed configuration of the Lidizen design, read from its own config.json keys.

A Lidizen model is a list of layers over several parallel residual streams that hyper-connections
mix at every sublayer. A layer's mixer is "attention" (grouped-query attention with scores mixed
across heads, a window that keeps the sequence's first positions, and values mixed with an earlier
layer's); its feed-forward is dense, a mixture of experts, or absent. The embedding adds a hashed
table of token pairs. Every size and every constant that may differ between models is a key; what
the design fixes is written in `models/lidizen.py`.
"""

from __future__ import annotations

import copy
from dataclasses import dataclass
from typing import Any

from atomserve_b200.config.gefilix_config import _need
from atomserve_b200.config.model_config import ModelConfigError

MIXERS = ("attention",)
FEED_FORWARDS = ("dense", "moe")


@dataclass(frozen=True)
class LidizenConfig:
    vocab: int
    width: int
    streams: int
    layers: tuple[dict[str, Any], ...]
    norm_eps: float
    bigram: dict[str, int]
    max_positions: int = 1 << 20  # no learned or tabulated positions: no limit of the design's own

    architecture = "Lidizen"

    @classmethod
    def from_dict(cls, raw: dict) -> "LidizenConfig":
        name = raw.get("architecture") or (raw.get("architectures") or [None])[0]
        if name != cls.architecture:
            raise ModelConfigError(f"expected architecture {cls.architecture!r}, got {name!r}")
        _need(raw, ("vocab", "width", "streams", "layers", "norm", "embedding"), "config.json")
        _need(raw["norm"], ("eps",), "config.json norm")
        _need(raw["embedding"], ("bigram",), "config.json embedding")
        _need(raw["embedding"]["bigram"], ("buckets", "mul_prev", "mul_cur"), "config.json embedding bigram")
        config = cls(
            vocab=int(raw["vocab"]),
            width=int(raw["width"]),
            streams=int(raw["streams"]),
            layers=tuple(copy.deepcopy(layer) for layer in raw["layers"]),
            norm_eps=float(raw["norm"]["eps"]),
            bigram={k: int(raw["embedding"]["bigram"][k]) for k in ("buckets", "mul_prev", "mul_cur")},
            max_positions=int(raw.get("max_positions", 1 << 20)),
        )
        config.validate()
        return config

    def first_value_layer(self) -> int | None:
        """The first layer that mixes values: later ones mix theirs with its."""
        return next((i for i, layer in enumerate(self.layers) if layer["mixer"].get("v_mix")), None)

    def validate(self) -> None:
        if self.vocab < 1 or self.width < 1 or not self.layers:
            raise ModelConfigError("vocab, width and the number of layers must be positive")
        if not 1 <= self.streams <= 16:
            raise ModelConfigError(f"streams {self.streams} must be between 1 and 16")
        if not self.norm_eps >= 0:
            raise ModelConfigError("norm.eps must be >= 0")
        if self.bigram["buckets"] < 1 or self.bigram["mul_prev"] < 0 or self.bigram["mul_cur"] < 0:
            raise ModelConfigError("embedding.bigram needs buckets >= 1 and multipliers >= 0")
        for i, layer in enumerate(self.layers):
            where = f"layer {i}"
            _need(layer, ("type", "mixer"), where)
            m = layer["mixer"]
            if layer["type"] not in MIXERS:
                raise ModelConfigError(f"{where}: mixer type {layer['type']!r} is not one of {MIXERS}")
            _need(m, ("heads", "kv_heads", "dim", "vdim", "scale"), where + " mixer")
            if m["heads"] < 1 or m["kv_heads"] < 1 or m["heads"] % m["kv_heads"]:
                raise ModelConfigError(f"{where}: {m['heads']} heads are not a multiple of {m['kv_heads']} kv heads")
            rot = m.get("rot")
            if rot is not None:
                _need(rot, ("base", "dims"), where + " mixer rot")
                if rot["dims"] % 2 or not 0 <= rot["dims"] <= m["dim"]:
                    raise ModelConfigError(f"{where}: rot.dims {rot['dims']} must be even and at most dim {m['dim']}")
            mask = m.get("mask")
            if mask is not None:
                _need(mask, ("size",), where + " mixer mask")
                if mask["size"] < 1 or mask.get("keep_first", 0) < 0:
                    raise ModelConfigError(f"{where}: mask.size must be positive and mask.keep_first not negative")
            first = self.first_value_layer()
            if m.get("v_mix") and (m["kv_heads"], m["vdim"]) != tuple(self.layers[first]["mixer"][k] for k in ("kv_heads", "vdim")):
                raise ModelConfigError(f"{where}: its values do not have the shape of layer {first}'s, with which they are mixed")
            mlp = layer.get("mlp")
            if mlp is None:
                continue
            _need(mlp, ("kind",), where + " mlp")
            if mlp["kind"] not in FEED_FORWARDS:
                raise ModelConfigError(f"{where}: mlp kind {mlp['kind']!r} is not one of {FEED_FORWARDS}")
            if mlp["kind"] == "dense":
                _need(mlp, ("ff",), where + " mlp")
                continue
            _need(mlp, ("expert", "router"), where + " mlp")
            _need(mlp["expert"], ("ff",), where + " mlp expert")
            _need(mlp["router"], ("experts", "top"), where + " mlp router")
            r = mlp["router"]
            if not 1 <= r["top"] <= min(r["experts"], 32):
                raise ModelConfigError(f"{where}: cannot choose {r['top']} of {r['experts']} experts (at most 32)")

    def to_dict(self) -> dict:
        """The config.json this configuration round-trips through."""
        return {
            "architecture": self.architecture,
            "embedding": {"bigram": dict(self.bigram)},
            "layers": [copy.deepcopy(layer) for layer in self.layers],
            "norm": {"eps": self.norm_eps},
            "streams": self.streams,
            "vocab": self.vocab,
            "width": self.width,
        }
