"""Typed configuration of the Vilulix design, read from its own config.json keys.

A Vilulix model is a list of layers around a float32 residual stream; a layer adds its mixer and its
feed-forward, both reading the same stream through norms of their own. A layer's mixer is "mlstm" (a
matrix memory with exponential gating), "latent_attention" (attention over a cached latent, queries
through a latent of their own) or "parallel" (attention in a sliding window beside a gated delta rule,
each with a factor); its feed-forward is dense or absent. `loop` names a stretch of layers that runs
several times with the same weights. Every size and every constant that may differ between models is a
key; what the design fixes is written in `models/vilulix.py`.
"""

from __future__ import annotations

import copy
from dataclasses import dataclass
from typing import Any

from atomserve_b200.config.gefilix_config import _need
from atomserve_b200.config.model_config import ModelConfigError

MIXERS = ("mlstm", "latent_attention", "parallel")


@dataclass(frozen=True)
class VilulixConfig:
    vocab: int
    width: int
    layers: tuple[dict[str, Any], ...]
    norm_eps: float
    logit_softcap: float | None = None
    loop: dict[str, int] | None = None
    max_positions: int = 1 << 20  # no learned or tabulated positions: no limit of the design's own

    architecture = "Vilulix"

    @classmethod
    def from_dict(cls, raw: dict) -> "VilulixConfig":
        name = raw.get("architecture") or (raw.get("architectures") or [None])[0]
        if name != cls.architecture:
            raise ModelConfigError(f"expected architecture {cls.architecture!r}, got {name!r}")
        _need(raw, ("vocab", "width", "layers", "norm"), "config.json")
        _need(raw["norm"], ("eps",), "config.json norm")
        loop = raw.get("loop")
        if loop is not None:
            _need(loop, ("start", "stop", "times"), "config.json loop")
            loop = {k: int(loop[k]) for k in ("start", "stop", "times")}
        cap = raw.get("logit_softcap")
        config = cls(
            vocab=int(raw["vocab"]),
            width=int(raw["width"]),
            layers=tuple(copy.deepcopy(layer) for layer in raw["layers"]),
            norm_eps=float(raw["norm"]["eps"]),
            logit_softcap=float(cap) if cap is not None else None,
            loop=loop,
            max_positions=int(raw.get("max_positions", 1 << 20)),
        )
        config.validate()
        return config

    def run_order(self) -> list[tuple[int, int | None]]:
        """(layer, the number of the pass it opens or None), in the order the layers run; the first pass
        of the loop opens with nothing, so it counts as None."""
        n = len(self.layers)
        if self.loop is None:
            return [(i, None) for i in range(n)]
        start, stop, times = self.loop["start"], self.loop["stop"], self.loop["times"]
        order: list[tuple[int, int | None]] = [(i, None) for i in range(start)]
        for t in range(times):
            order += [(i, t if t > 0 and i == start else None) for i in range(start, stop)]
        return order + [(i, None) for i in range(stop, n)]

    def validate(self) -> None:
        if self.vocab < 1 or self.width < 1 or not self.layers:
            raise ModelConfigError("vocab, width and the number of layers must be positive")
        if not self.norm_eps >= 0:
            raise ModelConfigError("norm.eps must be >= 0")
        if self.logit_softcap is not None and not self.logit_softcap > 0:
            raise ModelConfigError("logit_softcap must be positive")
        if self.loop is not None:
            start, stop, times = self.loop["start"], self.loop["stop"], self.loop["times"]
            if not 0 <= start < stop <= len(self.layers) or times < 1:
                raise ModelConfigError(f"loop {start}..{stop} x {times} does not fit {len(self.layers)} layers")
        for i, layer in enumerate(self.layers):
            where = f"layer {i}"
            _need(layer, ("type", "mixer"), where)
            if layer["type"] not in MIXERS:
                raise ModelConfigError(f"{where}: mixer type {layer['type']!r} is not one of {MIXERS}")
            getattr(self, "_check_" + layer["type"])(layer["mixer"], where)
            mlp = layer.get("mlp")
            if mlp is None:
                continue
            _need(mlp, ("kind", "ff"), where + " mlp")
            if mlp["kind"] != "dense":
                raise ModelConfigError(f"{where}: mlp kind {mlp['kind']!r} is not 'dense'")

    @staticmethod
    def _check_heads(m: dict, where: str) -> None:
        if m["heads"] < 1 or m["kv_heads"] < 1 or m["heads"] % m["kv_heads"]:
            raise ModelConfigError(f"{where}: {m['heads']} heads are not a multiple of {m['kv_heads']} kv heads")

    @staticmethod
    def _check_rotation(rot: dict, size: int, where: str) -> None:
        _need(rot, ("base", "dims"), where + " rot")
        if rot["dims"] % 2 or not 0 <= rot["dims"] <= size:
            raise ModelConfigError(f"{where}: rot.dims {rot['dims']} must be even and at most {size}")

    @staticmethod
    def _check_mlstm(m: dict, where: str) -> None:
        _need(m, ("heads", "dim", "vdim", "gate_cap"), where + " mixer")
        if not m["gate_cap"] > 0:
            raise ModelConfigError(f"{where}: gate_cap must be positive")

    @classmethod
    def _check_latent_attention(cls, m: dict, where: str) -> None:
        _need(m, ("heads", "dim", "rot_dim", "vdim", "kv_rank", "q_rank", "scale", "rot"), where + " mixer")
        if m["rot_dim"] < 2:
            raise ModelConfigError(f"{where}: rot_dim must be at least 2")
        cls._check_rotation(m["rot"], m["rot_dim"], where + " mixer")

    @classmethod
    def _check_parallel(cls, m: dict, where: str) -> None:
        _need(m, ("left", "right", "left_scale", "right_scale"), where + " mixer")
        left, right = m["left"], m["right"]
        _need(left, ("heads", "kv_heads", "dim", "vdim", "scale"), where + " mixer left")
        cls._check_heads(left, where + " left")
        if left.get("rot") is not None:
            cls._check_rotation(left["rot"], left["dim"], where + " left")
        if left.get("mask") is not None:
            _need(left["mask"], ("size",), where + " mixer left mask")
            if left["mask"]["size"] < 1:
                raise ModelConfigError(f"{where}: mask.size must be positive")
        _need(right, ("heads", "kv_heads", "dim", "vdim", "conv"), where + " mixer right")
        cls._check_heads(right, where + " right")
        if right["conv"] < 1:
            raise ModelConfigError(f"{where}: a convolution needs at least one tap")

    def to_dict(self) -> dict:
        """The config.json this configuration round-trips through."""
        out = {
            "architecture": self.architecture,
            "layers": [copy.deepcopy(layer) for layer in self.layers],
            "norm": {"eps": self.norm_eps},
            "vocab": self.vocab,
            "width": self.width,
        }
        if self.logit_softcap is not None:
            out["logit_softcap"] = self.logit_softcap
        if self.loop is not None:
            out["loop"] = dict(self.loop)
        return out
