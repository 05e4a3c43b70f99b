"""Typed configuration of the Safupel decoder, read from its own config.json keys.

config.json gives ``vocab``, ``width``, ``norm.eps``, ``logit_scale`` and a list ``layers``.  A layer names its mixer
``type`` ("rglru": a real-gated linear recurrence; "parallel": chunked attention and matrix memory side by side), the
mixer's sizes and constants under ``mixer`` (``width``, ``blocks``, ``conv``; or ``left``: ``heads``, ``kv_heads``, ``dim``,
``vdim``, ``scale``, ``mask.size``, ``right``: ``heads``, ``dim``, ``vdim``, ``gate_cap``, and ``left_scale`` / ``right_scale``),
and its feed-forward under ``mlp`` (null: none; ``kind`` "dense" with ``ff``; ``kind`` "moe" with ``expert.ff``,
``router.experts`` / ``router.top`` and optionally ``shared.ff``).  Every size and constant of a model comes from this
object.
"""

from __future__ import annotations

import math
from dataclasses import dataclass
from typing import Any

from tokasaurus_b200.config.daborax_config import _number, _pos_int
from tokasaurus_b200.config.model_config import ConfigError


@dataclass(frozen=True)
class GatedRecurrenceConfig:
    width: int
    blocks: int
    taps: int

    @staticmethod
    def from_dict(d: dict, where: str) -> "GatedRecurrenceConfig":
        width, blocks = _pos_int(d, "width", where), _pos_int(d, "blocks", where)
        if width % blocks:
            raise ConfigError(f"{where}: width={width} does not divide into blocks={blocks} equal parts")
        return GatedRecurrenceConfig(width, blocks, _pos_int(d, "conv", where))


@dataclass(frozen=True)
class ChunkedAttentionConfig:
    heads: int
    kv_heads: int
    dim: int
    vdim: int
    scale: float
    chunk: int | None

    @staticmethod
    def from_dict(d: dict, where: str) -> "ChunkedAttentionConfig":
        heads, dim = _pos_int(d, "heads", where), _pos_int(d, "dim", where)
        kv_heads = _pos_int(d, "kv_heads", where) if "kv_heads" in d else heads
        if heads % kv_heads:
            raise ConfigError(f"{where}: {heads} heads are no multiple of {kv_heads} kv_heads")
        mask = d.get("mask") or {}
        chunk = _pos_int(mask, "size", where + ".mask") if mask.get("size") is not None else None
        return ChunkedAttentionConfig(heads, kv_heads, dim, _pos_int(d, "vdim", where) if "vdim" in d else dim,
                                      _number(d, "scale", where, 1.0 / math.sqrt(dim)), chunk)


@dataclass(frozen=True)
class MatrixMemoryConfig:
    heads: int
    dim: int
    vdim: int
    gate_cap: float

    @staticmethod
    def from_dict(d: dict, where: str) -> "MatrixMemoryConfig":
        dim = _pos_int(d, "dim", where)
        cap = _number(d, "gate_cap", where)
        if cap <= 0:
            raise ConfigError(f"{where}.gate_cap must be positive, got {cap!r}")
        return MatrixMemoryConfig(_pos_int(d, "heads", where), dim, _pos_int(d, "vdim", where) if "vdim" in d else dim, cap)


@dataclass(frozen=True)
class ParallelConfig:
    left: ChunkedAttentionConfig
    right: MatrixMemoryConfig
    left_scale: float
    right_scale: float

    @staticmethod
    def from_dict(d: dict, where: str) -> "ParallelConfig":
        for side in ("left", "right"):
            if not isinstance(d.get(side), dict):
                raise ConfigError(f"{where}.{side} must give the sizes of the mixer on that side")
        return ParallelConfig(ChunkedAttentionConfig.from_dict(d["left"], where + ".left"),
                              MatrixMemoryConfig.from_dict(d["right"], where + ".right"),
                              _number(d, "left_scale", where, 1.0), _number(d, "right_scale", where, 1.0))


@dataclass(frozen=True)
class FeedForwardConfig:
    kind: str  # "dense" or "moe"
    ff: int
    experts: int = 0
    top: int = 0
    shared_ff: int | None = None

    @staticmethod
    def from_dict(d: dict | None, where: str) -> "FeedForwardConfig | None":
        if d is None:
            return None
        kind = d.get("kind")
        if kind == "dense":
            return FeedForwardConfig("dense", _pos_int(d, "ff", where))
        if kind != "moe":
            raise ConfigError(f"{where}.kind={kind!r} is not known ('dense', 'moe')")
        r, sh = d.get("router") or {}, d.get("shared")
        experts, top = _pos_int(r, "experts", where + ".router"), _pos_int(r, "top", where + ".router")
        if top > experts:
            raise ConfigError(f"{where}.router: top={top} of {experts} experts")
        return FeedForwardConfig("moe", _pos_int(d.get("expert") or {}, "ff", where + ".expert"), experts, top,
                                 _pos_int(sh, "ff", where + ".shared") if sh else None)


_MIXERS = {"rglru": GatedRecurrenceConfig, "parallel": ParallelConfig}


@dataclass(frozen=True)
class SafupelLayerConfig:
    type: str
    mixer: GatedRecurrenceConfig | ParallelConfig
    mlp: FeedForwardConfig | None


@dataclass(frozen=True)
class SafupelConfig:
    vocab: int
    width: int
    norm_eps: float
    logit_scale: float
    layers: tuple[SafupelLayerConfig, ...]
    eos_token_id: tuple[int, ...] = ()

    @property
    def vocab_size(self) -> int:
        return self.vocab

    @staticmethod
    def from_dict(d: dict[str, Any]) -> "SafupelConfig":
        for key in ("vocab", "width", "layers"):
            if key not in d:
                raise ConfigError(f"config.json lacks the key {key!r}")
        if not isinstance(d["layers"], list) or not d["layers"]:
            raise ConfigError("config.json: 'layers' must be a non-empty list")
        layers = []
        for i, ld in enumerate(d["layers"]):
            where = f"layers[{i}]"
            kind = ld.get("type")
            if kind not in _MIXERS:
                raise ConfigError(f"{where}.type={kind!r} is not known ({', '.join(repr(k) for k in _MIXERS)})")
            layers.append(SafupelLayerConfig(kind, _MIXERS[kind].from_dict(ld.get("mixer") or {}, where + ".mixer"),
                                             FeedForwardConfig.from_dict(ld.get("mlp"), where + ".mlp")))
        eps = float((d.get("norm") or {}).get("eps", 1e-6))
        if not (eps > 0 and math.isfinite(eps)):
            raise ConfigError(f"norm.eps must be positive and finite, got {eps!r}")
        eos = d.get("eos_token_id")
        eos_t = () if eos is None else ((eos,) if isinstance(eos, int) else tuple(int(e) for e in eos))
        return SafupelConfig(vocab=_pos_int(d, "vocab", "config"), width=_pos_int(d, "width", "config"), norm_eps=eps,
                             logit_scale=_number(d, "logit_scale", "config", 1.0), layers=tuple(layers),
                             eos_token_id=eos_t)
