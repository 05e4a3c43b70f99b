"""Typed configuration of the Deletar decoder, read from its own config.json keys.

config.json gives ``vocab``, ``width``, ``norm.eps``, ``embedding.scale``, optionally ``logit_softcap``, and a list
``layers``.  A layer names its mixer ``type`` ("attention", "attention_2" or "attention_3"), the mixer's sizes and constants
under ``mixer`` (``heads``, ``kv_heads``, ``dim``, ``vdim``, ``scale``, ``mask.size``, ``rot.base`` / ``rot.dims`` /
``rot.scaling``: ``factor``, ``low``, ``high``, ``original``; ``conv``: the taps of "attention"; ``softcap`` of the two
others; ``kv_from``: the layer whose cached keys and values are read), and its feed-forward under ``mlp`` (null: none;
``kind`` "dense" with ``ff``; ``kind`` "moe" with ``expert.ff``, ``router.experts`` / ``router.top`` and optionally
``shared.ff``).  Every size and constant of a model comes from this object.
"""

from __future__ import annotations

import math
from dataclasses import dataclass
from typing import Any

from tokasaurus_b200.config.daborax_config import _number, _pos_int
from tokasaurus_b200.config.model_config import ConfigError


@dataclass(frozen=True)
class RotationScaling:
    """Long wavelengths divided by ``factor``, short ones kept, a blend between ``original / high`` and ``original / low``."""

    factor: float
    low: float
    high: float
    original: float


@dataclass(frozen=True)
class Rotation:
    dims: int
    base: float
    scaling: RotationScaling | None

    @staticmethod
    def from_dict(d: dict | None, most: int, where: str) -> "Rotation | None":
        if d is None:
            return None
        dims = d.get("dims", most)
        if not isinstance(dims, int) or isinstance(dims, bool) or dims < 0 or dims > most or dims % 2:
            raise ConfigError(f"{where}.dims must be an even number from 0 to {most}, got {dims!r}")
        base = _number(d, "base", where, 10000.0)
        if base <= 0:
            raise ConfigError(f"{where}.base must be positive, got {base!r}")
        scaling = None
        sc = d.get("scaling")
        if sc is not None:
            w = where + ".scaling"
            scaling = RotationScaling(_number(sc, "factor", w), _number(sc, "low", w), _number(sc, "high", w),
                                      _number(sc, "original", w))
            if min(scaling.factor, scaling.low, scaling.high, scaling.original) <= 0 or scaling.high < scaling.low:
                raise ConfigError(f"{w}: positive numbers with low <= high are wanted, got {scaling}")
        return Rotation(dims, base, scaling) if dims else None


def _positive_or_none(d: dict, key: str, where: str) -> float | None:
    if d.get(key) is None:
        return None
    v = _number(d, key, where)
    if v <= 0:
        raise ConfigError(f"{where}.{key} must be positive, got {v!r}")
    return v


@dataclass(frozen=True)
class AttentionConfig:
    heads: int
    kv_heads: int
    dim: int
    vdim: int
    scale: float
    window: int | None
    rot: Rotation | None
    taps: int | None       # "attention": the short convolution's
    softcap: float | None  # the others: the cap on the scores
    kv_from: int | None

    @staticmethod
    def from_dict(kind: str, d: dict, where: str) -> "AttentionConfig":
        heads, dim = _pos_int(d, "heads", where), _pos_int(d, "dim", where)
        kv_heads = _pos_int(d, "kv_heads", where) if "kv_heads" in d else heads
        if heads % kv_heads:
            raise ConfigError(f"{where}: {heads} heads are no multiple of {kv_heads} kv_heads")
        vdim = _pos_int(d, "vdim", where) if "vdim" in d else dim
        if kind == "attention_2" and vdim != dim:
            raise ConfigError(f"{where}: values that are the keys have the keys' size {dim}, not {vdim}")
        mask = d.get("mask") or {}
        window = _pos_int(mask, "size", where + ".mask") if mask.get("size") is not None else None
        kv_from = d.get("kv_from")
        if kv_from is not None and (not isinstance(kv_from, int) or isinstance(kv_from, bool) or kv_from < 0):
            raise ConfigError(f"{where}.kv_from must name a layer, got {kv_from!r}")
        return AttentionConfig(
            heads, kv_heads, dim, vdim, _number(d, "scale", where, 1.0 / math.sqrt(dim)), window,
            Rotation.from_dict(d.get("rot"), dim, where + ".rot"),
            _pos_int(d, "conv", where) if kind == "attention" else None,
            None if kind == "attention" else _positive_or_none(d, "softcap", where), kv_from)


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


MIXER_TYPES = ("attention", "attention_2", "attention_3")


@dataclass(frozen=True)
class DeletarLayerConfig:
    type: str
    mixer: AttentionConfig
    mlp: FeedForwardConfig | None


@dataclass(frozen=True)
class DeletarConfig:
    vocab: int
    width: int
    norm_eps: float
    embedding_scale: float
    logit_softcap: float | None
    layers: tuple[DeletarLayerConfig, ...]
    eos_token_id: tuple[int, ...] = ()

    @property
    def vocab_size(self) -> int:
        return self.vocab

    @staticmethod
    def from_dict(d: dict[str, Any]) -> "DeletarConfig":
        for key in ("vocab", "width", "layers"):
            if key not in d:
                raise ConfigError(f"config.json lacks the key {key!r}")
        if not isinstance(d["layers"], list) or not d["layers"]:
            raise ConfigError("config.json: 'layers' must be a non-empty list")
        layers: list[DeletarLayerConfig] = []
        for i, ld in enumerate(d["layers"]):
            where = f"layers[{i}]"
            kind = ld.get("type")
            if kind not in MIXER_TYPES:
                raise ConfigError(f"{where}.type={kind!r} is not known ({', '.join(repr(k) for k in MIXER_TYPES)})")
            m = AttentionConfig.from_dict(kind, ld.get("mixer") or {}, where + ".mixer")
            if m.kv_from is not None:
                src = layers[m.kv_from].mixer if m.kv_from < i else None
                if src is None or src.kv_from is not None:
                    raise ConfigError(f"{where}.mixer.kv_from={m.kv_from} must name an earlier layer that makes its own keys")
                if (src.kv_heads, src.dim, src.vdim, src.rot) != (m.kv_heads, m.dim, m.vdim, m.rot):
                    raise ConfigError(f"{where} reads layer {m.kv_from}'s keys but differs in kv_heads, dim, vdim or rotation")
            layers.append(DeletarLayerConfig(kind, m, FeedForwardConfig.from_dict(ld.get("mlp"), where + ".mlp")))
        eps = float((d.get("norm") or {}).get("eps", 1e-6))
        if not (eps > 0 and math.isfinite(eps)):
            raise ConfigError(f"norm.eps must be positive and finite, got {eps!r}")
        eos = d.get("eos_token_id")
        eos_t = () if eos is None else ((eos,) if isinstance(eos, int) else tuple(int(e) for e in eos))
        return DeletarConfig(vocab=_pos_int(d, "vocab", "config"), width=_pos_int(d, "width", "config"), norm_eps=eps,
                             embedding_scale=_number(d.get("embedding") or {}, "scale", "embedding", 1.0),
                             logit_softcap=_positive_or_none(d, "logit_softcap", "config"), layers=tuple(layers),
                             eos_token_id=eos_t)
