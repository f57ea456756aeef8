"""Typed configuration of Bikovik, read from its own config.json keys.

A Bikovik folder names itself with `"architecture": "Bikovik"`.  `layers` lists the layers; each entry has a `type` (which mixer:
`attention`, softmax attention with mixed scores, a window and kept first positions; `hgrn2`, a matrix memory whose forget gate decides
what is written; `retention`, a matrix memory with a constant decay per head), the mixer's sizes and constants under `mixer` and its
feed-forward under `mlp` (null: none; `kind` `dense`).  `embedding.scale`, `logit_softcap`, `norm.eps`, `vocab` and `width` are
model-wide.  Every size and constant that can differ between models is read here and nowhere else.
"""
from __future__ import annotations

from dataclasses import dataclass
from typing import Optional, Tuple

from .errors import InvalidConfig
from .fasesun import _integer, _number, _object
from .metadata import metadata_from_json

ARCHITECTURE = "Bikovik"
MODEL_TYPE = "bikovik"
MIXER_TYPES = ("attention", "hgrn2", "retention")


@dataclass(frozen=True)
class TalkingAttentionConfig:
    heads: int
    kv_heads: int
    dim: int
    vdim: int
    scale: float
    window: int
    keep_first: int
    rot_base: float
    rot_dims: int
    v_mix: bool
    type: str = "attention"


@dataclass(frozen=True)
class ForgetMemoryConfig:
    heads: int
    dim: int
    vdim: int
    type: str = "hgrn2"


@dataclass(frozen=True)
class RetentionConfig:
    heads: int
    dim: int
    vdim: int
    decays: Tuple[float, ...]
    rot_base: float
    rot_dims: int
    type: str = "retention"


@dataclass(frozen=True)
class ClampedConfig:
    ff: int
    limit: float
    kind: str = "dense"


@dataclass(frozen=True)
class LayerConfig:
    mixer: object
    mlp: Optional[ClampedConfig]


def _rotation(raw: dict, where: str, dim: int) -> Tuple[float, int]:
    if raw.get("rot") is None:       # no entry: nothing is rotated
        return 1.0, 0
    rot = _object(raw, "rot", where)
    dims = _integer(rot, "dims", where + "rot.", 0)
    if dims % 2 or dims > dim:
        raise InvalidConfig(f"config.json: {where}rot.dims must be even and at most dim ({dim}), found {dims}")
    return (_number(rot, "base", where + "rot.") if dims else 1.0), dims


def _attention(raw: dict, where: str) -> TalkingAttentionConfig:
    heads, kv_heads, dim, vdim = (_integer(raw, key, where) for key in ("heads", "kv_heads", "dim", "vdim"))
    if heads % kv_heads:
        raise InvalidConfig(f"config.json: {where}heads ({heads}) must be a multiple of kv_heads ({kv_heads})")
    mask = _object(raw, "mask", where)
    base, dims = _rotation(raw, where, dim)
    v_mix = raw.get("v_mix", False)
    if not isinstance(v_mix, bool):
        raise InvalidConfig(f"config.json: {where}v_mix must be true or false, found {v_mix!r}")
    return TalkingAttentionConfig(heads, kv_heads, dim, vdim, _number(raw, "scale", where), _integer(mask, "size", where + "mask."),
                                  _integer(mask, "keep_first", where + "mask.", 0) if mask.get("keep_first") is not None else 0, base, dims, v_mix)


def _hgrn2(raw: dict, where: str) -> ForgetMemoryConfig:
    return ForgetMemoryConfig(*(_integer(raw, key, where) for key in ("heads", "dim", "vdim")))


def _retention(raw: dict, where: str) -> RetentionConfig:
    heads, dim, vdim = (_integer(raw, key, where) for key in ("heads", "dim", "vdim"))
    decay = raw.get("decay")
    if not isinstance(decay, list) or len(decay) != heads or any(isinstance(value, bool) or not isinstance(value, (int, float)) or not 0 <= value <= 1 for value in decay):
        raise InvalidConfig(f"config.json: {where}decay must list one number from 0 to 1 for each of the {heads} heads")
    return RetentionConfig(heads, dim, vdim, tuple(float(value) for value in decay), *_rotation(raw, where, dim))


_MIXERS = {"attention": _attention, "hgrn2": _hgrn2, "retention": _retention}


def _mlp(raw, where: str) -> Optional[ClampedConfig]:
    if raw is None:
        return None
    if not isinstance(raw, dict) or raw.get("kind") != "dense":
        raise InvalidConfig(f"config.json: {where} must be null or an object of kind 'dense'")
    return ClampedConfig(_integer(raw, "ff", where + "."), _number(raw, "limit", where + "."))


@dataclass(frozen=True)
class BikovikConfig:
    vocab: int
    width: int
    eps: float
    embedding_scale: float
    logit_softcap: float
    layers: Tuple[LayerConfig, ...]
    declared_dtype: Optional[str] = None

    architecture = ARCHITECTURE
    model_type = MODEL_TYPE

    @classmethod
    def from_json(cls, raw: dict) -> "BikovikConfig":
        metadata = metadata_from_json(raw)
        if metadata.architecture != ARCHITECTURE:
            raise InvalidConfig(f"expected {ARCHITECTURE}, found {metadata.architecture}")
        listed = raw.get("layers")
        if not isinstance(listed, list) or not listed:
            raise InvalidConfig("config.json: 'layers' must be a list with at least one layer")
        layers, mixed_width = [], None
        for index, entry in enumerate(listed):
            where = f"layers[{index}]."
            if not isinstance(entry, dict) or entry.get("type") not in MIXER_TYPES:
                raise InvalidConfig(f"config.json: {where}type must be one of {', '.join(MIXER_TYPES)}")
            mixer = _MIXERS[entry["type"]](_object(entry, "mixer", where), where + "mixer.")
            if mixer.type == "attention" and mixer.v_mix:
                width = mixer.kv_heads * mixer.vdim
                if mixed_width is not None and width != mixed_width:
                    raise InvalidConfig(f"config.json: {where}mixer has {width} numbers in a token's values; the first layer with v_mix has {mixed_width}")
                mixed_width = width
            layers.append(LayerConfig(mixer, _mlp(entry.get("mlp"), where + "mlp")))
        return cls(vocab=_integer(raw, "vocab", ""), width=_integer(raw, "width", ""), eps=_number(_object(raw, "norm", ""), "eps", "norm."),
                   embedding_scale=_number(_object(raw, "embedding", ""), "scale", "embedding.", positive=False),
                   logit_softcap=_number(raw, "logit_softcap", ""), layers=tuple(layers), declared_dtype=metadata.declared_dtype)


__all__ = ["ARCHITECTURE", "MODEL_TYPE", "BikovikConfig"]
