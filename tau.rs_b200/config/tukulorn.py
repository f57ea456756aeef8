"""Typed configuration of Tukulorn, read from its own config.json keys.

A Tukulorn folder names itself with `"architecture": "Tukulorn"`.  `layers` lists the layers; each entry has a `type` (which mixer:
`attention`, a differential attention with biases and a query temperature; `latent_attention`, an attention over a cached latent with a
sliding window and a gate per head), the mixer's sizes and constants under `mixer` and its feed-forward under `mlp` (null: none; `kind`
`dense` or `moe`, the latter with a router that chooses among groups of experts).  `loop` makes the layers `start .. stop-1` run `times`
times in a row with the same weights.  `norm.eps`, `vocab` and `width` are model-wide.  Every size and constant that can differ between
models is read here and nowhere else.
"""
from __future__ import annotations

from dataclasses import dataclass
from typing import Optional, Tuple

from .errors import InvalidConfig
from .fasesun import _integer, _number, _object
from .metadata import metadata_from_json

ARCHITECTURE = "Tukulorn"
MODEL_TYPE = "tukulorn"
MIXER_TYPES = ("attention", "latent_attention")


@dataclass(frozen=True)
class BiasedDifferentialConfig:
    heads: int
    kv_heads: int
    dim: int
    vdim: int
    scale: float
    diff: float
    temperature: Optional[Tuple[float, int]]      # (coef, every); None: queries stay as they are
    type: str = "attention"


@dataclass(frozen=True)
class WindowedLatentConfig:
    heads: int
    dim: int
    rot_dim: int
    vdim: int
    kv_rank: int
    scale: float
    window: Optional[int]
    rot_base: float
    rot_dims: int
    type: str = "latent_attention"


@dataclass(frozen=True)
class DenseConfig:
    ff: int
    kind: str = "dense"


@dataclass(frozen=True)
class GroupedMoEConfig:
    experts: int
    top: int
    groups: int
    keep: int
    scale: float
    expert_ff: int
    limit: float
    kind: str = "moe"


@dataclass(frozen=True)
class LayerConfig:
    mixer: object
    mlp: Optional[object]


def _attention(raw: dict, where: str) -> BiasedDifferentialConfig:
    heads, kv_heads, dim, vdim = (_integer(raw, key, where) for key in ("heads", "kv_heads", "dim", "vdim"))
    if heads % kv_heads:
        raise InvalidConfig(f"config.json: {where}heads ({heads}) must be a multiple of kv_heads ({kv_heads})")
    temperature = None
    if raw.get("q_temp") is not None:
        listed = _object(raw, "q_temp", where)
        temperature = (_number(listed, "coef", where + "q_temp.", positive=False), _integer(listed, "every", where + "q_temp."))
    return BiasedDifferentialConfig(heads, kv_heads, dim, vdim, _number(raw, "scale", where), _number(raw, "diff", where, positive=False), temperature)


def _latent_attention(raw: dict, where: str) -> WindowedLatentConfig:
    heads, dim, rot_dim, vdim, kv_rank = (_integer(raw, key, where) for key in ("heads", "dim", "rot_dim", "vdim", "kv_rank"))
    rot = _object(raw, "rot", where)
    rot_dims = _integer(rot, "dims", where + "rot.", 0)
    if rot_dims % 2 or rot_dims > rot_dim:
        raise InvalidConfig(f"config.json: {where}rot.dims must be even and at most rot_dim ({rot_dim}), found {rot_dims}")
    window = None if raw.get("mask") is None else _integer(_object(raw, "mask", where), "size", where + "mask.")
    return WindowedLatentConfig(heads, dim, rot_dim, vdim, kv_rank, _number(raw, "scale", where), window,
                                _number(rot, "base", where + "rot.") if rot_dims else 1.0, rot_dims)


_MIXERS = {"attention": _attention, "latent_attention": _latent_attention}


def _mlp(raw, where: str):
    if raw is None:
        return None
    if not isinstance(raw, dict) or raw.get("kind") not in ("dense", "moe"):
        raise InvalidConfig(f"config.json: {where} must be null or an object of kind 'dense' or 'moe'")
    if raw["kind"] == "dense":
        return DenseConfig(_integer(raw, "ff", where + "."))
    router, expert = _object(raw, "router", where + "."), _object(raw, "expert", where + ".")
    experts, top = _integer(router, "experts", where + ".router."), _integer(router, "top", where + ".router.")
    groups = keep = 1
    if router.get("groups") is not None:
        listed = _object(router, "groups", where + ".router.")
        groups, keep = _integer(listed, "count", where + ".router.groups."), _integer(listed, "keep", where + ".router.groups.")
    if experts % groups or keep > groups:
        raise InvalidConfig(f"config.json: {where}.router.groups must cut the {experts} experts into equal groups and keep at most all of them")
    if top > keep * (experts // groups):
        raise InvalidConfig(f"config.json: {where}.router.top ({top}) exceeds the experts of the groups that are kept ({keep * (experts // groups)})")
    return GroupedMoEConfig(experts, top, groups, keep, _number(router, "scale", where + ".router."), _integer(expert, "ff", where + ".expert."),
                            _number(expert, "limit", where + ".expert."))


@dataclass(frozen=True)
class TukulornConfig:
    vocab: int
    width: int
    eps: float
    layers: Tuple[LayerConfig, ...]
    loop_start: int
    loop_stop: int
    loop_times: int
    declared_dtype: Optional[str] = None

    architecture = ARCHITECTURE
    model_type = MODEL_TYPE

    def layer_runs(self) -> Tuple[Tuple[int, bool], ...]:
        """The layers in the order in which they run, and whether a run opens a pass of the loop other than the first."""
        passes = [(index, turn > 0 and index == self.loop_start) for turn in range(self.loop_times) for index in range(self.loop_start, self.loop_stop)]
        return (*((index, False) for index in range(self.loop_start)), *passes, *((index, False) for index in range(self.loop_stop, len(self.layers))))

    @classmethod
    def from_json(cls, raw: dict) -> "TukulornConfig":
        metadata = metadata_from_json(raw)
        if metadata.architecture != ARCHITECTURE:
            raise InvalidConfig(f"expected {ARCHITECTURE}, found {metadata.architecture}")
        listed = raw.get("layers")
        if not isinstance(listed, list) or not listed:
            raise InvalidConfig("config.json: 'layers' must be a list with at least one layer")
        layers = []
        for index, entry in enumerate(listed):
            where = f"layers[{index}]."
            if not isinstance(entry, dict) or entry.get("type") not in MIXER_TYPES:
                raise InvalidConfig(f"config.json: {where}type must be one of {', '.join(MIXER_TYPES)}")
            layers.append(LayerConfig(_MIXERS[entry["type"]](_object(entry, "mixer", where), where + "mixer."), _mlp(entry.get("mlp"), where + "mlp")))
        start, stop, times = 0, 0, 1
        if raw.get("loop") is not None:
            loop = _object(raw, "loop", "")
            start, stop, times = _integer(loop, "start", "loop.", 0), _integer(loop, "stop", "loop.", 0), _integer(loop, "times", "loop.", 1)
            if not start <= stop <= len(layers):
                raise InvalidConfig(f"config.json: loop must satisfy 0 <= start <= stop <= {len(layers)}")
        return cls(vocab=_integer(raw, "vocab", ""), width=_integer(raw, "width", ""), eps=_number(_object(raw, "norm", ""), "eps", "norm."),
                   layers=tuple(layers), loop_start=start, loop_stop=stop, loop_times=times, declared_dtype=metadata.declared_dtype)


__all__ = ["ARCHITECTURE", "MODEL_TYPE", "TukulornConfig"]
