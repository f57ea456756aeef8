"""Interfaces of the parts.

A part owns its weights (declared by name through `tensor_specs`, received through
`assign`) and a `forward`.  Activations are packed: row `i` of every activation tensor
belongs to token `i` of the step, whichever sequence it is from; `StepContext` says
which sequence and which position each row has.
"""
from __future__ import annotations

from dataclasses import dataclass
from typing import Dict, Optional, Tuple

import torch

from ..weights.tensor_spec import TensorSpec


@dataclass(frozen=True)
class CacheNeed:
    """What a mixer wants the cache to keep for it, per cache layer.

    `kind == "kv"`: keys and values of `n_kv_heads` heads of `head_dim` elements for
    every position (or for the last `window` positions).  `kind == "rows"`: one row of
    `row_width` elements for every position (or for the last `window`), paged like keys
    and values (a latent that keys and values are expanded from, say).  With `chunk` a
    query reads only the positions of its own chunk of `chunk` positions (chunks counted from
    position 0), so that what lies before the newest chunk need not be kept.  `kind == "state"`:
    one tensor of `state_shape` and `state_dtype` for each sequence, zero when the sequence
    starts, whatever its length.  `keep_first` (beside a window): the first that many positions
    are read by every query and kept as long as the sequence lives.
    """

    kind: str
    n_kv_heads: int = 0
    head_dim: int = 0
    window: Optional[int] = None
    state_shape: Tuple[int, ...] = ()
    state_dtype: torch.dtype = torch.float32
    row_width: int = 0
    chunk: Optional[int] = None
    keep_first: int = 0


class Pending(tuple):
    """What has yet to join the residual stream: results (up to two tensors), the factors that they join it with (one number, and a
    32-bit vector over the channels or None), and rows of a table (None, or `(table, row numbers, factor)`): the norm that adds them
    computes `stream + scale * channel_scale * (sum of the results) + factor * table[row numbers]`."""

    scale, channel_scale, rows = 1.0, None, None

    def __new__(cls, results, scale: float = 1.0, channel_scale=None, rows=None):
        pending = super().__new__(cls, results)
        pending.scale, pending.channel_scale, pending.rows = float(scale), channel_scale, rows
        return pending

    @classmethod
    def with_rows(cls, branch, rows) -> "Pending":
        """`branch` (None, a tensor, a tuple or a Pending) and the rows of a table beside it."""
        results = () if branch is None else tuple(branch) if isinstance(branch, (tuple, list)) else (branch,)
        if getattr(branch, "rows", None) is not None:
            raise ValueError("rows of a table are pending already")
        return cls(results, getattr(branch, "scale", 1.0), getattr(branch, "channel_scale", None), rows)


def require_plain_pending(branch) -> None:
    """For norms that add results alone: refuses a factor per channel and rows of a table."""
    if getattr(branch, "channel_scale", None) is not None or getattr(branch, "rows", None) is not None:
        raise ValueError("a norm of this kind adds results with one factor; a factor per channel or rows of a table are not served")


class Part:
    def tensor_specs(self) -> Dict[str, TensorSpec]:
        return {}

    def assign(self, name: str, tensor: torch.Tensor) -> None:
        raise KeyError(name)

    def finalize_weights(self) -> None:
        pass

    def bytes_read_per_step(self, dtype) -> int:
        """Bytes of this part's weights that one step reads: every tensor once, unless the part knows better (a feed-forward
        that routes each token to a few of its experts reads only those).  The roofline of a decode step is built on it."""
        from ..weights.loader import device_dtype

        total = 0
        for spec in self.tensor_specs().values():
            count = 1
            for extent in spec.shape:
                count *= extent
            total += count * torch.empty((), dtype=device_dtype(spec, dtype)).element_size()
        return total


class Mixer(Part):
    """Mixes information between the tokens of a sequence.

    `forward(hidden, step, cache, writes_cache)` takes `[tokens, hidden]` and returns
    the same shape.  `cache` is the view of this run's cache layer (`KVLayerView` or
    `StateLayerView`), or None if `cache_need()` is None.
    """

    # False: a decode step through this mixer cannot be captured in a CUDA graph (its `forward` reads device values on the
    # host, say); an engine whose model has such a part runs its decode steps launch by launch.
    capturable = True

    def cache_need(self) -> Optional[CacheNeed]:
        return None

    def decode_blocks(self) -> Optional[int]:
        """Blocks that the mixer's decode kernel launches per sequence and context split, where the mixer splits the
        context of a decode step at all (None: it does not).  The number of splits is chosen so that all blocks of a step
        are resident at once, and it is part of a captured graph's key."""
        return None

    def extra_cache_needs(self) -> Dict[str, CacheNeed]:
        """What the mixer keeps for a sequence beside `cache_need()`, by role (the tail of inputs of a convolution, say); `forward`
        finds the views under `cache.extra[role]`.  The block hands the roles on (`Block.extra_cache_needs`)."""
        return {}

    def forward(self, hidden, step, cache, writes_cache: bool):
        raise NotImplementedError


class FeedForward(Part):
    """`forward(hidden, step)`: `[tokens, hidden] -> [tokens, hidden]`, token by token."""

    capturable = True   # as for a mixer

    def forward(self, hidden, step):
        raise NotImplementedError


class Norm(Part):
    """`forward(x, rows=None, branch=None)` normalises rows (optionally only the rows listed,
    optionally of `x + branch` rounded to the storage dtype); `x` is left as it is.

    `add_forward(branch, residual)` rounds `residual + branch` into `residual` and
    returns its normalisation, as one fused operation.
    """

    def forward(self, values, rows=None, branch=None):
        raise NotImplementedError

    def add_forward(self, branch, residual):
        raise NotImplementedError


class Block(Part):
    """Arrangement of a mixer and a feed-forward around the residual stream.

    The residual stream travels as a pair `(residual, branch)` whose sum is the hidden
    state, so that the sum can be fused with the next norm wherever that is.
    `forward(residual, branch, step, cache, writes_cache) -> (residual, branch)`.
    """

    capturable = True   # False if a part of the block is not

    def cache_need(self) -> Optional[CacheNeed]:
        return None

    def decode_blocks(self) -> Optional[int]:
        """The mixer's answer (see `Mixer.decode_blocks`)."""
        return None

    def extra_cache_needs(self) -> Dict[str, CacheNeed]:
        """What the block keeps for a sequence beside its mixer's cache, by role (the tail of inputs of a convolution, say).  The
        schedule entry names a cache group and layer for each role (`ScheduleEntry.extra_cache`); `forward` finds the views under
        `cache.extra[role]`."""
        return {}

    def shared_tensor_names(self) -> Tuple[str, ...]:
        """Names among `ModelSpec.shared_tensors` that the block reads; the model hands each over through `bind_shared`."""
        return ()

    def bind_shared(self, name: str, tensor) -> None:
        raise KeyError(name)

    def forward(self, residual, branch, step, cache, writes_cache: bool):
        raise NotImplementedError
