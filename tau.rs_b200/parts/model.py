"""A decoder built from a `ModelSpec`: embedding, scheduled blocks, final norm, head.

The traversal is crates/models/src/qwen3_5_common/model.rs:168-195 (embed, each layer,
final norm) and :295-299,317-320 (the head is `lm_head.weight` or the embedding table
when tied; logits are computed only at the positions that are asked for).  Which blocks
run, in which order and on which cache layer is the spec's schedule, not code.
"""
from __future__ import annotations

from typing import Dict, Optional, Tuple

import torch

from ..config.specs import ModelSpec
from ..csrc import kernels
from ..weights.tensor_spec import TensorSpec
from .base import CacheNeed, Pending
from .registry import build


class DecoderModel:
    def __init__(self, spec: ModelSpec, dtype: torch.dtype, device):
        self.spec, self.dtype, self.device = spec, dtype, device
        self.residual_dtype = torch.float32 if getattr(spec, "residual_dtype", None) == "float32" else dtype
        self.blocks = [build("block", block, dtype=dtype, device=device) for block in spec.blocks]
        self.final_norm = build("norm", spec.final_norm, name=spec.final_norm_name, dtype=dtype, device=device)
        self.input_position = None if spec.input_position is None else build("position", spec.input_position, device=device)
        self.embedding: Optional[torch.Tensor] = None
        self.head: Optional[torch.Tensor] = None
        self._owner: Dict[str, object] = {}
        self._parts = (*self.blocks, self.final_norm) + (() if self.input_position is None else (self.input_position,))
        for part in self._parts:
            for name in part.tensor_specs():
                if name in self._owner:
                    raise ValueError(f"two parts ask for the tensor {name}")
                self._owner[name] = part
        for entry in spec.schedule:
            if not 0 <= entry.layer < len(self.blocks):
                raise ValueError(f"schedule names layer {entry.layer}, the model has {len(self.blocks)}")
            if getattr(entry, "joins_embedding", False) and (self.residual_dtype != torch.float32 or spec.input_position is not None):
                raise ValueError("the embedding output joins again on a stream kept in 32-bit and without an encoding added to it")
        self._groups = self._collect_cache_groups()
        self._shared = {name: TensorSpec(tuple(shape), role=role) for name, shape, role in getattr(spec, "shared_tensors", ())}
        self.shared: Dict[str, torch.Tensor] = {}
        for name in self._shared:
            if name in self._owner:
                raise ValueError(f"the shared tensor {name} is also a part's own")

    # ---- cache needs -------------------------------------------------------------
    def _collect_cache_groups(self) -> Dict[str, Tuple[CacheNeed, int]]:
        groups: Dict[str, Tuple[CacheNeed, int]] = {}
        written = set()
        for entry in self.spec.schedule:
            need = self.blocks[entry.layer].cache_need()
            if need is None:
                continue
            if entry.cache_group is None:
                raise ValueError(f"layer {entry.layer} keeps a cache but its schedule entry names no cache group")
            known = groups.get(entry.cache_group)
            if known is not None and known[0] != need:
                raise ValueError(f"cache group {entry.cache_group!r} is shared by layers with different needs")
            layers = max(known[1] if known else 0, entry.cache_layer + 1)
            groups[entry.cache_group] = (need, layers)
            key = (entry.cache_group, entry.cache_layer)
            if entry.writes_cache:
                written.add(key)
            elif key not in written:
                raise ValueError(f"schedule entry for layer {entry.layer} reads cache {key} before any entry writes it")
        # What blocks keep beside their mixers' caches: a group and a cache layer for every role that a block names.
        for entry in self.spec.schedule:
            needs = self.blocks[entry.layer].extra_cache_needs()
            named = {role: (group, layer) for role, group, layer in getattr(entry, "extra_cache", ())}
            if set(named) != set(needs):
                raise ValueError(f"layer {entry.layer} keeps {sorted(needs)} beside its mixer's cache; its schedule entry names {sorted(named)}")
            for role, need in needs.items():
                group, layer = named[role]
                known = groups.get(group)
                if known is not None and known[0] != need:
                    raise ValueError(f"cache group {group!r} is shared by layers with different needs")
                groups[group] = (need, max(known[1] if known else 0, layer + 1))
        return groups

    def cache_groups(self) -> Dict[str, Tuple[CacheNeed, int]]:
        """Group name -> (what each of its cache layers keeps, number of cache layers)."""
        return dict(self._groups)

    # ---- weights -----------------------------------------------------------------
    def tensor_specs(self) -> Dict[str, TensorSpec]:
        spec = self.spec
        specs = {spec.embedding_name: TensorSpec((spec.vocab_size, spec.hidden), role="matrix")}
        for part in self._parts:
            specs.update(part.tensor_specs())
        specs.update(self._shared)
        if not spec.tie_head:
            specs[spec.head_name] = TensorSpec((spec.vocab_size, spec.hidden), role="matrix", fallback=spec.embedding_name)
        return specs

    @staticmethod
    def tensor_specs_of(spec: ModelSpec) -> Dict[str, TensorSpec]:
        return DecoderModel(spec, torch.float32, "cpu").tensor_specs()

    def ignored_tensors(self):
        """A tied model may still carry a copy of the head; it is not read."""
        return {self.spec.head_name} if self.spec.tie_head else set()

    def assign(self, name: str, tensor: torch.Tensor) -> None:
        if name == self.spec.embedding_name:
            self.embedding = tensor
        elif name == self.spec.head_name and not self.spec.tie_head:
            self.head = tensor
        elif name in self._shared:
            self.shared[name] = tensor
        else:
            self._owner[name].assign(name, tensor)

    def finalize_weights(self) -> None:
        for block in self.blocks:
            for name in block.shared_tensor_names():
                block.bind_shared(name, self.shared[name])
        for part in self._parts:
            part.finalize_weights()
        if self.spec.tie_head:
            self.head = self.embedding
        scale = getattr(self.spec, "logit_scale", 1.0)
        if scale != 1.0:      # the head is linear: the last norm's weight (and bias) carry the logits' factor
            norm = self.final_norm
            norm.weight = (norm.weight * scale).contiguous()
            if getattr(norm, "bias", None) is not None:
                norm.bias = (norm.bias * scale).contiguous()

    def weight_bytes(self) -> int:
        """Bytes of weights that one step reads: what each part says it reads (every tensor once, unless a part knows
        better), the head, and nothing of the embedding table, which is read by row (it counts only where it is the head
        as well); a block that the schedule never names is left out."""
        scheduled = {entry.layer for entry in self.spec.schedule}
        total = sum(block.bytes_read_per_step(self.dtype) for index, block in enumerate(self.blocks) if index in scheduled)
        total += self.final_norm.bytes_read_per_step(self.dtype)
        return total + self.spec.vocab_size * self.spec.hidden * torch.empty((), dtype=self.dtype).element_size()

    def decode_splits(self, n_seqs: int, max_len: int) -> int:
        """Context splits for a decode step of `n_seqs` sequences (part of a captured graph's key)."""
        blocks = [count for count in (block.decode_blocks() for block in self.blocks) if count]
        return kernels.decode_splits(n_seqs, max_len, min(blocks)) if blocks else 1

    # ---- forward -----------------------------------------------------------------
    def forward(self, step, cache) -> Optional[torch.Tensor]:
        """Runs the step's tokens; returns 32-bit logits `[wanted, vocab]`, or None if nothing is wanted."""
        spec = self.spec
        if getattr(spec, "keeps_results", False):      # the embedding output and every run's result stay until the step ends
            step.results = torch.empty((len(spec.schedule) + 1, step.n_tokens, spec.hidden), dtype=self.residual_dtype, device=self.device)
            residual = step.results[0]
        else:
            residual = torch.empty((step.n_tokens, spec.hidden), dtype=self.residual_dtype, device=self.device)
        kernels.embedding(step.token_ids, self.embedding, residual, getattr(spec, "embedding_scale", 1.0))
        if self.input_position is not None:
            self.input_position.add_to(residual, step)
        branch = None
        for run, entry in enumerate(spec.schedule):
            view = None if entry.cache_group is None else cache.layer_view(entry.cache_group, entry.cache_layer)
            extra = getattr(entry, "extra_cache", ())
            if extra:
                if view is None:
                    raise ValueError("a block that keeps something beside its mixer's cache needs that cache as well")
                view.extra = {role: cache.layer_view(group, layer) for role, group, layer in extra}
            step.run = run
            if getattr(entry, "joins_embedding", False):      # looked up again by the norm that adds it, so that no copy is kept
                branch = Pending.with_rows(branch, (self.embedding, step.token_ids, getattr(spec, "embedding_scale", 1.0)))
            residual, branch = self.blocks[entry.layer].forward(residual, branch, step, view, entry.writes_cache)
        step.results = None
        step.handed_on.clear()
        if step.n_wanted == 0:
            return None
        normalized = self.final_norm.forward(residual, rows=step.want_rows, branch=branch)
        logits = torch.empty((step.n_wanted, spec.vocab_size), dtype=torch.float32, device=self.device)
        kernels.linear(normalized, self.head, None, logits)
        if getattr(spec, "logit_cap", 0.0):
            kernels.soft_cap(logits, spec.logit_cap)
        return logits
