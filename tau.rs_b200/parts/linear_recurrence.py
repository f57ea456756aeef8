"""Mixers with a matrix state per head that is carried from token to token: `S_t = a_t S_(t-1) + b_t k_t v_t^T`, read `S_t^T q_t`.

Three gatings (`LinearRecurrenceSpec.gating`):

* `"decay"` (lightning attention): `a_t` is a constant per head, `b_t = 1`; q, k and v pass through SiLU; the concatenated
  heads are divided by their common root mean square.
* `"exponential"` (the matrix memory of xLSTM, mLSTM): a log input gate `i = cap tanh((W_i h + b_i) / cap)` and a log forget
  gate `f = logsigmoid(cap tanh((W_f h + b_f) / cap))` per head; a running maximum `m_t = max(f + m_(t-1), i)` starting at 0;
  `a_t = exp(f + m_(t-1) - m_t)`, `b_t = exp(i - m_t)`; a normaliser `n_t` with the same recurrence over `k` alone; the
  read-out is divided by `max(|n_t . q_t|, exp(-m_t)) + 1e-6`; queries are scaled by `key_dim^-1/2`; each head is divided
  by its own root mean square.

* `"forget"` (HGRN2): the forget gate decides what is written as well, `S_t = diag(f_t) S_(t-1) + (1 - f_t) v_t^T` per head, with
  `f = l + (1 - l) sigmoid(W_f h + b_f)` per head and key channel and `l` the channel's lower bound; queries pass through SiLU.

With `position` queries and keys are turned by it and `key_scale` multiplies the keys behind that (retention: `"decay"` with a
rotation, `key_dim^-1/2`, no activation, no norm weight and a SiLU gate).

All end the same way: divided by the root mean square, times the weight `norm` (all heads' width, or one head's width shared by the
heads, or none), times `sigmoid(W_g h)` or `silu(W_g h)` if there is a gate, then `W_o`.  The state is
32-bit, zero when a sequence starts, and lives in the cache's state group; gates, decays, exponentials, the state and the
norms are computed in 32-bit, the projections in the run's dtype.  One kernel walks a run of new tokens of any length, so
prompts, parts of prompts and single tokens are the same code: `linear_recurrence` for the exponential gating and for decays behind
an activation; the walk of `wkv`, which takes several tokens between two barriers, for the forget gating and for plain or turned
queries and keys, whose projections then leave their product in 32-bit.  Tensor names under the prefix: `q`, `k`, `v`, `g`, `o`,
`norm`, for the exponential gates `i`, `i.b`, `f`, `f.b`, for the forget gate `f`, `f.b`, `lower`.
"""
from __future__ import annotations

import torch

from ..csrc import kernels
from ..weights.tensor_spec import TensorSpec
from .base import CacheNeed, Mixer
from .linear import StackedLinear
from .registry import build, register_mixer


@register_mixer("linear_recurrence")
class LinearRecurrence(Mixer):
    def __init__(self, spec, prefix: str, dtype, device):
        if spec.gating not in ("decay", "exponential", "forget"):
            raise ValueError(f"unknown gating {spec.gating!r}")
        if spec.norm_groups not in ("head", "all"):
            raise ValueError(f"unknown norm_groups {spec.norm_groups!r}")
        if spec.gating == "decay" and len(spec.decays) != spec.n_heads:
            raise ValueError("one decay per head is needed")
        if spec.activation not in (None, "silu"):
            raise ValueError(f"unknown activation {spec.activation!r}")
        if spec.norm_weight not in (None, "full", "head"):
            raise ValueError(f"unknown norm_weight {spec.norm_weight!r}")
        if spec.gate_activation not in (None, "sigmoid", "silu"):
            raise ValueError(f"unknown gate_activation {spec.gate_activation!r}")
        if not 1 <= spec.key_dim <= kernels.RECURRENCE_MAX_KEY_DIM:
            raise ValueError(f"key_dim must lie between 1 and {kernels.RECURRENCE_MAX_KEY_DIM}")
        self.forget = spec.gating == "forget"
        self.exponential = spec.gating == "exponential"
        self.walked = self.forget or (spec.gating == "decay" and spec.activation is None)     # by `kernels.wkv`, from projections in 32-bit
        if (spec.position is not None or spec.key_scale != 1.0) and (not self.walked or self.forget):
            raise ValueError("a rotation or a key scale needs constant decays without an activation")
        if spec.position is not None and spec.position.rotary_dim > spec.key_dim:
            raise ValueError("the rotation is wider than a head")
        if self.walked and spec.query_scale != 1.0:
            raise ValueError("this gating has no query scale")
        self.spec, self.prefix, self.device = spec, prefix, device
        self.k_width, self.v_width = spec.n_heads * spec.key_dim, spec.n_heads * spec.value_dim
        self.gate_width = 0 if spec.gate_activation is None else self.v_width
        plain = dict(weight_suffix="", bias_suffix=".b")
        second = "f" if self.forget else "k"
        pieces = [(f"{prefix}.q", self.k_width), (f"{prefix}.{second}", self.k_width), (f"{prefix}.v", self.v_width)]
        if self.gate_width:
            pieces.append((f"{prefix}.g", self.v_width))
        self.inputs = StackedLinear(pieces, spec.hidden, self.forget, dtype, device, biased=[f"{prefix}.f"] if self.forget else None, **plain)
        self.gates = None
        if self.exponential:
            self.gates = StackedLinear([(f"{prefix}.i", spec.n_heads), (f"{prefix}.f", spec.n_heads)], spec.hidden, True, dtype, device, **plain)
        self.out = StackedLinear([(f"{prefix}.o", spec.hidden)], self.v_width, False, dtype, device, **plain)
        self._linears = tuple(part for part in (self.inputs, self.gates, self.out) if part is not None)
        self.position = None if spec.position is None else build("position", spec.position, device=device)
        self._own = {}
        if spec.norm_weight is not None:
            self._own[f"{prefix}.norm"] = TensorSpec((self.v_width if spec.norm_weight == "full" else spec.value_dim,), role="vector", init="ones")
        if self.forget:
            self._own[f"{prefix}.lower"] = TensorSpec((self.k_width,), role="vector", std=0.1)
        self._held = {}
        self.norm_weight = self.decays = self.lower = None

    def state_floats(self) -> int:
        spec = self.spec
        per_head = (spec.value_dim + 1) * spec.key_dim + 1 if self.exponential else spec.value_dim * spec.key_dim
        return spec.n_heads * per_head

    def cache_need(self):
        return CacheNeed("state", state_shape=(self.state_floats(),), state_dtype=torch.float32)

    def tensor_specs(self):
        specs = dict(self._own)
        for part in self._linears:
            specs.update(part.tensor_specs())
        return specs

    def assign(self, name, tensor):
        if name in self._own:
            self._held[name] = tensor
            return
        for part in self._linears:
            if name in part.tensor_specs():
                return part.assign(name, tensor)
        raise KeyError(name)

    def finalize_weights(self):
        spec, prefix = self.spec, self.prefix
        for part in self._linears:
            part.finalize_weights()
        if spec.norm_weight is not None:
            weight = self._held.pop(f"{prefix}.norm")
            self.norm_weight = weight.repeat(spec.n_heads).contiguous() if spec.norm_weight == "head" else weight
        if self.forget:
            self.lower = self._held.pop(f"{prefix}.lower")
        if self.position is not None:
            self.position.finalize_weights()
        if spec.gating == "decay":
            self.decays = torch.tensor(spec.decays, dtype=torch.float64).to(torch.float32).to(self.device)

    def _walk(self, projected, step, cache, read):
        spec, width = self.spec, self.k_width
        queries, keys, values = projected[:, :width], projected[:, width : 2 * width], projected[:, 2 * width : 2 * width + self.v_width]
        if self.forget:
            kernels.forget_gates(projected, 0, width, self.lower)
            kernels.wkv(queries, None, values, keys, None, cache.state, step.cu_seqlens, step.seq_slot, read, spec.n_heads, spec.key_dim, spec.value_dim, form="forget_writes")
            return
        if self.position is not None or spec.key_scale != 1.0:
            rotary = 0 if spec.position is None else spec.position.rotary_dim
            kernels.turn_heads(projected, step.positions, None if self.position is None else self.position.frequency, rotary, 2 * spec.n_heads, spec.key_dim, spec.n_heads,
                               spec.key_scale)
        kernels.wkv(queries, keys, values, None, self.decays, cache.state, step.cu_seqlens, step.seq_slot, read, spec.n_heads, spec.key_dim, spec.value_dim,
                    form="constant_decay")

    def forward(self, hidden, step, cache, writes_cache: bool):
        spec = self.spec
        tokens = hidden.shape[0]
        projected = self.inputs.forward(hidden, out_dtype=torch.float32 if self.walked else None)
        gates = self.gates.forward(hidden, out_dtype=torch.float32) if self.exponential else None
        read = torch.empty((tokens, self.v_width), dtype=torch.float32, device=hidden.device)
        k_end, v_end = 2 * self.k_width, 2 * self.k_width + self.v_width
        if self.walked:
            self._walk(projected, step, cache, read)
        else:
            kernels.linear_recurrence(projected[:, : self.k_width], projected[:, self.k_width : k_end], projected[:, k_end:v_end], gates, self.decays,
                                      cache.state, step.cu_seqlens, step.seq_slot, read, spec.n_heads, spec.key_dim, spec.value_dim,
                                      self.exponential, spec.gate_cap, spec.query_scale, spec.activation == "silu")
        gated = torch.empty((tokens, self.v_width), dtype=hidden.dtype, device=hidden.device)
        kernels.gated_group_norm(read, self.norm_weight, projected[:, v_end:] if self.gate_width else None, gated,
                                 spec.n_heads if spec.norm_groups == "head" else 1, spec.eps, True, silu_gate=spec.gate_activation == "silu")
        return self.out.forward(gated, out_dtype=torch.float32 if self.walked else None)
