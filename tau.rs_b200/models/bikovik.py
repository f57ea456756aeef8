"""Bikovik as a list of blocks: the only place that knows this architecture.

Every layer is a pre-norm block on a 32-bit residual stream (`parts.block.StreamPreNormBlock`) whose norms are an element-wise tanh
(`parts.norm.DynamicTanh`).  The mixer is one of three: softmax attention with biases, a rotation of halves, scores mixed over the heads,
a sliding window beside the sequence's first positions, and values mixed with those of the first such layer
(`parts.masked_attention` with those options); a matrix memory whose forget gate decides what is written (HGRN2); or one with a
constant decay per head behind rotated queries and keys (retention), both `parts.linear_recurrence`.  The feed-forward is a gated one
with clamped gate and up values, or absent.  The embedded rows are scaled, and the logits pass a soft cap.  Tensor names: `embed`,
`l<i>.norm1`, `l<i>.mix.*`, `l<i>.norm2`, `l<i>.mlp.*`, `final.norm`, `head`; a norm's `b` and `alpha` lie under its name.
"""
from __future__ import annotations

from ..config.bikovik import ARCHITECTURE, MODEL_TYPE, BikovikConfig
from ..config.registry import register_architecture
from ..config.specs import BlockSpec, LinearRecurrenceSpec, MaskedAttentionSpec, ModelSpec, NormSpec, ScaledRotationSpec, ScheduleEntry, SwiGLUSpec

# The design keeps no table over positions; the limit is that of a 32-bit position.
MAX_POSITIONS = (1 << 31) - 1


def _rotation(mixer):
    return ScaledRotationSpec(rotary_dim=mixer.rot_dims, theta=mixer.rot_base) if mixer.rot_dims else None


def _mixer_spec(mixer, width: int, eps: float, value_mix):
    if mixer.type == "attention":
        return MaskedAttentionSpec(hidden=width, n_heads=mixer.heads, n_kv_heads=mixer.kv_heads, dim=mixer.dim, value_dim=mixer.vdim, softmax_scale=mixer.scale,
                                   eps=eps, position=_rotation(mixer), window=mixer.window, bias=True, keep_first=mixer.keep_first, talk=True, value_mix=value_mix)
    if mixer.type == "hgrn2":
        return LinearRecurrenceSpec(hidden=width, n_heads=mixer.heads, key_dim=mixer.dim, value_dim=mixer.vdim, gating="forget", eps=eps, norm_groups="head",
                                    norm_weight="head", gate_activation=None)
    return LinearRecurrenceSpec(hidden=width, n_heads=mixer.heads, key_dim=mixer.dim, value_dim=mixer.vdim, gating="decay", eps=eps, norm_groups="head",
                                decays=mixer.decays, position=_rotation(mixer), key_scale=mixer.dim ** -0.5, norm_weight=None, gate_activation="silu")


def _feed_forward_spec(mlp, width: int):
    if mlp is None:
        return None
    return SwiGLUSpec(hidden=width, intermediate=mlp.ff, gate_name="gate", up_name="up", down_name="down", weight_suffix="", activation="clamped", limit=mlp.limit,
                      wide_result=True)


def build_bikovik_spec(config: BikovikConfig) -> ModelSpec:
    norm = NormSpec(width=config.width, eps=config.eps, kind="dynamic_tanh", bias_suffix=".b")
    blocks, schedule, counters, names = [], [], {}, {}
    mixing = False      # a layer whose values the later ones mix in has been seen
    for index, layer in enumerate(config.layers):
        value_mix = None
        if layer.mixer.type == "attention" and layer.mixer.v_mix:
            value_mix, mixing = ("mix" if mixing else "first"), True
        mixer = _mixer_spec(layer.mixer, config.width, config.eps, value_mix)
        blocks.append(BlockSpec(prefix=f"l{index}", mixer=mixer, feed_forward=_feed_forward_spec(layer.mlp, config.width), mixer_norm=norm,
                                feed_forward_norm=norm if layer.mlp is not None else None, kind="pre_norm_stream"))
        # Layers whose mixers keep the same thing share a cache group with a cache layer each.
        if mixer.kind == "masked_attention":
            need, label = ("keys", mixer.n_kv_heads, mixer.dim, mixer.value_dim, mixer.window, mixer.keep_first), "keys"
        else:
            need, label = ("memory", mixer.n_heads, mixer.key_dim, mixer.value_dim), "memory"
        group = names.setdefault(need, f"{label}.{len(names)}")
        counters[group] = counters.get(group, -1) + 1
        schedule.append(ScheduleEntry(layer=index, cache_group=group, cache_layer=counters[group]))
    return ModelSpec(
        architecture=ARCHITECTURE, vocab_size=config.vocab, hidden=config.width, max_positions=MAX_POSITIONS, embedding_name="embed",
        blocks=tuple(blocks), schedule=tuple(schedule), final_norm=norm, final_norm_name="final.norm", head_name="head", tie_head=False,
        declared_dtype=config.declared_dtype, residual_dtype="float32", embedding_scale=config.embedding_scale, logit_cap=config.logit_softcap,
    )


register_architecture(ARCHITECTURE, MODEL_TYPE, BikovikConfig.from_json, build_bikovik_spec, storage_dtype="bfloat16")
