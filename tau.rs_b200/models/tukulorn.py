"""Tukulorn as a list of blocks: the only place that knows this architecture.

Every layer is a pre-norm block on a 32-bit residual stream (`parts.block.StreamPreNormBlock`) whose norms are RMS norms with weights
stored around zero and whose results are scaled per channel before they join the stream.  The mixer is one of two: differential
attention with biases and a query temperature, no rotation (`parts.differential_attention` with those options), or latent attention
with a sliding window, queries straight from the layer's input and a gate per head (`parts.latent_attention`).  The feed-forward is
gated (SwiGLU), or routed experts with a clamped gate whose router chooses among groups of experts, or absent.  A run of layers may
repeat with the same weights; each pass keeps caches of its own, and the embedding output joins the stream before every pass but the
first.  Tensor names: `embed`, `l<i>.norm1`, `l<i>.mix.*`, `l<i>.ls1`, `l<i>.norm2`, `l<i>.mlp.*`, `l<i>.ls2`, `final.norm`, `head`.
"""
from __future__ import annotations

from ..config.registry import register_architecture
from ..config.specs import (BlockSpec, DifferentialAttentionSpec, LatentAttentionSpec, ModelSpec, NormSpec, PairRotationSpec, RoutedExpertsSpec,
                            ScheduleEntry, SwiGLUSpec)
from ..config.tukulorn import ARCHITECTURE, MODEL_TYPE, TukulornConfig

# The design keeps no table over positions; the limit is that of a 32-bit position.
MAX_POSITIONS = (1 << 31) - 1


def _mixer_spec(mixer, width: int, eps: float):
    if mixer.type == "attention":
        return DifferentialAttentionSpec(hidden=width, n_heads=mixer.heads, n_kv_heads=mixer.kv_heads, dim=mixer.dim, value_dim=mixer.vdim,
                                         softmax_scale=mixer.scale, diff=mixer.diff, eps=eps, gate=False, qk_norm=False, bias=True,
                                         temperature=mixer.temperature)
    position = PairRotationSpec(rotary_dim=mixer.rot_dims, theta=mixer.rot_base) if mixer.rot_dims else None
    return LatentAttentionSpec(hidden=width, n_heads=mixer.heads, head_dim=mixer.dim, rot_dim=mixer.rot_dim, value_dim=mixer.vdim, q_rank=None,
                               kv_rank=mixer.kv_rank, softmax_scale=mixer.scale, eps=eps, position=position, sink=False, gate=True, gate_per_head=True,
                               window=mixer.window, wide_result=True)


def _feed_forward_spec(mlp, width: int):
    if mlp is None:
        return None
    if mlp.kind == "dense":
        return SwiGLUSpec(hidden=width, intermediate=mlp.ff, gate_name="gate", up_name="up", down_name="down", weight_suffix="", wide_result=True)
    return RoutedExpertsSpec(hidden=width, intermediate=mlp.expert_ff, experts=mlp.experts, top=mlp.top, score="sigmoid", correction=False, renormalize=True,
                             groups=mlp.groups, keep_groups=mlp.keep, scale=mlp.scale, activation="clamped", limit=mlp.limit)


def build_tukulorn_spec(config: TukulornConfig) -> ModelSpec:
    norm = NormSpec(width=config.width, eps=config.eps, weight_offset=1.0)
    blocks = tuple(
        BlockSpec(prefix=f"l{index}", mixer=_mixer_spec(layer.mixer, config.width, config.eps), feed_forward=_feed_forward_spec(layer.mlp, config.width),
                  mixer_norm=norm, feed_forward_norm=norm if layer.mlp is not None else None, kind="pre_norm_stream", layer_scale=True)
        for index, layer in enumerate(config.layers)
    )
    # Runs whose mixers keep the same thing share a cache group; each run has a cache layer of its own there.
    schedule, kinds, layers_of = [], [], {}
    for index, opens_pass in config.layer_runs():
        mixer = blocks[index].mixer
        if mixer not in kinds:
            kinds.append(mixer)
        group = f"{mixer.kind}.{kinds.index(mixer)}"
        schedule.append(ScheduleEntry(layer=index, cache_group=group, cache_layer=layers_of.get(group, 0), joins_embedding=opens_pass))
        layers_of[group] = layers_of.get(group, 0) + 1
    return ModelSpec(
        architecture=ARCHITECTURE, vocab_size=config.vocab, hidden=config.width, max_positions=MAX_POSITIONS, embedding_name="embed",
        blocks=blocks, schedule=tuple(schedule), final_norm=norm, final_norm_name="final.norm", head_name="head", tie_head=False,
        declared_dtype=config.declared_dtype, residual_dtype="float32",
    )


register_architecture(ARCHITECTURE, MODEL_TYPE, TukulornConfig.from_json, build_tukulorn_spec, storage_dtype="bfloat16")
