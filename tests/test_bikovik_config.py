"""Bikovik on the host: its configuration, the blocks and schedule built from it, what its cache keeps and gives back, and the plain
statement against itself and against closed forms."""
import copy
import math

import pytest
import torch

import bikovik_models as bm
import plain_bikovik as plain
from tau_rs_b200.cache.sequence_cache import PAGE_TOKENS, SequenceCache
from tau_rs_b200.config import BikovikConfig, InvalidConfig
from tau_rs_b200.config.metadata import metadata_from_json
from tau_rs_b200.config.registry import architecture_for, spec_from_config_json
from tau_rs_b200.parts import DecoderModel
from tau_rs_b200.parts.base import CacheNeed

ALL = (bm.MIXED, bm.ODD, bm.PEAKY, bm.HEADY, bm.WIDE, bm.LONG_MEMORY, *bm.ONLY.values())


def test_the_architecture_is_registered_and_stores_bfloat16():
    metadata = metadata_from_json(bm.MIXED)
    assert (metadata.architecture, metadata.model_type, metadata.declared_dtype) == ("Bikovik", "bikovik", None)
    assert architecture_for(bm.MIXED).storage_dtype == "bfloat16"


def test_every_size_and_constant_is_read_from_the_configuration():
    config = BikovikConfig.from_json(bm.MIXED)
    assert (config.vocab, config.width, config.eps, config.embedding_scale, config.logit_softcap) == (211, 96, 1e-5, 1.7, 4.0)
    mixer = config.layers[4].mixer
    assert (mixer.heads, mixer.kv_heads, mixer.dim, mixer.vdim, mixer.scale, mixer.window, mixer.keep_first, mixer.rot_base, mixer.rot_dims, mixer.v_mix) == (
        6, 3, 8, 16, 8 ** -0.5, 65, 64, 5000.0, 8, True)
    assert (config.layers[1].mixer.heads, config.layers[1].mixer.dim, config.layers[1].mixer.vdim) == (3, 16, 24)
    mixer = config.layers[5].mixer
    assert (mixer.heads, mixer.dim, mixer.vdim, mixer.rot_base, mixer.rot_dims) == (2, 24, 8, 3000.0, 24) and mixer.decays == tuple(bm.MIXED["layers"][5]["mixer"]["decay"])
    assert (config.layers[4].mlp.ff, config.layers[4].mlp.limit) == (40, 0.7) and config.layers[5].mlp is None and not config.layers[0].mixer.v_mix


@pytest.mark.parametrize("change, message", [
    (lambda c: c["layers"][0].update(type="wkv"), "type must be one of"),
    (lambda c: c["layers"][0]["mixer"].update(kv_heads=3), "multiple of kv_heads"),
    (lambda c: c["layers"][0]["mixer"]["rot"].update(dims=18), "rot.dims"),
    (lambda c: c["layers"][0]["mixer"].pop("mask"), "'mask'"),
    (lambda c: c["layers"][0]["mixer"]["mask"].update(size=0), "'size'"),
    (lambda c: c["layers"][0]["mixer"]["mask"].update(keep_first=-1), "'keep_first'"),
    (lambda c: c["layers"][0]["mixer"].update(v_mix=1), "v_mix"),
    (lambda c: c["layers"][2]["mixer"].update(vdim=8), "first layer with v_mix"),
    (lambda c: c["layers"][1]["mixer"].update(dim=0), "'dim'"),
    (lambda c: c["layers"][3]["mixer"].update(decay=[0.5]), "decay"),
    (lambda c: c["layers"][3]["mixer"].update(decay=[0.5, 0.5, 1.5]), "decay"),
    (lambda c: c["layers"][0]["mlp"].pop("limit"), "'limit'"),
    (lambda c: c["layers"][0]["mlp"].update(kind="moe"), "kind 'dense'"),
    (lambda c: c.pop("embedding"), "'embedding'"),
    (lambda c: c.update(logit_softcap=0), "'logit_softcap'"),
    (lambda c: c.pop("norm"), "'norm'"),
])
def test_a_configuration_that_does_not_fit_is_refused_by_name(change, message):
    raw = copy.deepcopy(bm.MIXED)
    change(raw)
    with pytest.raises(InvalidConfig, match=message):
        BikovikConfig.from_json(raw)


def test_blocks_schedule_and_cache_groups():
    spec = spec_from_config_json(bm.MIXED)
    assert spec.residual_dtype == "float32" and not spec.tie_head and spec.embedding_scale == 1.7 and spec.logit_cap == 4.0
    assert all(block.kind == "pre_norm_stream" and block.mixer_norm.kind == "dynamic_tanh" for block in spec.blocks) and spec.final_norm.kind == "dynamic_tanh"
    assert [block.mixer.kind for block in spec.blocks] == ["masked_attention", "linear_recurrence", "masked_attention", "linear_recurrence", "masked_attention", "linear_recurrence",
                                                           "masked_attention", "linear_recurrence", "masked_attention"]
    assert [getattr(block.mixer, "value_mix", None) for block in spec.blocks] == [None, None, "first", None, "mix", None, None, None, "mix"]
    first = spec.blocks[0].mixer
    assert first.talk and first.bias and (first.window, first.keep_first) == (70, 9) and first.weights == "softmax" and not first.sink and first.gate is None
    forget, retention = spec.blocks[1].mixer, spec.blocks[3].mixer
    assert forget.gating == "forget" and forget.norm_weight == "head" and forget.gate_activation is None and forget.norm_groups == "head" and forget.position is None
    assert retention.gating == "decay" and retention.norm_weight is None and retention.gate_activation == "silu" and retention.key_scale == 0.25 and retention.activation is None
    assert (retention.position.rotary_dim, retention.position.theta) == (8, 3000.0)
    assert spec.blocks[4].feed_forward.activation == "clamped" and spec.blocks[4].feed_forward.limit == 0.7
    assert spec.blocks[5].feed_forward is None and spec.blocks[5].feed_forward_norm is None
    places = [(entry.cache_group, entry.cache_layer) for entry in spec.schedule]
    assert len(set(places)) == len(places)
    groups = DecoderModel(spec, torch.float32, "cpu").cache_groups()
    rows = sorted((need.row_width, need.window, need.keep_first, layers) for need, layers in groups.values() if need.kind == "rows")
    assert rows == sorted([(80, 70, 9, 1), (80, 40, 5, 1), (72, 65, 64, 1), (72, 17, 70, 1), (56, 130, 1, 1)])
    # The two kinds of memory with equal sizes share a group of states.
    assert sorted((need.state_shape, layers) for need, layers in groups.values() if need.kind == "state") == [((384,), 2), ((1152,), 2)]


def test_keys_and_values_as_wide_as_ordinary_heads_lie_in_pages_of_heads():
    groups = DecoderModel(spec_from_config_json(bm.HEADY), torch.float32, "cpu").cache_groups()
    assert not [need for need, _ in groups.values() if need.kind == "rows"]
    assert sorted((need.n_kv_heads, need.head_dim, need.window, need.keep_first) for need, _ in groups.values() if need.kind == "kv") == [(1, 128, 64, 1), (2, 64, 90, 20), (3, 128, 200, 130)]


def test_the_model_asks_for_exactly_the_tensors_of_the_design():
    for cfg in ALL:
        wanted = DecoderModel.tensor_specs_of(spec_from_config_json(cfg))
        made = bm.weights(cfg, 1)
        assert set(wanted) == set(made)
        for name, value in made.items():
            assert tuple(wanted[name].shape) == tuple(value.shape), name


@pytest.mark.parametrize("window, keep_first", [(70, 0), (70, 1), (70, 64), (70, 65), (64, 200), (1, 3), (300, 100)])
def test_a_windowed_cache_keeps_the_first_pages_and_gives_back_those_between(window, keep_first):
    """Two sequences in turn through a cache of few pages: whatever a query may see lies in a page that the sequence holds and its table
    names; pages between the kept ones and the window go back; nothing is lost or shared."""
    pages = -(-keep_first // PAGE_TOKENS) + window // PAGE_TOKENS + 3
    cache = SequenceCache({"keys": (CacheNeed("rows", row_width=4, window=window, keep_first=keep_first), 2)}, 2 * pages * PAGE_TOKENS, 1 << 20, torch.float32, "cpu")
    group = cache.kv["keys"]
    slots = [cache.open(), cache.open()]
    lengths = [0, 0]
    most = 0
    for step in range(400):
        which = step % 2
        count = [1, 7, 30, 2, 1, 25][step % 6] if step < 60 else 3
        slot, length = slots[which], lengths[which]
        cache.reserve(slot, length + count)
        table = cache.page_rows("keys", [slot], -(-(length + count) // PAGE_TOKENS))[0]
        held = set(group.held[slot])
        for position in range(length, length + count):
            for key in [*range(min(keep_first, position + 1)), *range(max(0, position - window + 1), position + 1)]:
                assert int(table[key // PAGE_TOKENS]) in held
        lengths[which] = length + count
        cache.advance(slot, lengths[which])
        cache.check()
        most = max(most, len(group.held[slot]))
    assert most <= pages and group.tokens_read(1000) == min(1000, window + keep_first)
    for slot in slots:
        cache.close(slot)
    cache.check()
    assert group.pool.in_use == 0


def _double(values):
    return {name: value.double() for name, value in values.items()}


def test_the_plain_statement_is_causal():
    for cfg in (bm.MIXED, bm.ODD):
        values = _double(bm.weights(cfg, 3))
        tokens = torch.randint(0, cfg["vocab"], (70,), generator=torch.Generator().manual_seed(5)).tolist()
        whole = plain.forward(tokens, values, cfg)
        assert torch.allclose(plain.forward(tokens[:41], values, cfg), whole[:41], atol=1e-9)


def test_the_plain_mechanisms_against_closed_forms():
    generator = torch.Generator().manual_seed(9)
    rand = lambda *shape: torch.randn(*shape, dtype=torch.float64, generator=generator)
    ones = lambda *shape: torch.ones(*shape, dtype=torch.float64)
    # The mask: by hand for one query; a window of one sees itself and the kept positions.
    seen = plain.visible_keys(12, 4, 3)
    assert seen[9].nonzero().flatten().tolist() == [0, 1, 2, 6, 7, 8, 9] and seen[2].nonzero().flatten().tolist() == [0, 1, 2]
    assert plain.visible_keys(5, 1, 0).equal(torch.eye(5, dtype=torch.bool))
    # Mixing by the identity is ordinary grouped attention; a row of zeros gives even weights; a permutation swaps the heads' weights.
    q, k, v = rand(9, 2, 4), rand(9, 1, 4), rand(9, 1, 3)
    visible = plain.visible_keys(9, 100, 0)
    out = plain.talking_attention(q, k, v, 0.5, torch.eye(2, dtype=torch.float64), visible)
    scores = (q[:, 0] @ k[:, 0].T) * 0.5 + torch.triu(torch.full((9, 9), -math.inf, dtype=torch.float64), 1)
    assert torch.allclose(out[:, 0], torch.softmax(scores, -1) @ v[:, 0], atol=1e-12)
    even = plain.talking_attention(q, k, v, 0.5, torch.zeros(2, 2, dtype=torch.float64), visible)
    assert torch.allclose(even[5, 1], v[:6, 0].mean(0), atol=1e-12)
    swapped = plain.talking_attention(q, k, v, 0.5, torch.tensor([[0.0, 1.0], [1.0, 0.0]], dtype=torch.float64), visible)
    assert torch.allclose(swapped[:, 0], out[:, 1], atol=1e-12) and torch.allclose(swapped[:, 1], out[:, 0], atol=1e-12)
    # A rotation keeps lengths and makes scores depend on the distance alone.
    turned = plain.rotate_halves(rand(1, 1, 6).repeat(8, 1, 1), {"dims": 4, "base": 100.0})
    assert torch.allclose((turned[3] * turned[1]).sum(), (turned[6] * turned[4]).sum(), atol=1e-12) and torch.allclose(turned[:, :, 4:], turned[:1, :, 4:].repeat(8, 1, 1))
    # The forget gate: at one nothing is written, at zero the state is the token's own; a constant f is a decay with keys 1 - f.
    queries, values = rand(6, 2, 4), rand(6, 2, 3)
    assert plain.forget_write_recurrence(queries, ones(6, 2, 4), values).abs().max() == 0.0
    own = plain.forget_write_recurrence(queries, torch.zeros(6, 2, 4, dtype=torch.float64), values)
    assert torch.allclose(own, queries.sum(-1, keepdim=True) * values, atol=1e-12)
    constant = plain.forget_write_recurrence(queries, 0.8 * ones(6, 2, 4), values)
    assert torch.allclose(constant, plain.decay_recurrence(queries, 0.2 * ones(6, 2, 4), values, 0.8 * ones(2)), atol=1e-12)
    assert torch.allclose(plain.forget_gate(torch.tensor([-100.0, 100.0], dtype=torch.float64), torch.tensor([0.3, 0.3], dtype=torch.float64)), torch.tensor([0.3, 1.0], dtype=torch.float64))
    # Decays: sum over the earlier tokens by hand.
    keys, decay = rand(6, 2, 4), torch.tensor([0.5, 1.0], dtype=torch.float64)
    read = plain.decay_recurrence(queries, keys, values, decay)
    by_hand = sum(decay[0] ** (4 - j) * (queries[4, 0] * keys[j, 0]).sum() * values[j, 0] for j in range(5))
    assert torch.allclose(read[4, 0], by_hand, atol=1e-12)
    # The clamped gate and the soft cap.
    gate, up = torch.tensor([5.0, -5.0, 0.5], dtype=torch.float64), torch.tensor([9.0, -9.0, 0.25], dtype=torch.float64)
    expected = torch.tensor([2.0 / (1.0 + math.exp(-3.404)) * 3.0, -5.0 / (1.0 + math.exp(8.51)) * -1.0, 0.5 / (1.0 + math.exp(-0.851)) * 1.25], dtype=torch.float64)
    assert torch.allclose(plain.clamped_activation(gate, up, 2.0), expected, atol=1e-12)
    assert torch.allclose(plain.soft_cap(torch.tensor([0.01, 1e6, -1e6], dtype=torch.float64), 3.0), torch.tensor([0.01, 3.0, -3.0], dtype=torch.float64), atol=1e-6)
    assert torch.allclose(plain.dynamic_tanh(torch.tensor([0.0, 1e9], dtype=torch.float64), 0.5, 2.0, 0.25), torch.tensor([0.25, 2.25], dtype=torch.float64))
    assert torch.allclose(plain.mixed_values(values, queries[..., :3], 0.25), 0.75 * values + 0.25 * queries[..., :3]) and plain.mixed_values(values, None, 0.25) is values
