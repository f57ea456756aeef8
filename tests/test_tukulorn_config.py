"""Tukulorn on the host: its configuration, the blocks and schedule built from it, what its cache keeps, and the plain statement
against closed forms and against itself with single mistakes planted in it (each must move the logits well beyond the tolerances)."""
import copy
import math

import pytest
import torch

import plain_tukulorn as plain
import tukulorn_models as tm
from tau_rs_b200.cache import SequenceCache
from tau_rs_b200.config import InvalidConfig, TukulornConfig
from tau_rs_b200.config.metadata import metadata_from_json
from tau_rs_b200.config.registry import architecture_for, spec_from_config_json
from tau_rs_b200.parts import DecoderModel
from tau_rs_b200.parts.base import Pending

MODELS = {"mixed": tm.MIXED, "odd": tm.ODD, "wide": tm.WIDE, "peaky": tm.PEAKY, "edgy": tm.EDGY}


def test_the_architecture_is_registered_and_stores_bfloat16():
    metadata = metadata_from_json(tm.MIXED)
    assert (metadata.architecture, metadata.model_type, metadata.declared_dtype) == ("Tukulorn", "tukulorn", None)
    assert architecture_for(tm.MIXED).storage_dtype == "bfloat16"


def test_every_size_and_constant_is_read_from_the_configuration():
    config = TukulornConfig.from_json(tm.MIXED)
    assert (config.vocab, config.width, config.eps, config.loop_start, config.loop_stop, config.loop_times) == (211, 96, 1e-5, 1, 4, 3)
    first, second, fourth = (config.layers[index] for index in (0, 1, 3))
    assert (first.mixer.heads, first.mixer.dim, first.mixer.rot_dim, first.mixer.vdim, first.mixer.kv_rank, first.mixer.window) == (3, 24, 8, 20, 40, 37)
    assert (first.mixer.rot_dims, first.mixer.rot_base, first.mixer.scale) == (8, 5000.0, 32 ** -0.5)
    assert (first.mlp.experts, first.mlp.top, first.mlp.groups, first.mlp.keep, first.mlp.scale, first.mlp.expert_ff, first.mlp.limit) == (12, 3, 4, 2, 1.7, 40, 0.8)
    assert (second.mixer.heads, second.mixer.kv_heads, second.mixer.dim, second.mixer.vdim, second.mixer.diff) == (4, 2, 16, 24, 0.3)
    assert second.mixer.temperature == (0.4, 30) and fourth.mixer.temperature == (-0.2, 7) and fourth.mlp is None
    assert config.layers[2].mlp.kind == "dense" and config.layers[2].mlp.ff == 80
    bare = copy.deepcopy(tm.MIXED)
    del bare["loop"], bare["layers"][1]["mixer"]["q_temp"], bare["layers"][0]["mlp"]["router"]["groups"], bare["layers"][0]["mixer"]["mask"]
    config = TukulornConfig.from_json(bare)
    assert config.layer_runs() == tuple((index, False) for index in range(5)) and config.layers[1].mixer.temperature is None
    assert (config.layers[0].mlp.groups, config.layers[0].mlp.keep, config.layers[0].mixer.window) == (1, 1, None)


def test_blocks_schedule_and_cache_groups():
    spec = spec_from_config_json(tm.MIXED)
    assert spec.residual_dtype == "float32" and not spec.tie_head and spec.final_norm.weight_offset == 1.0
    assert all(block.kind == "pre_norm_stream" and block.layer_scale and block.mixer_norm.weight_offset == 1.0 for block in spec.blocks)
    assert [(entry.layer, entry.joins_embedding) for entry in spec.schedule] == [
        (0, False), (1, False), (2, False), (3, False), (1, True), (2, False), (3, False), (1, True), (2, False), (3, False), (4, False)]
    seen = {(entry.cache_group, entry.cache_layer) for entry in spec.schedule}
    assert len(seen) == len(spec.schedule)                    # every pass of the loop has a cache of its own
    groups = DecoderModel(spec, torch.float32, "cpu").cache_groups()
    rows = sorted((need.row_width, need.window or 0, layers) for need, layers in groups.values() if need.kind == "rows")
    assert rows == sorted([(40 + 8, 37, 1), (64 + 16, 100, 3), (22 + 6, 64, 1), (2 * (2 * 16 + 24), 0, 3)])
    # Where the wider of a key and a value is a multiple of 16, every map is an ordinary head of that width.
    assert [(need.n_kv_heads, need.head_dim, need.window, layers) for need, layers in groups.values() if need.kind == "kv"] == [(6, 48, None, 3)]


@pytest.mark.parametrize("name", sorted(MODELS))
def test_the_model_asks_for_exactly_the_tensors_of_the_design(name):
    wanted = DecoderModel.tensor_specs_of(spec_from_config_json(MODELS[name]))
    made = tm.weights(MODELS[name], 0)
    assert set(wanted) == set(made)
    for tensor, spec in wanted.items():
        assert tuple(spec.shape) == tuple(made[tensor].shape), tensor


@pytest.mark.parametrize("change, message", [
    (lambda c: c["layers"][0].update(type="mamba"), "type must be one of"),
    (lambda c: c["layers"][0]["mixer"]["rot"].update(dims=7), "rot.dims"),
    (lambda c: c["layers"][0]["mixer"]["rot"].update(dims=10), "rot.dims"),
    (lambda c: c["layers"][0]["mixer"].pop("kv_rank"), "'kv_rank'"),
    (lambda c: c["layers"][0]["mixer"]["mask"].update(size=0), "'size'"),
    (lambda c: c["layers"][1]["mixer"].update(kv_heads=3), "multiple of kv_heads"),
    (lambda c: c["layers"][1]["mixer"].pop("diff"), "'diff'"),
    (lambda c: c["layers"][1]["mixer"]["q_temp"].update(every=0), "'every'"),
    (lambda c: c["layers"][0]["mlp"]["router"]["groups"].update(count=5), "equal groups"),
    (lambda c: c["layers"][0]["mlp"]["router"]["groups"].update(keep=5), "keep at most all"),
    (lambda c: c["layers"][0]["mlp"]["router"].update(top=7), "exceeds"),
    (lambda c: c["layers"][0]["mlp"]["expert"].pop("limit"), "'limit'"),
    (lambda c: c["layers"][2]["mlp"].update(kind="glu"), "kind"),
    (lambda c: c["loop"].update(stop=6), "loop must satisfy"),
    (lambda c: c.update(width=-3), "'width'"),
])
def test_a_bad_configuration_is_refused_by_name(change, message):
    raw = copy.deepcopy(tm.MIXED)
    change(raw)
    with pytest.raises(InvalidConfig, match=message):
        TukulornConfig.from_json(raw)


def test_a_window_cache_holds_a_few_pages_however_long_the_sequence():
    model = DecoderModel(spec_from_config_json(tm.EDGY), torch.float32, "cpu")
    cache = SequenceCache(model.cache_groups(), 64 * 6, 1 << 20, torch.float32, "cpu")
    slot = cache.open()
    for length in range(1, 900, 7):
        cache.reserve(slot, length)
        cache.advance(slot, length)
        cache.check()
        assert all(len(group.held[slot]) <= 3 for group in cache.kv.values())
    cache.close(slot)
    cache.check()


def test_what_is_pending_keeps_its_factors_when_rows_of_a_table_join():
    result, factors, rows = torch.ones(2, 3), torch.arange(3.0), ("table", "numbers", 1.0)
    pending = Pending.with_rows(Pending((result,), 0.5, factors), rows)
    assert len(pending) == 1 and pending[0] is result and pending.scale == 0.5 and pending.channel_scale is factors and pending.rows is rows
    assert tuple(Pending.with_rows(None, rows)) == () and Pending.with_rows(result, rows)[0] is result
    with pytest.raises(ValueError, match="already"):
        Pending.with_rows(pending, rows)


def test_a_loop_on_a_stream_of_the_run_dtype_is_refused():
    import dataclasses

    spec = dataclasses.replace(spec_from_config_json(tm.MIXED), residual_dtype=None)
    with pytest.raises(ValueError, match="joins again"):
        DecoderModel(spec, torch.bfloat16, "cpu")


# ---- the plain statement ----------------------------------------------------------------------------------------------
def test_the_plain_mechanisms_against_closed_forms():
    torch.manual_seed(0)
    # The window: by hand; the temperature: one up to position every - 2, then steps.
    seen = plain.visible(9, 3)
    assert seen[7].nonzero().flatten().tolist() == [5, 6, 7] and seen[0].nonzero().flatten().tolist() == [0]
    factors = plain.query_temperature(10, 0.5, 4)
    assert factors[:3].tolist() == [1.0] * 3 and math.isclose(factors[3], 1 + 0.5 * math.log(2)) and math.isclose(factors[7], 1 + 0.5 * math.log(3))
    # A rotation keeps lengths, leaves position 0 and turns by the difference of positions.
    x = torch.randn(1, 8, dtype=plain.F).expand(6, 8)
    turned = plain.rotate_pairs(x, 8, 50.0)
    assert torch.allclose(turned[0], x[0]) and torch.allclose(turned.norm(dim=-1), x.norm(dim=-1))
    assert torch.allclose((turned[5] * turned[3]).sum(), (turned[2] * turned[0]).sum())
    # Groups: the best pair, not the best expert, ranks a group; the choice among the kept ones is by score.
    scores = [0.9, 0.1, 0.6, 0.5, 0.2, 0.3, 0.55, 0.54]
    assert plain.choose_experts(scores, 2, 4, 1) == [2, 3]
    assert plain.choose_experts(scores, 3, 4, 2) == [2, 6, 7]
    assert plain.choose_experts(scores, 3, 4, 3) == [0, 2, 6] and plain.choose_experts(scores, 2, 8, 2) == [0, 2]
    assert plain.choose_experts([0.5, 0.5, 0.5, 0.5], 2, 2, 1) == [0, 1]              # the lowest number among equals
    # Both maps equal and lambda one: nothing is left but eps.
    a = torch.randn(4, 6, dtype=plain.F)
    assert torch.allclose(plain.map_difference(a, a, 1.0, 0.2, 1e-3), torch.zeros(4, 6, dtype=plain.F))
    assert torch.allclose(plain.map_difference(a, a, 0.0, 0.2, 0.0), 0.8 * a / a.pow(2).mean(-1, keepdim=True).sqrt())


@pytest.mark.parametrize("name", ["mixed", "odd"])
def test_the_plain_statement_is_causal(name):
    cfg = MODELS[name]
    values = {key: value.double() for key, value in tm.weights(cfg, 3).items()}
    tokens = torch.randint(0, cfg["vocab"], (70,), generator=torch.Generator().manual_seed(5)).tolist()
    whole = plain.forward(tokens, values, cfg)
    assert torch.allclose(plain.forward(tokens[:41], values, cfg), whole[:41], atol=1e-9)


MISTAKES = {
    "no embedding before later passes": lambda m: m.setattr(plain, "runs", lambda config, real=plain.runs: [(index, False) for index, _ in real(config)]),
    "a weight around one": lambda m: m.setattr(plain, "zero_centred_norm", lambda x, weight, eps: plain.unit_rms(x, eps) * weight),
    "a window one too long": lambda m: m.setattr(plain, "visible", lambda tokens, window=None, real=plain.visible: real(tokens, None if window is None else window + 1)),
    "a window one too short": lambda m: m.setattr(plain, "visible", lambda tokens, window=None, real=plain.visible: real(tokens, None if window is None else window - 1)),
    "no query temperature": lambda m: m.setattr(plain, "query_temperature", lambda tokens, coef, every: torch.ones(tokens, dtype=plain.F)),
    "a temperature one position late": lambda m: m.setattr(plain, "query_temperature", lambda tokens, coef, every, real=plain.query_temperature: torch.cat([torch.ones(1, dtype=plain.F), real(tokens, coef, every)[:-1]])),
    "no rotation": lambda m: m.setattr(plain, "rotate_pairs", lambda x, rotary_dim, base: x),
    "lambda without diff": lambda m: m.setattr(plain, "map_difference", lambda a, b, lam, diff, eps, real=plain.map_difference: real(a, b, lam - diff, diff, eps)),
    "no groups": lambda m: m.setattr(plain, "choose_experts", lambda scores, top, groups, keep, real=plain.choose_experts: real(scores, top, 1, 1)),
    "no clamp": lambda m: m.setattr(plain, "clamped_expert", lambda h, weights, prefix, limit, real=plain.clamped_expert: real(h, weights, prefix, 1e9)),
}


@pytest.mark.parametrize("mistake", sorted(MISTAKES))
def test_a_mistake_in_one_mechanism_shows(mistake, monkeypatch):
    """Each mechanism of the small models counts: with the mistake planted in the plain statement the logits of some position move by a
    hundred times what float32 is held to."""
    cfg = tm.MIXED if "window" not in mistake else tm.EDGY
    values = {key: value.double() for key, value in tm.weights(cfg, 11).items()}
    tokens = torch.randint(0, cfg["vocab"], (120,), generator=torch.Generator().manual_seed(6)).tolist()
    wanted = plain.forward(tokens, values, cfg)
    MISTAKES[mistake](monkeypatch)
    found = plain.forward(tokens, values, cfg)
    assert float((found - wanted).abs().max() / wanted.abs().max()) > 5e-3
