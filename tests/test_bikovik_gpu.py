"""Bikovik on the GPU against the plain statement in `plain_bikovik.py`: each mechanism's kernels alone, then whole models: whole prompts,
single tokens, portions, unequal batches, slots, pages and states that are used again, keys at every window's edge, among the first
positions and at page borders, long decoding, odd sizes, greedy generation through `generate()`, the command line and the trace replay."""
import json
import os
import subprocess
import sys
from types import SimpleNamespace

import numpy as np
import pytest
import torch

import bikovik_models as bm
import plain_bikovik as plain
from helpers import relative_error, run_batched, run_tail_stepwise, run_whole
from tau_rs_b200 import Engine, StepEntry, generate, load_model
from tau_rs_b200.csrc import kernels

pytestmark = pytest.mark.gpu
ROOT = os.path.dirname(os.path.dirname(os.path.abspath(__file__)))
TOLERANCE = {"float32": 5e-5, "bfloat16": 4e-2}
TORCH = {"float32": torch.float32, "bfloat16": torch.bfloat16}
DEVICE = "cuda"
F = torch.float64


def close(found, wanted, dtype) -> bool:
    """float32: every logit within 5e-5 of the largest.  bfloat16 (the plain statement rounds nothing): half of the positions within
    3e-2 of the largest logit and all but one in twenty (or two) within 8e-2."""
    if dtype == "float32":
        return relative_error(found, wanted) < TOLERANCE[dtype]
    rows = (found.double() - wanted.double()).abs().amax(dim=-1) / wanted.double().abs().max()
    return float(rows.median()) < 3e-2 and int((rows >= 8e-2).sum()) <= max(2, rows.numel() // 20)


def tokens_for(cfg, count, seed):
    return np.random.default_rng(seed).integers(0, cfg["vocab"], size=count).tolist()


_PLAIN = {}


def plain_logits(cfg, values, tokens):
    key = (id(values), tuple(tokens))
    if key not in _PLAIN:
        _PLAIN[key] = plain.forward(tokens, {name: value.double() for name, value in values.items()}, cfg).float()
    return _PLAIN[key]


@pytest.fixture(scope="module")
def models(tmp_path_factory):
    root = tmp_path_factory.mktemp("bikovik")
    made = {}
    listed = [("mixed", bm.MIXED, 11, {}), ("odd", bm.ODD, 12, {}), ("peaky", bm.PEAKY, 14, {}), ("heady", bm.HEADY, 17, {}), ("wide", bm.WIDE, 18, {}),
              ("long_memory", bm.LONG_MEMORY, 16, {"slow_forgetting": True})]
    listed += [("only_" + name, cfg, 20 + index, {}) for index, (name, cfg) in enumerate(bm.ONLY.items())]
    for name, cfg, seed, options in listed:
        folder = str(root / name)
        made[name] = (folder, cfg, bm.write_model(folder, cfg, seed, **options))
    return made


def engine_of(models, name, dtype, max_tokens=1024):
    folder, cfg, values = models[name]
    return Engine(load_model(folder, dtype, "gpu"), max_tokens), cfg, values


def on_device(tensor, dtype=torch.float32):
    return tensor.to(DEVICE, dtype).contiguous()


def as_ints(values):
    return torch.tensor(np.asarray(values, dtype=np.int32), device=DEVICE)


def packed_step(runs, slots):
    """The metadata of a step in which sequence i brings `runs[i]` tokens and sits in cache slot `slots[i]`."""
    bounds = np.concatenate([[0], np.cumsum(runs)]).astype(np.int32)
    token_seq = np.concatenate([np.full(count, index, dtype=np.int32) for index, count in enumerate(runs)])
    return SimpleNamespace(n_seqs=len(runs), token_seq=as_ints(token_seq), cu_seqlens=as_ints(bounds), seq_slot=as_ints(slots),
                           all_single=all(count == 1 for count in runs))


def rand(generator, *shape):
    return torch.randn(*shape, dtype=F, generator=generator)


# ---- the element-wise norm, the soft cap, the clamped gate ---------------------------------------------------------------
@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("width", [96, 100, 33, 1028, 4100, 1])
def test_the_dynamic_tanh_on_the_sum(dtype, width):
    generator = torch.Generator().manual_seed(width)
    stream, a, b, weight, bias = rand(generator, 9, width), rand(generator, 9, width), rand(generator, 9, width), rand(generator, width), rand(generator, width)
    alpha, kind = torch.tensor(0.7, dtype=F), TORCH[dtype]
    a_dev, b_dev = on_device(a, kind), on_device(b)              # a branch in the run's dtype beside one in 32-bit
    held = on_device(stream)
    tensors = (on_device(alpha), on_device(weight), on_device(bias))
    tolerance = 1e-6 if dtype == "float32" else 5e-3
    norm = lambda x: plain.dynamic_tanh(x, alpha.float().double(), weight.float().double(), bias.float().double())
    # Out of place, some rows only, in another order; the stream stays.
    rows = [7, 0, 3]
    out = torch.empty((3, width), dtype=kind, device=DEVICE)
    summed = stream.float().double() + 0.7 * (a_dev.double().cpu() + b_dev.double().cpu())
    kernels.stream_add_tanh(held, (a_dev, b_dev), *tensors, out, rows=as_ints(rows), update=False, branch_scale=0.7)
    assert relative_error(out.float().cpu(), norm(summed)[rows]) < tolerance and torch.equal(held.cpu(), stream.float())
    # No branch at all, then one in place: the stream takes the sum, the output its tanh.
    out = torch.empty((9, width), dtype=kind, device=DEVICE)
    kernels.stream_add_tanh(held, None, *tensors, out, update=False)
    assert relative_error(out.float().cpu(), norm(stream.float().double())) < tolerance
    kernels.stream_add_tanh(held, a_dev, *tensors, out, update=True)
    summed = stream.float().double() + a_dev.double().cpu()
    assert relative_error(held.cpu(), summed) < 1e-6 and relative_error(out.float().cpu(), norm(summed)) < tolerance


@pytest.mark.parametrize("shape", [(3, 211), (5, 64), (1, 1), (7, 1000)])
def test_the_soft_cap_on_logits(shape):
    values = rand(torch.Generator().manual_seed(shape[1]), *shape) * 20.0
    values[0, 0] = 1e6
    held = on_device(values)
    kernels.soft_cap(held, 7.5)
    assert relative_error(held.cpu(), plain.soft_cap(values.float().double(), 7.5)) < 1e-6
    assert float(held.abs().max()) <= 7.5


@pytest.mark.parametrize("dtype, hidden, ff, tokens", [("float32", 40, 24, 50), ("float32", 33, 7, 3), ("bfloat16", 64, 32, 3), ("bfloat16", 64, 40, 12), ("bfloat16", 64, 40, 300),
                                                       ("bfloat16", 96, 1032, 1100), ("bfloat16", 72, 30, 9), ("bfloat16", 1024, 512, 64)])
def test_the_clamped_feed_forward(dtype, hidden, ff, tokens):
    """As an epilogue of the skinny and the tensor-core products (with and without a cut along K, on pairs of SMs) and as a kernel of its
    own where the sizes do not allow that; gates and up values lie on both sides of the limit."""
    from tau_rs_b200.config.specs import SwiGLUSpec
    from tau_rs_b200.parts.registry import build

    generator = torch.Generator().manual_seed(hidden + ff)
    kind = TORCH[dtype]
    values = {"m.gate": rand(generator, ff, hidden) * 2.0 / hidden ** 0.5, "m.up": rand(generator, ff, hidden) * 2.0 / hidden ** 0.5, "m.down": rand(generator, hidden, ff) / ff ** 0.5}
    values = {name: value.to(torch.bfloat16).double() for name, value in values.items()}
    h = rand(generator, tokens, hidden).to(kind).double()
    part = build("feed_forward", SwiGLUSpec(hidden=hidden, intermediate=ff, gate_name="gate", up_name="up", down_name="down", weight_suffix="", activation="clamped", limit=1.3,
                                            wide_result=True), prefix="m", dtype=kind, device=DEVICE)
    for name in part.tensor_specs():
        part.assign(name, on_device(values[name], kind))
    part.finalize_weights()
    found = part.forward(on_device(h, kind), None)
    assert found.dtype == torch.float32
    assert relative_error(found.cpu(), plain.clamped_feed_forward(h, values, "m", 1.3)) < (1e-5 if dtype == "float32" else 1.5e-2)


# ---- the walks -------------------------------------------------------------------------------------------------------------
WALKS = [(3, 16, 24), (1, 20, 70), (5, 6, 1), (2, 100, 10), (4, 64, 64), (1, 256, 33), (2, 1, 5), (1, 300, 8), (16, 64, 96)]


@pytest.mark.parametrize("heads, dim, vdim", WALKS)
def test_what_is_forgotten_is_written_over_steps_with_slots_out_of_order(heads, dim, vdim):
    generator = torch.Generator().manual_seed(heads * dim + vdim)
    lengths, cuts, slots = [37, 5, 22], [(20, 1, 9), (1, 2, 1), (15, 1, 11), (1, 1, 1)], [4, 0, 2]
    width = 2 * heads * dim + heads * vdim
    state = torch.zeros((6, heads * vdim * dim), dtype=torch.float32, device=DEVICE)
    lower = 0.9 * torch.rand(heads * dim, dtype=F, generator=generator).float().double()
    rows = [rand(generator, length, width).float().double() for length in lengths]
    wanted = []
    for sequence in rows:
        q = plain.silu(sequence[:, : heads * dim]).reshape(-1, heads, dim)
        f = plain.forget_gate(sequence[:, heads * dim : 2 * heads * dim], lower).reshape(-1, heads, dim)
        wanted.append(plain.forget_write_recurrence(q, f, sequence[:, 2 * heads * dim :].reshape(-1, heads, vdim)).reshape(-1, heads * vdim))
    at = [0, 0, 0]
    for counts in cuts:
        step = packed_step(counts, slots)
        projected = on_device(torch.cat([rows[i][at[i] : at[i] + count] for i, count in enumerate(counts)]))
        read = torch.empty((sum(counts), heads * vdim), dtype=torch.float32, device=DEVICE)
        kernels.forget_gates(projected, 0, heads * dim, on_device(lower))
        kernels.wkv(projected[:, : heads * dim], None, projected[:, 2 * heads * dim :], projected[:, heads * dim : 2 * heads * dim], None, state, step.cu_seqlens, step.seq_slot,
                    read, heads, dim, vdim, form="forget_writes")
        expected = torch.cat([wanted[i][at[i] : at[i] + count] for i, count in enumerate(counts)])
        assert relative_error(read.cpu(), expected) < 2e-5
        at = [start + count for start, count in zip(at, counts)]
    assert at == lengths and not state[[1, 3, 5]].any()


@pytest.mark.parametrize("heads, dim, vdim", WALKS)
def test_turned_queries_and_keys_with_constant_decays_over_steps(heads, dim, vdim):
    generator = torch.Generator().manual_seed(heads * dim + vdim + 1)
    lengths, cuts, slots = [37, 5, 22], [(20, 1, 9), (1, 2, 1), (15, 1, 11), (1, 1, 1)], [4, 0, 2]
    rotary = dim // 4 * 2 if dim >= 4 else 0
    rot = {"dims": rotary, "base": 500.0}
    frequency = torch.tensor([500.0 ** (-2.0 * i / rotary) for i in range(rotary // 2)], dtype=F) if rotary else None
    width, k_width = 2 * heads * dim + heads * vdim + 3, heads * dim                # a few columns behind the values belong to somebody else
    decay = (1.0 - 0.5 * torch.rand(heads, dtype=F, generator=generator)).float().double()
    decay[0] = 1.0
    state = torch.zeros((6, heads * vdim * dim), dtype=torch.float32, device=DEVICE)
    rows = [rand(generator, length, width).float().double() for length in lengths]
    wanted = []
    for sequence in rows:
        heads_of = [sequence[:, begin : begin + k_width].reshape(-1, heads, dim) for begin in (0, k_width)]
        q, k = [plain.rotate_halves(part, rot) if rotary else part for part in heads_of]
        wanted.append(plain.decay_recurrence(q, k * 0.3, sequence[:, 2 * k_width : 2 * k_width + heads * vdim].reshape(-1, heads, vdim), decay).reshape(-1, heads * vdim))
    at = [0, 0, 0]
    for counts in cuts:
        step = packed_step(counts, slots)
        positions = as_ints([position for i, count in enumerate(counts) for position in range(at[i], at[i] + count)])
        projected = on_device(torch.cat([rows[i][at[i] : at[i] + count] for i, count in enumerate(counts)]))
        behind = projected[:, 2 * k_width :].clone()
        read = torch.empty((sum(counts), heads * vdim), dtype=torch.float32, device=DEVICE)
        kernels.turn_heads(projected, positions, None if frequency is None else on_device(frequency), rotary, 2 * heads, dim, heads, 0.3)
        assert torch.equal(projected[:, 2 * k_width :], behind)
        kernels.wkv(projected[:, :k_width], projected[:, k_width : 2 * k_width], projected[:, 2 * k_width : 2 * k_width + heads * vdim], None, on_device(decay), state,
                    step.cu_seqlens, step.seq_slot, read, heads, dim, vdim, form="constant_decay")
        expected = torch.cat([wanted[i][at[i] : at[i] + count] for i, count in enumerate(counts)])
        assert relative_error(read.cpu(), expected) < 2e-5
        at = [start + count for start, count in zip(at, counts)]
    assert at == lengths and not state[[1, 3, 5]].any()


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_a_gate_of_another_dtype_behind_the_norm_per_head(dtype):
    generator = torch.Generator().manual_seed(2)
    read, gate = rand(generator, 7, 60), rand(generator, 7, 60)
    out = torch.empty((7, 60), dtype=TORCH[dtype], device=DEVICE)
    kernels.gated_group_norm(on_device(read), None, on_device(gate), out, 5, 1e-3, True, silu_gate=True)
    wanted = plain.unit_rms(read.float().double().reshape(7, 5, 12), 1e-3).reshape(7, 60) * plain.silu(gate.float().double())
    assert relative_error(out.float().cpu(), wanted) < (1e-5 if dtype == "float32" else 1e-2)


# ---- attention -------------------------------------------------------------------------------------------------------------
def run_attention(q, k, v, scale, talk, window, keep_first, dtype, page_of, heads_layout, single_from, mode):
    """One sequence: the first `single_from` tokens as one run, the others one by one.  `mode` says how: "kernel" (mixed queries against all
    key heads, a warp per head), "single" (single tokens through the kernel that mixes scores), "side" (single tokens, mixed queries on the tensor cores), "tensor" (runs on the
    tensor cores)."""
    tokens, heads, dim = q.shape
    kv_heads, vdim = v.shape[1], v.shape[2]
    kind, n_pages = TORCH[dtype], max(page_of) + 2
    keys = torch.full((n_pages, kv_heads, 64, dim) if heads_layout else (n_pages, 64, kv_heads * (dim + vdim)), 9.0, dtype=kind, device=DEVICE)
    values = torch.full((n_pages, kv_heads, 64, vdim), 9.0, dtype=kind, device=DEVICE) if heads_layout else None
    pages, out = as_ints([page_of]), torch.empty((tokens, heads * vdim), dtype=kind, device=DEVICE)
    projected = on_device(torch.cat([part.reshape(tokens, -1) for part in (q, k, v)], dim=1), kind)
    talk = on_device(talk)
    for begin, end in [(0, single_from)] + [(position, position + 1) for position in range(single_from, tokens)]:
        step = SimpleNamespace(positions=as_ints(list(range(begin, end))), token_seq=as_ints([0] * (end - begin)))
        single = mode == "single" and end - begin == 1
        queries = torch.empty((end - begin, heads, dim if single else kv_heads * dim), dtype=kind, device=DEVICE)
        kernels.masked_prepare(projected[begin:end], None, None, 1e-5, None, 0, 1.0, queries, keys, step.positions, step.token_seq, pages, heads, kv_heads, dim, vdim, True, values,
                               talk=None if single else talk)
        if single:
            kernels.talking_decode(queries, keys, talk, out[begin:end], step, pages, kv_heads, vdim, scale, window, keep_first, 1.0, values, splits=1 + (begin - single_from) % 5)
        elif mode == "side" and end - begin == 1:
            kernels.shared_key_decode(queries, keys, out[begin:end], step, pages, kv_heads, vdim, scale, window, keep_first, 1.0, values, splits=1 + (begin - single_from) % 5)
        elif mode == "tensor" and end - begin > 1:
            kernels.attention_prefill_tc(queries.view(end - begin, -1), keys, values, out[begin:end], as_ints([0, end - begin]), as_ints([begin]), pages, heads, kv_heads, dim,
                                         scale, window, keep_first=keep_first, segmented=True)
        else:
            kernels.masked_attention(queries, keys, out[begin:end], step, pages, kv_heads, vdim, scale, window, value_pages=values, keep_first=keep_first, shared_keys=True)
    return out.float().cpu()


SIZES = [(4, 2, 16, 24, False), (1, 1, 12, 150, False), (9, 3, 10, 6, False), (6, 1, 96, 96, False), (2, 1, 64, 64, True), (4, 2, 128, 128, True), (5, 5, 8, 16, False),
         (16, 4, 128, 128, True), (8, 8, 64, 64, True), (20, 4, 32, 48, False), (8, 8, 128, 128, True), (40, 2, 48, 40, False), (18, 6, 16, 8, False)]


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("heads, kv_heads, dim, vdim, heads_layout", SIZES)
@pytest.mark.parametrize("window, keep_first", [(70, 9), (64, 64), (1, 0), (300, 5), (33, 130)])
def test_mixed_scores_with_a_window_and_kept_positions_over_scattered_pages(dtype, heads, kv_heads, dim, vdim, heads_layout, window, keep_first):
    generator = torch.Generator().manual_seed(heads * 10 + dim + window)
    tokens, kind = 240, TORCH[dtype]
    rounded = lambda t: t.to(kind).double()
    q, k, v = rounded(rand(generator, tokens, heads, dim)), rounded(rand(generator, tokens, kv_heads, dim)), rounded(rand(generator, tokens, kv_heads, vdim))
    talk = (torch.eye(heads, dtype=F) + 0.5 * rand(generator, heads, heads) / heads ** 0.5).float().double()
    wanted = plain.talking_attention(q, k, v, dim ** -0.5, talk, plain.visible_keys(tokens, window, keep_first)).reshape(tokens, -1)
    tolerance = 2e-5 if dtype == "float32" else 2e-2
    per = 4 if dtype == "float32" else 8
    modes = ["kernel"] + (["single"] if dim % per == 0 and vdim % per == 0 and kernels.talking_decode_fits(kind, heads, kv_heads, dim, vdim) else [])
    if kernels.shared_key_decode_fits(kind, heads, kv_heads, dim, vdim):
        modes.append("side")
    assert dtype == "float32" or dim % 16 or "side" in modes
    if heads_layout and dtype == "bfloat16":      # (8 key heads of 128: the pieces of the queries travel with the keys)
        modes.append("tensor")
    for mode in modes:
        found = run_attention(q, k, v, dim ** -0.5, talk, window, keep_first, dtype, [5, 2, 7, 0], heads_layout, 210, mode)
        assert relative_error(found, wanted) < tolerance, mode
    if heads_layout:
        assert kernels.attention_prefill_tc_status(dim) == 0


@pytest.mark.parametrize("heads, kv_heads, dim, tokens, window, keep_first", [(16, 4, 128, 1500, 600, 70), (32, 8, 64, 1100, 1000, 1), (16, 8, 128, 1300, 64, 200), (24, 1, 128, 1250, 333, 0)])
def test_long_runs_with_more_tiles_than_the_machine_holds_blocks(heads, kv_heads, dim, tokens, window, keep_first):
    """Every block of the tensor-core kernel walks several items with odd and even numbers of pages."""
    generator = torch.Generator().manual_seed(tokens)
    rounded = lambda t: t.to(torch.bfloat16).double()
    q, k, v = rounded(rand(generator, tokens, heads, dim)), rounded(rand(generator, tokens, kv_heads, dim)), rounded(rand(generator, tokens, kv_heads, dim))
    talk = (torch.eye(heads, dtype=F) + 0.5 * rand(generator, heads, heads) / heads ** 0.5).float().double()
    wanted = plain.talking_attention(q, k, v, dim ** -0.5, talk, plain.visible_keys(tokens, window, keep_first)).reshape(tokens, -1)
    pages = torch.randperm(-(-tokens // 64), generator=generator).tolist()
    found = run_attention(q, k, v, dim ** -0.5, talk, window, keep_first, "bfloat16", pages, True, tokens, "tensor")
    assert kernels.attention_prefill_tc_status(dim) == 0
    assert relative_error(found, wanted) < 2e-2


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("dim, heads_layout", [(16, False), (64, True), (128, True)])
@pytest.mark.parametrize("window, keep_first", [(64, 3), (70, 64), (100, 65), (129, 1)])
def test_one_key_that_stands_out_is_seen_exactly_inside_the_window_and_among_the_first(dtype, dim, heads_layout, window, keep_first):
    """Every key but one scores far below the rest, so a query that sees that key returns its value, and one that does not sees it gone:
    the key stands at the last kept position, the first one behind the kept ones, and at a page's border; queries sit at the window's
    last visible and first hidden distance, in a run and as single tokens."""
    generator = torch.Generator().manual_seed(window)
    tokens, heads, kv_heads = 330, 2, 2
    talk = torch.tensor([[0.5, 0.5], [0.25, 1.0]], dtype=F)
    for far in sorted({0, keep_first - 1, keep_first, 63, 64, 127, 128, 190}):
        k = rand(generator, tokens, kv_heads, dim) * 0.02
        k[:, :, 3] = -4.0
        k[far, :, 3] = 4.0
        q = torch.zeros(tokens, heads, dim, dtype=F)
        q[:, :, 3] = 8.0
        v = rand(generator, tokens, kv_heads, dim)
        rounded = v.to(TORCH[dtype]).double()
        edges = [far, far + window - 1, far + window, far + 300]
        for mode in ["single"] + (["side"] if dtype == "bfloat16" else []) + (["tensor"] if heads_layout and dtype == "bfloat16" else ["kernel"]):
            single_from = 2 if mode in ("single", "side") else tokens
            found = run_attention(q, k, v, 1.0, talk, window, keep_first, dtype, [4, 1, 6, 3, 0, 2], heads_layout, single_from, mode).reshape(tokens, heads, dim)
            for position in edges:
                if position >= tokens:
                    continue
                seen = position - far < window or far < keep_first
                error = float((found[position].double() - rounded[far]).abs().max() / rounded[far].abs().max())
                assert (error < 2e-2) == seen and (seen or error > 0.1), (far, position, mode)


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_values_are_mixed_with_the_first_layers_values_before_they_are_cached(dtype):
    generator = torch.Generator().manual_seed(8)
    heads, kv_heads, dim, vdim, tokens, kind = 3, 1, 10, 6, 50, TORCH[dtype]
    projected = rand(generator, tokens, heads * dim + kv_heads * (dim + vdim)).to(kind)
    first = rand(generator, tokens, 30).to(kind)
    share = torch.tensor(0.3, dtype=torch.float32)
    rows = torch.full((4, 64, kv_heads * (dim + vdim)), 9.0, dtype=kind, device=DEVICE)
    queries = torch.empty((tokens, heads, dim), dtype=kind, device=DEVICE)
    kernels.masked_prepare(on_device(projected, kind), None, None, 1e-5, None, 0, 1.0, queries, rows, as_ints(list(range(tokens))), as_ints([0] * tokens), as_ints([[2, 0]]), heads,
                           kv_heads, dim, vdim, first_values=on_device(first, kind)[:, 7:13], value_share=share.to(DEVICE))
    wanted = plain.mixed_values(projected[:, heads * dim + dim :].double(), first[:, 7:13].double(), share.double())
    assert relative_error(rows[2, :tokens, dim:].float().cpu(), wanted) < (1e-6 if dtype == "float32" else 5e-3)
    assert torch.equal(rows[2, :tokens, :dim].cpu(), projected[:, heads * dim : heads * dim + dim])


# ---- whole models: one mechanism to a model, then all together ----------------------------------------------------------
@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("name", ["only_attention", "only_mixed_values", "only_hgrn2", "only_retention", "only_dense", "mixed", "odd", "heady", "wide"])
def test_whole_prompts_single_tokens_and_the_first_positions(models, name, dtype):
    engine, cfg, values = engine_of(models, name, dtype)
    tokens = tokens_for(cfg, 200, 21)
    wanted = plain_logits(cfg, values, tokens)
    whole = run_whole(engine, tokens)
    assert close(whole, wanted, dtype)
    assert close(whole[:4], wanted[:4], dtype)               # the first tokens: empty states, one key
    assert close(run_whole(engine, tokens[:1]), wanted[:1], dtype)
    stepwise = run_tail_stepwise(engine, tokens, 199)                              # every token but the first alone, through the graphs
    assert close(stepwise, wanted[1:], dtype)
    if dtype == "float32":
        assert relative_error(stepwise, whole[1:]) < 2e-5


def test_the_residual_stream_after_every_layer(models):
    """Layer by layer in 32-bit: the stream that the model hands from block to block, with what is still to join it, against the
    plain statement's."""
    folder, cfg, values = models["mixed"]
    tokens = tokens_for(cfg, 90, 26)
    _, layers = plain.forward(tokens, {name: value.double() for name, value in values.items()}, cfg, return_layers=True)
    model = load_model(folder, "float32", "gpu")
    engine = Engine(model, 256)
    kept = []
    for block in model.blocks:
        original = block.forward

        def recording(hidden, *args, _original=original, **kwargs):
            stream, pending = _original(hidden, *args, **kwargs)
            kept.append(stream.double().cpu() + pending.double().cpu())
            return stream, pending

        block.forward = recording
    run_whole(engine, tokens)
    assert len(kept) == len(cfg["layers"])
    for index, (found, wanted) in enumerate(zip(kept, layers)):
        assert relative_error(found, wanted) < 2e-5, index


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("name", ["mixed", "odd", "long_memory", "heady"])
def test_portions_down_to_two_tokens_and_page_borders(models, name, dtype):
    engine, cfg, values = engine_of(models, name, dtype)
    tokens = tokens_for(cfg, 330, 22)
    wanted = plain_logits(cfg, values, tokens)
    slot = engine.open_sequence()
    found, position = [], 0
    for count in [2, 2, 3, 56, 1, 1, 62, 2, 64, 1, 63, 2, 5, 64, 2]:               # runs that end at, before and behind positions 63/64, 127/128, ...
        piece = tokens[position : position + count]
        found.append(engine.step([StepEntry(slot, piece, list(range(count)))]).float().cpu().clone())
        position += count
        engine.cache.check()
    assert position == 330
    engine.close_sequence(slot)
    assert close(torch.cat(found), wanted, dtype)


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("name", ["peaky", "heady"])
def test_sharp_weights_lose_no_key_at_a_windows_edge_or_among_the_first(models, name, dtype):
    engine, cfg, values = engine_of(models, name, dtype)
    tokens = tokens_for(cfg, 400, 23)
    wanted = plain_logits(cfg, values, tokens)
    assert close(run_whole(engine, tokens), wanted, dtype)
    tail = run_tail_stepwise(engine, tokens, 150)                                  # decoded queries cross page borders
    assert close(tail, wanted[-150:], dtype)
    slot = engine.open_sequence()                                                  # portions that read keys of earlier portions
    found = [engine.step([StepEntry(slot, tokens[begin : begin + 50], list(range(50)))]).float().cpu().clone() for begin in range(0, 400, 50)]
    engine.close_sequence(slot)
    assert close(torch.cat(found), wanted, dtype)
    # The test would see a window that is one token off or a first position that is lost.
    doubles = {key: value.double() for key, value in values.items()}
    for key, change in (("size", 1), ("size", -1), ("keep_first", 1), ("keep_first", -1)):
        moved = json.loads(json.dumps(cfg))
        for layer in moved["layers"]:
            layer["mixer"]["mask"][key] += change
        assert relative_error(plain.forward(tokens, doubles, moved)[-150:], wanted[-150:]) > 1e-3


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("name", ["mixed", "odd", "heady"])
def test_unequal_batches_against_each_request_alone(models, name, dtype):
    engine, cfg, values = engine_of(models, name, dtype, 2048)
    lengths, prompts = [90, 31, 140, 5, 66], [70, 1, 129, 3, 64]
    requests = [tokens_for(cfg, length, 30 + index) for index, length in enumerate(lengths)]
    together = run_batched(engine, requests, prompts)
    for request, prompt, rows in zip(requests, prompts, together):
        wanted = plain_logits(cfg, values, request)[prompt - 1 :]
        assert close(rows, wanted, dtype)
    engine.cache.check()
    assert engine.cache.slots.in_use == 0


def test_slots_pages_and_states_that_are_used_again_start_clean(models):
    """A cache of three pages and as many slots: every request takes a slot whose states another left behind, and pages that another wrote."""
    engine, cfg, values = engine_of(models, "mixed", "float32", 64 * 3)
    for round_number in range(4):
        requests = [tokens_for(cfg, length, 40 + 3 * round_number + index) for index, length in enumerate([60 + round_number, 40, 17])]
        together = run_batched(engine, requests, [len(request) - 6 for request in requests])
        for request, rows in zip(requests, together):
            assert relative_error(rows, plain_logits(cfg, values, request)[len(request) - 7 :]) < TOLERANCE["float32"]
        engine.cache.check()


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_a_sequence_longer_than_its_cache_keeps_its_first_pages(models, dtype):
    """600 positions through a cache of 9 pages: pages between the first ones and the window go back and are taken again, and no query
    loses a key of either kind."""
    engine, cfg, values = engine_of(models, "heady", dtype, 64 * 9)
    tokens = tokens_for(cfg, 600, 25)
    wanted = plain_logits(cfg, values, tokens)
    slot = engine.open_sequence()
    found, position = [], 0
    while position < 600:
        count = min([50, 1, 1, 64, 30, 1][len(found) % 6], 600 - position)
        found.append(engine.step([StepEntry(slot, tokens[position : position + count], list(range(count)))]).float().cpu().clone())
        position += count
        engine.cache.check()
    engine.close_sequence(slot)
    assert close(torch.cat(found), wanted, dtype)


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_states_that_forget_slowly_over_long_decoding(models, dtype):
    """Decays close to one: a state that was lost, restarted or carried by the wrong sequence shows hundreds of tokens later."""
    engine, cfg, values = engine_of(models, "long_memory", dtype)
    tokens = tokens_for(cfg, 420, 24)
    wanted = plain_logits(cfg, values, tokens)
    assert close(run_tail_stepwise(engine, tokens, 400), wanted[-400:], dtype)
    shortened = plain_logits(cfg, values, tokens[100:])                            # the test would see a state that began later
    assert relative_error(shortened[-50:], wanted[-50:]) > 1e-3


def test_long_decoding_in_bfloat16_stays_with_the_plain_statement(models):
    engine, cfg, values = engine_of(models, "mixed", "bfloat16")
    tokens = tokens_for(cfg, 420, 24)
    wanted = plain_logits(cfg, values, tokens)
    assert close(run_tail_stepwise(engine, tokens, 400), wanted[-400:], "bfloat16")


@pytest.mark.parametrize("name", ["mixed", "odd"])
def test_greedy_generation_through_the_library_entry_point(models, name):
    folder, cfg, values = models[name]
    prompts = [tokens_for(cfg, length, 60 + index) for index, length in enumerate([9, 30, 2])]
    output = generate(folder, prompts, max_new_tokens=12, dtype="float32", stop_tokens=[])
    for prompt, result in zip(prompts, output):
        tokens = list(prompt)
        for _ in range(12):
            logits = plain_logits(cfg, values, tokens)[-1]
            best, second = torch.topk(logits, 2).values
            if float(best - second) < 1e-3 * float(logits.abs().max()):
                break                                                                # a close call proves nothing either way
            tokens.append(int(torch.argmax(logits)))
        made = len(tokens) - len(prompt)
        assert list(result.tokens[:made]) == tokens[len(prompt) :] and made >= 1


def test_trace_replay_of_a_bikovik_folder(models, tmp_path):
    folder, cfg, values = models["mixed"]
    first, second = tokens_for(cfg, 70, 70), tokens_for(cfg, 33, 71)
    steps = [{"step": 0, "entries": [{"id": "a", "tokens": first[:66], "want": [0, 65]}, {"id": "b", "tokens": second[:30], "want": [29]}], "end": []}]
    for index in range(3):
        steps.append({"step": index + 1, "entries": [{"id": "a", "tokens": [first[66 + index]], "want": [0]}, {"id": "b", "tokens": [second[30 + index]], "want": [0]}],
                      "end": ["b"] if index == 2 else []})
    steps.append({"step": 4, "entries": [{"id": "a", "tokens": [first[69]], "want": []}], "end": ["a"]})
    out = tmp_path / "out"
    done = subprocess.run([sys.executable, os.path.join(ROOT, "bin", "trace_run"), "--model", folder, "--dtype", "float32", "--out", str(out), "--max-tokens", "256"],
                          input="\n".join(json.dumps(step) for step in steps) + "\n", capture_output=True, text=True, timeout=900)
    assert done.returncode == 0, done.stderr[-2000:]
    assert [line for line in done.stdout.split("\n") if line.startswith("done")] == [f"done {index}" for index in range(5)]
    wanted_a, wanted_b = plain_logits(cfg, values, first), plain_logits(cfg, values, second)
    rows = np.fromfile(out / "0.f32", dtype="<f4").reshape(3, cfg["vocab"])
    assert relative_error(torch.from_numpy(rows), torch.stack([wanted_a[0], wanted_a[65], wanted_b[29]])) < TOLERANCE["float32"]
    rows = np.fromfile(out / "3.f32", dtype="<f4").reshape(2, cfg["vocab"])
    assert relative_error(torch.from_numpy(rows), torch.stack([wanted_a[68], wanted_b[32]])) < TOLERANCE["float32"]
    assert not (out / "4.f32").exists()


def test_the_command_line_on_a_bikovik_folder(models, tmp_path):
    """`bin/tau` on a Bikovik folder: greedy tokens in 32-bit equal those of `generate()`, with graphs and without, in chunks of
    prompt tokens; bfloat16 runs from the same folder; random weights are written for a Bikovik config.json and read back."""
    folder, cfg, values = models["mixed"]
    prompts = [tokens_for(cfg, 40, 80), tokens_for(cfg, 7, 81)]
    wanted = [list(result.tokens) for result in generate(folder, prompts, max_new_tokens=8, dtype="float32", stop_tokens=[])]

    def run(arguments):
        done = subprocess.run([os.path.join(ROOT, "bin", "tau")] + arguments, capture_output=True, text=True, timeout=900)
        assert done.returncode == 0, done.stderr[-2000:]
        return [json.loads(line) for line in done.stdout.splitlines() if line.startswith("{")]

    base = ["--model", folder, "--max-tokens", "8", "--stop-ids", ""]
    for prompt in prompts:
        base += ["--prompt-ids", ",".join(str(token) for token in prompt)]
    records = run(base + ["--dtype", "f32"])
    assert [record["tokens"] for record in records if "tokens" in record] == wanted
    records = run(base + ["--dtype", "f32", "--cuda-graph", "none", "--prefill-chunk-size", "16"])
    assert [record["tokens"] for record in records if "tokens" in record] == wanted
    records = run(base + ["--dtype", "bf16"])
    assert all(len(record["tokens"]) == 8 for record in records if "tokens" in record)
    config_path = tmp_path / "config.json"
    config_path.write_text(json.dumps(bm.PEAKY))
    drawn = str(tmp_path / "drawn")
    records = run(["--random-weights", str(config_path), "--model", drawn, "--seed", "4", "--max-tokens", "5", "--stop-ids", "", "--prompt-ids", "1,2,3"])
    assert [len(record["tokens"]) for record in records if "tokens" in record] == [5]
