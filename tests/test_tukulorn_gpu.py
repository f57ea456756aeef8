"""Tukulorn on the GPU against the plain statement in `plain_tukulorn.py`: each mechanism alone, then whole models: whole prompts, single
tokens, portions, unequal batches, slots and pages that are used again, windows' edges and page borders, keys far back, the stream
behind every run, long decoding, odd sizes, greedy generation through `generate()`, the command line and the trace replay."""
import json
import os
import subprocess
import sys
from types import SimpleNamespace

import numpy as np
import pytest
import torch

import plain_tukulorn as plain
import tukulorn_models as tm
from helpers import relative_error, run_batched, run_tail_stepwise, run_whole
from tau_rs_b200 import Engine, StepEntry, generate, load_model
from tau_rs_b200.config import DifferentialAttentionSpec, LatentAttentionSpec, NormSpec, PairRotationSpec, RoutedExpertsSpec
from tau_rs_b200.parts.base import Pending
from tau_rs_b200.parts.registry import build

pytestmark = pytest.mark.gpu
ROOT = os.path.dirname(os.path.dirname(os.path.abspath(__file__)))
TORCH = {"float32": torch.float32, "bfloat16": torch.bfloat16}
DEVICE = "cuda"


def close(found, wanted, dtype) -> bool:
    """float32: every logit within 5e-5 of the largest.  bfloat16 (the plain statement rounds nothing): half of the positions within
    2e-2 of the largest logit and nine in ten within 6e-2; where two experts or groups were a close call the library and the plain
    statement may choose differently at a position, which says nothing about either (the float32 runs pin every choice)."""
    if dtype == "float32":
        return relative_error(found, wanted) < 5e-5
    rows = (found.double() - wanted.double()).abs().amax(dim=-1) / wanted.double().abs().max()
    return float(rows.median()) < 2e-2 and float(torch.quantile(rows, 0.9)) < 6e-2


def tokens_for(cfg, count, seed):
    return np.random.default_rng(seed).integers(0, cfg["vocab"], size=count).tolist()


def doubled(values):
    return {name: value.double() for name, value in values.items()}


_PLAIN = {}


def plain_logits(cfg, values, tokens):
    key = (id(values), tuple(tokens))
    if key not in _PLAIN:
        _PLAIN[key] = plain.forward(tokens, doubled(values), cfg).float()
    return _PLAIN[key]


@pytest.fixture(scope="module")
def models(tmp_path_factory):
    root = tmp_path_factory.mktemp("tukulorn")
    made = {}
    for name, cfg, seed in (("mixed", tm.MIXED, 11), ("odd", tm.ODD, 12), ("wide", tm.WIDE, 13), ("peaky", tm.PEAKY, 14), ("edgy", tm.EDGY, 15)):
        folder = str(root / name)
        made[name] = (folder, cfg, tm.write_model(folder, cfg, seed))
    return made


def engine_of(models, name, dtype, max_tokens=1024):
    folder, cfg, values = models[name]
    return Engine(load_model(folder, dtype, "gpu"), max_tokens), cfg, values


def on_device(tensor, dtype=torch.float32):
    return tensor.to(DEVICE, dtype).contiguous()


# ---- each mechanism alone ----------------------------------------------------------------------------------------------
@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("width, groups", [(320, 1), (1364, 1), (4100, 1), (203, 1), (8196, 1), (96, 4)])      # 16-byte pieces of one to eight a thread; single columns; pieces normalised one by one
def test_the_norm_around_zero_on_what_joins_the_stream(dtype, width, groups):
    """Two results, factors per channel, one number, and looked-up rows with a factor of their own, together and alone."""
    torch.manual_seed(width)
    rows, vocab, eps = 13, 9, 1e-3
    norm = build("norm", NormSpec(width=width, eps=eps, groups=groups, weight_offset=1.0), name="n", dtype=TORCH[dtype], device=DEVICE)
    weight = 0.3 * torch.randn(width)
    assert set(norm.tensor_specs()) == {"n"}
    norm.assign("n", on_device(weight))
    norm.finalize_weights()

    def normed(x):
        return plain.unit_rms(x.view(-1, groups, width // groups), eps).view(-1, width) * (1.0 + weight.double())

    stream, a, b = torch.randn(rows, width), torch.randn(rows, width).to(TORCH[dtype]).float(), torch.randn(rows, width)
    factors, table, numbers = torch.randn(width), torch.randn(vocab, width).to(TORCH[dtype]).float(), torch.randint(0, vocab, (rows,), dtype=torch.int32)
    looked_up = (on_device(table, TORCH[dtype]), numbers.to(DEVICE), 1.5)
    cases = [(Pending((on_device(a, TORCH[dtype]), on_device(b)), 0.5, on_device(factors)), 0.5 * factors.double() * (a.double() + b.double())),
             (Pending((on_device(a, TORCH[dtype]),), channel_scale=on_device(factors), rows=looked_up), factors.double() * a.double() + 1.5 * table.double()[numbers.long()]),
             (Pending.with_rows(None, looked_up), 1.5 * table.double()[numbers.long()]),
             (Pending.with_rows(on_device(b), looked_up), b.double() + 1.5 * table.double()[numbers.long()])]
    tolerance = 3e-6 if dtype == "float32" else 6e-3
    for pending, joined in cases:
        held = on_device(stream)
        out = norm.add_forward(pending, held)
        wanted = stream.double() + joined
        assert out.dtype == TORCH[dtype] and relative_error(held.cpu(), wanted) < 2e-6
        assert relative_error(out.float().cpu(), normed(wanted)) < tolerance
        held, chosen = on_device(stream), torch.tensor([rows - 1, 0, 4, 4], dtype=torch.int32)
        out = norm.forward(held, rows=chosen.to(DEVICE), branch=pending)              # gathered rows; the stream stays as it is
        assert torch.equal(held.cpu(), stream) and relative_error(out.float().cpu(), normed(wanted)[chosen.long()]) < tolerance
    assert relative_error(norm.forward(on_device(stream)).float().cpu(), normed(stream.double())) < tolerance


@pytest.mark.parametrize("heads, width, value_dim", [(3, 24, 20), (1, 10, 10), (9, 13, 7), (16, 192, 128)])
@pytest.mark.parametrize("per_head", [True, False])
def test_the_gate_on_heads(heads, width, value_dim, per_head):
    from tau_rs_b200.csrc import kernels

    torch.manual_seed(heads)
    tokens = 17
    values, gate = torch.randn(tokens, heads * width), 2.0 * torch.randn(tokens, (heads if per_head else heads * value_dim) + 3)
    for values_dtype, dtype in (("float32", "float32"), ("float32", "bfloat16"), ("bfloat16", "bfloat16")):
        v, g = values.to(TORCH[values_dtype]), gate.to(TORCH[dtype])
        out = torch.empty(tokens, heads * value_dim, dtype=TORCH[dtype], device=DEVICE)
        kernels.head_gate(on_device(v, TORCH[values_dtype]), on_device(g, TORCH[dtype])[:, : gate.shape[1] - 3], out, heads, width, value_dim, per_head)
        z = plain.sigmoid(g.double()[:, : gate.shape[1] - 3]).view(tokens, heads, -1)
        wanted = v.double().view(tokens, heads, width)[:, :, :value_dim] * z
        assert relative_error(out.float().cpu(), wanted.reshape(tokens, -1)) < (1e-6 if dtype == "float32" else 5e-3)


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("experts, top, groups, keep, tokens, width", [
    (12, 3, 4, 2, 41, 72), (8, 2, 4, 3, 41, 72), (1, 1, 1, 1, 41, 72), (5, 2, 5, 3, 41, 72), (6, 6, 2, 2, 41, 72), (64, 6, 8, 3, 41, 72), (160, 4, 40, 7, 41, 72), (40, 1, 40, 1, 41, 72),
    (6, 2, 1, 1, 41, 72), (12, 3, 4, 2, 601, 72), (8, 2, 4, 3, 602, 75), (10, 2, 5, 2, 594, 300), (8, 2, 4, 3, 350, 75)])      # one token to a block of many warps, of few, four to a block
def test_the_router_chooses_among_the_best_groups(dtype, experts, top, groups, keep, tokens, width):
    from tau_rs_b200.csrc import kernels

    torch.manual_seed(experts + top)
    scale, shared = 2.3, torch.randn(width) * 0.2
    hidden, router = torch.randn(tokens, width).to(TORCH[dtype]).float(), torch.randn(experts, width) * 0.3
    if experts >= 8:
        router[experts // 2] = router[experts // 2 + 1]                     # two experts that always tie
    hidden[0] = 0.0                                                         # a token whose experts all tie: the lowest numbers
    chosen = torch.empty((tokens, top), dtype=torch.int32, device=DEVICE)
    weights = torch.empty((tokens, top), dtype=torch.float32, device=DEVICE)
    shared_gate = torch.empty(tokens, dtype=torch.float32, device=DEVICE)
    kernels.moe_route(on_device(hidden, TORCH[dtype]), on_device(router), None, on_device(shared), chosen, weights, shared_gate, top, False, True, None, groups=groups, keep=keep,
                      scale=scale)
    assert torch.allclose(shared_gate.cpu().double(), plain.sigmoid(hidden.double() @ shared.double()), atol=2e-6)
    chosen, weights = chosen.cpu(), weights.cpu()
    scores = plain.sigmoid(hidden.double() @ router.double().T)
    kept_apart = 0
    for token in range(tokens):
        row = scores[token].float().tolist()                                # ties are ties of the 32-bit scores
        wanted = plain.choose_experts(row, top, groups, keep)
        assert chosen[token].tolist() == wanted, token
        picked = scores[token][wanted]
        assert torch.allclose(weights[token].double(), picked / (picked.sum() + 1e-20) * scale, atol=2e-6)
        kept_apart += wanted != plain.choose_experts(row, top, 1, 1)
    assert kept_apart > 0 or groups == keep or experts == groups      # groups of one expert keep the best experts anyway


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("hidden, ff, tokens", [(96, 40, 5), (96, 40, 300), (100, 12, 300), (64, 24, 1)])      # streamed, grouped tensor-core products, sizes that those refuse
def test_clamped_experts_through_every_product(dtype, hidden, ff, tokens):
    mlp = tm.moe(experts=12, top=3, count=4, keep=2, ff=ff, limit=0.6, scale=1.7)
    values = {name.removeprefix("l0.mlp"): value for name, value in tm.weights(tm.config([tm.latent(mlp=mlp)], width=hidden), 31).items() if ".mlp." in name}
    values = {f"m{name}": value * (1.0 if "router" in name else 1.5) for name, value in values.items()}
    values = {name: value.to(torch.bfloat16).float() for name, value in values.items()}
    part = build("feed_forward", RoutedExpertsSpec(hidden=hidden, intermediate=ff, experts=12, top=3, correction=False, renormalize=True, groups=4, keep_groups=2, scale=1.7,
                                                   activation="clamped", limit=0.6), prefix="m", dtype=TORCH[dtype], device=DEVICE)
    for name, spec in part.tensor_specs().items():
        part.assign(name, on_device(values[name], TORCH[dtype] if spec.role == "matrix" else torch.float32))
    part.finalize_weights()
    torch.manual_seed(7)
    h = torch.randn(tokens, hidden).to(torch.bfloat16).float()
    found = part.forward(on_device(h, TORCH[dtype]), SimpleNamespace(all_single=tokens == 1)).cpu()
    wanted = plain.routed_feed_forward(h.double(), doubled(values), "m", mlp)
    unclamped = plain.routed_feed_forward(h.double(), doubled(values), "m", {**mlp, "expert": {"ff": ff, "limit": 100.0}})
    assert relative_error(unclamped, wanted) > 0.2
    rows = (found.double() - wanted).abs().amax(-1) / wanted.abs().max()
    assert float(rows.max()) < (1e-5 if dtype == "float32" else 2e-2)


class Alone:
    """One mixer and the pages of one sequence, scattered over a pool; runs of tokens go through the mixer one after the other."""

    def __init__(self, spec, values, dtype, page_of, pages=8, fill=float("nan")):
        self.part, self.dtype, self.page_of, self.length = build("mixer", spec, prefix="m", dtype=TORCH[dtype], device=DEVICE), TORCH[dtype], page_of, 0
        for name, tensor_spec in self.part.tensor_specs().items():
            self.part.assign(name, on_device(values[name], self.dtype if tensor_spec.role == "matrix" else torch.float32))
        self.part.finalize_weights()
        need = self.part.cache_need()
        shape = (pages, 64, need.row_width) if need.kind == "rows" else (pages, need.n_kv_heads, 64, need.head_dim)
        self.pools = [torch.full(shape, fill, dtype=self.dtype, device=DEVICE) for _ in range(1 if need.kind == "rows" else 2)]
        self.cache = SimpleNamespace(group="g", **(dict(rows=self.pools[0]) if need.kind == "rows" else dict(keys=self.pools[0], values=self.pools[1])))

    def run(self, h, splits=0):
        count, start = h.shape[0], self.length
        self.length += count
        ints = lambda values: torch.tensor(values, dtype=torch.int32, device=DEVICE)
        step = SimpleNamespace(positions=ints(list(range(start, start + count))), token_seq=ints([0] * count), n_seqs=1, all_single=count == 1, all_fresh=start == 0,
                               decode_splits=splits, max_len=start + count, max_new=count, cu_seqlens=ints([0, count]), seq_start=ints([start]), seq_len=ints([start + count]),
                               page_rows={"g": ints([self.page_of])})
        return self.part.forward(on_device(h, self.dtype), step, self.cache, True).float().cpu()

    def only_own_pages_were_written(self):
        others = [page for page in range(self.pools[0].shape[0]) if page not in self.page_of]
        return all(bool(torch.isnan(pool[others].float()).all()) for pool in self.pools)


def differential_spec(mixer, width, eps=1e-5):
    return DifferentialAttentionSpec(hidden=width, n_heads=mixer["heads"], n_kv_heads=mixer["kv_heads"], dim=mixer["dim"], value_dim=mixer["vdim"], softmax_scale=mixer["scale"],
                                     diff=mixer["diff"], eps=eps, gate=False, qk_norm=False, bias=True, temperature=(mixer["q_temp"]["coef"], mixer["q_temp"]["every"]))


def latent_spec(mixer, width, eps=1e-5):
    return LatentAttentionSpec(hidden=width, n_heads=mixer["heads"], head_dim=mixer["dim"], rot_dim=mixer["rot_dim"], value_dim=mixer["vdim"], q_rank=None, kv_rank=mixer["kv_rank"],
                               softmax_scale=mixer["scale"], eps=eps, position=PairRotationSpec(mixer["rot_dim"], mixer["rot"]["base"]), sink=False, gate=True, gate_per_head=True,
                               window=mixer["mask"]["size"], wide_result=True)


def mixer_values(layer, width, seed):
    values = tm.weights(tm.config([layer], width=width), seed)
    return {name.replace("l0.mix", "m"): value for name, value in values.items() if ".mix." in name}


CUTTINGS = [[210], [150] + [1] * 60, [40, 2, 3, 83, 2, 64, 16], [1] * 5 + [2, 120, 1, 82]]


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("heads, kv_heads, dim, vdim, coef, every", [(4, 2, 16, 24, 0.5, 30), (1, 1, 12, 150, 1.0, 1), (9, 3, 10, 6, -0.2, 64), (4, 2, 16, 32, 0.3, 50), (2, 1, 64, 128, 0.7, 100),
                                                                     (3, 3, 48, 16, 0.2, 1000), (8, 2, 32, 64, 0.4, 7), (1, 1, 16, 320, 0.0, 5), (2, 1, 80, 48, 0.3, 20)])
def test_differential_attention_alone_in_every_cutting(dtype, heads, kv_heads, dim, vdim, coef, every):
    """Biases, the temperature of queries, both cache layouts, over scattered pages: a whole prompt, a prompt and single tokens, portions."""
    layer, width = tm.attention(heads, kv_heads, dim, vdim, diff=0.35, coef=coef, every=every), 48
    values = mixer_values(layer, width, heads * 100 + dim)
    h = torch.randn(210, width, generator=torch.Generator().manual_seed(1)).to(torch.bfloat16).float()
    wanted = plain.differential_attention(h.double(), doubled(values), "m", layer["mixer"], 1e-5)
    for cutting in CUTTINGS:
        alone = Alone(differential_spec(layer["mixer"], width), values, dtype, [6, 1, 4, 0])
        found = torch.cat([alone.run(piece) for piece in torch.split(h, cutting)])
        assert relative_error(found, wanted) < (2e-5 if dtype == "float32" else 3e-2), cutting
        assert alone.only_own_pages_were_written()


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("heads, dim, rot_dim, vdim, kv_rank, window", [(3, 24, 8, 20, 40, 37), (1, 7, 2, 9, 13, 1), (5, 16, 16, 32, 64, 100), (9, 5, 4, 11, 30, 64), (10, 48, 32, 64, 800, 150),
                                                                        (2, 128, 64, 128, 512, 65), (4, 32, 16, 48, 128, 1000), (1, 40, 24, 64, 96, 63)])
def test_latent_attention_alone_in_every_cutting(dtype, heads, dim, rot_dim, vdim, kv_rank, window):
    """Queries straight from the input, a gate per head, a window shorter and longer than pages: prompts in the expanded form (where the
    sizes allow it) and over the latents, single tokens in one range and in several."""
    layer, width = tm.latent(heads, dim, rot_dim, vdim, kv_rank, window, base=300.0), 48
    values = mixer_values(layer, width, heads * 100 + dim)
    h = torch.randn(210, width, generator=torch.Generator().manual_seed(1)).to(torch.bfloat16).float()
    wanted = plain.latent_attention(h.double(), doubled(values), "m", layer["mixer"], 1e-5)
    for index, cutting in enumerate(CUTTINGS):
        alone = Alone(latent_spec(layer["mixer"], width), values, dtype, [6, 1, 4, 0])
        found = torch.cat([alone.run(piece, splits=(0, 1, 3, 16)[index]) for piece in torch.split(h, cutting)])
        assert relative_error(found, wanted) < (2e-5 if dtype == "float32" else 3e-2), cutting
        assert alone.only_own_pages_were_written()


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("window", [33, 64, 65])
@pytest.mark.parametrize("rot_dim", [16, 6])       # the expanded form of prompts; sizes that it does not serve
def test_one_latent_key_that_stands_out_at_the_window_edge(dtype, window, rot_dim):
    """The input is the query itself and the latent is part of the input: a position whose first elements equal those of an earlier one
    scores it far above all others.  The earlier one lies on the window's last visible position or one further, also across a page border."""
    torch.manual_seed(9)
    dim, rank, width, total = 16, 24, 64, 260
    mixer = tm.latent(2, dim, rot_dim, 20, rank, window, scale=3.0)["mixer"]
    values = {"m.q": torch.zeros(2 * (dim + rot_dim), width), "m.dkv": torch.zeros(rank + rot_dim, width), "m.dkv.norm": torch.ones(rank), "m.uk": torch.zeros(2 * dim, rank),
              "m.uv": torch.randn(40, rank) / 3, "m.g": torch.zeros(2, width), "m.o": torch.eye(width, 40)}
    for head in range(2):
        values["m.q"][head * (dim + rot_dim) : head * (dim + rot_dim) + dim, :dim] = torch.eye(dim)
        values["m.uk"][head * dim : (head + 1) * dim, :dim] = torch.eye(dim)
    values["m.dkv"][:rank, :rank] = torch.eye(rank)
    values = {name: value.to(torch.bfloat16).float() for name, value in values.items()}
    h = torch.randn(total, width).to(torch.bfloat16).float()
    for query in (70, 96, 127, 128, 150, 199, 255):
        h[query, :dim] = h[query - window + 1, :dim]           # just inside: the oldest position the query sees
    for query in (80, 95, 129, 160, 192, 230):
        h[query, :dim] = h[query - window, :dim]               # just outside
    wanted = plain.latent_attention(h.double(), doubled(values), "m", mixer, 1e-5)
    tolerance = 2e-5 if dtype == "float32" else 8e-2
    for cutting in ([total], [30] + [1] * (total - 30), [64, 66, 130]):
        alone = Alone(latent_spec(mixer, width), values, dtype, [2, 0, 3, 1, 6])
        assert relative_error(torch.cat([alone.run(piece) for piece in torch.split(h, cutting)]), wanted) < tolerance
    for off in (window - 1, window + 1):                       # the test would see a window that is one off
        other = plain.latent_attention(h.double(), doubled(values), "m", {**mixer, "mask": {"size": off}}, 1e-5)
        assert relative_error(other, wanted) > 0.3


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("vdim", [24, 32])      # one row per position; ordinary heads
def test_one_differential_key_that_stands_out_far_back(monkeypatch, dtype, vdim):
    """There is no window: a key hundreds of positions back, at page borders and at the very first position, is the whole first map of
    queries that equal it; and the temperature's factor makes or breaks a score that stands out against a second one."""
    torch.manual_seed(10)
    dim, width, total = 16, 64, 420
    mixer = tm.attention(2, 1, dim, vdim, scale=2.0, diff=0.2, coef=0.3, every=50)["mixer"]
    values = {"m.q": torch.eye(2 * 2 * dim, width), "m.k": torch.zeros(2 * dim, width), "m.v": torch.randn(vdim, width) / 5, "m.o": torch.eye(width, 2 * vdim)}
    values["m.k"][:dim, :dim] = torch.eye(dim)
    values["m.k"][dim:, dim : 2 * dim] = torch.eye(dim)
    values |= {f"m.{name}.b": 0.05 * torch.randn(values[f"m.{name}"].shape[0]) for name in "qkvo"}
    values |= {f"m.{name}": torch.zeros(dim) for name in ("lq1", "lk1", "lq2", "lk2")}
    values = {name: value.to(torch.bfloat16).float() for name, value in values.items()}
    h = torch.randn(total, width).to(torch.bfloat16).float()
    for query, key in ((400, 0), (380, 63), (381, 64), (350, 1), (300, 127), (257, 128), (256, 255), (100, 0), (419, 191)):
        h[query, :dim] = h[key, :dim]
    wanted = plain.differential_attention(h.double(), doubled(values), "m", mixer, 1e-5)
    tolerance = 2e-5 if dtype == "float32" else 8e-2
    for cutting in ([total], [240] + [1] * (total - 240), [64, 66, 2, 130, 158]):
        alone = Alone(differential_spec(mixer, width), values, dtype, [2, 0, 3, 1, 6, 7, 5])
        assert relative_error(torch.cat([alone.run(piece) for piece in torch.split(h, cutting)]), wanted) < tolerance
    cold = plain.differential_attention(h.double(), doubled(values), "m", {**mixer, "q_temp": {"coef": 0.0, "every": 50}}, 1e-5)
    assert relative_error(cold, wanted) > 0.2
    monkeypatch.setattr(plain, "visible", lambda tokens, window=None, real=plain.visible: real(tokens, 300))      # the far keys forgotten
    assert relative_error(plain.differential_attention(h.double(), doubled(values), "m", mixer, 1e-5), wanted) > 0.3


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("rows, batch, features, depth", [(1, 3, 40, 24), (8, 16, 512, 128), (9, 2, 70, 512), (16, 1, 1, 8), (17, 5, 33, 64), (3, 4, 50, 22), (2, 2, 9, 2048)])
def test_the_batched_product_of_few_rows(dtype, rows, batch, features, depth):
    """Views whose rows and batches lie further apart than they are long; sizes that whole 16-byte pieces serve and others."""
    from tau_rs_b200.csrc import kernels

    torch.manual_seed(rows)
    values, weight = torch.randn(rows, batch, depth + 8), torch.randn(batch, features, depth)
    for out_dtype in {dtype, "float32"}:
        out = torch.full((rows, batch, features + 3), float("nan"), dtype=TORCH[out_dtype], device=DEVICE)
        kernels.gemm_simt_batched(on_device(values, TORCH[dtype])[:, :, :depth], on_device(weight, TORCH[dtype]), out[:, :, :features])
        wanted = torch.einsum("mbk,bnk->mbn", values[:, :, :depth].to(TORCH[dtype]).double(), weight.to(TORCH[dtype]).double())
        assert relative_error(out[:, :, :features].float().cpu(), wanted) < (2e-6 if out_dtype == "float32" else 5e-3)
        assert torch.isnan(out[:, :, features:].float()).all()


# ---- whole models: cuttings, batches, reuse ----------------------------------------------------------------------------
@pytest.mark.parametrize("name", ["mixed", "odd", "wide"])
def test_the_stream_behind_every_run(models, name):
    """In 32-bit: what every run of a layer (each pass of the loop counts) leaves on the stream, against the plain statement."""
    engine, cfg, values = engine_of(models, name, "float32")
    tokens = tokens_for(cfg, 150, 20)
    seen = []
    for block in engine.model.blocks:
        def watched(residual, branch, *rest, forward=block.forward):
            residual, left = forward(residual, branch, *rest)
            seen.append((residual + left.channel_scale * sum(left)).cpu())
            return residual, left
        block.forward = watched
    run_whole(engine, tokens)
    _, wanted = plain.forward(tokens, doubled(values), cfg, return_layers=True)
    assert len(seen) == len(wanted) == len(plain.runs(cfg))
    for found, layer in zip(seen, wanted):
        assert relative_error(found, layer) < 1e-5


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("name", ["mixed", "odd", "wide"])
def test_whole_prompts_single_tokens_and_the_first_positions(models, name, dtype):
    engine, cfg, values = engine_of(models, name, dtype)
    tokens = tokens_for(cfg, 200, 21)
    wanted = plain_logits(cfg, values, tokens)
    whole = run_whole(engine, tokens)
    assert close(whole, wanted, dtype)
    if dtype == "float32":
        assert close(whole[:4], wanted[:4], dtype) and close(run_whole(engine, tokens[:1]), wanted[:1], dtype)
    stepwise = run_tail_stepwise(engine, tokens, 199)                              # every token but the first alone, through the graphs
    assert close(stepwise, wanted[1:], dtype)
    if dtype == "float32":
        assert relative_error(stepwise, whole[1:]) < 2e-5


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("name", ["mixed", "odd"])
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
    assert position == 330
    engine.close_sequence(slot)
    assert close(torch.cat(found), wanted, dtype)


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("name", ["peaky", "edgy"])
def test_a_sharp_softmax_loses_no_key_far_back_at_a_page_border_or_at_the_window_edge(models, name, dtype):
    engine, cfg, values = engine_of(models, name, dtype)
    tokens = tokens_for(cfg, 400, 23)
    wanted = plain_logits(cfg, values, tokens)
    assert close(run_whole(engine, tokens), wanted, dtype)
    assert close(run_tail_stepwise(engine, tokens, 150), wanted[-150:], dtype)     # decoded queries cross the borders at 256 and 320
    slot = engine.open_sequence()                                                  # portions whose windows reach into earlier portions
    found = [engine.step([StepEntry(slot, tokens[begin : begin + 50], list(range(50)))]).float().cpu().clone() for begin in range(0, 400, 50)]
    engine.close_sequence(slot)
    assert close(torch.cat(found), wanted, dtype)


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("name", ["mixed", "odd", "edgy"])
def test_unequal_batches_against_each_request_alone(models, name, dtype):
    engine, cfg, values = engine_of(models, name, dtype, 2048)
    lengths, prompts = [90, 31, 140, 5, 66], [70, 1, 129, 3, 64]
    requests = [tokens_for(cfg, length, 30 + index) for index, length in enumerate(lengths)]
    together = run_batched(engine, requests, prompts)
    found = torch.cat(together)
    wanted = torch.cat([plain_logits(cfg, values, request)[prompt - 1 :] for request, prompt in zip(requests, prompts)])
    assert close(found, wanted, dtype)
    engine.cache.check()
    assert engine.cache.slots.in_use == 0


def test_a_step_that_mixes_prompts_portions_and_single_tokens(models):
    """One batch in which a request starts, one goes on by a portion and one by a single token."""
    engine, cfg, values = engine_of(models, "mixed", "float32", 2048)
    a, b, c = (tokens_for(cfg, count, 50 + count) for count in (150, 90, 140))
    slots = [engine.open_sequence() for _ in range(3)]
    engine.step([StepEntry(slots[0], a[:130], []), StepEntry(slots[1], b[:40], [])])
    found = engine.step([StepEntry(slots[2], c, list(range(140))), StepEntry(slots[0], a[130:149], list(range(19))), StepEntry(slots[1], b[40:41], [0])]).cpu().clone()
    wanted = torch.cat([plain_logits(cfg, values, c), plain_logits(cfg, values, a)[130:149], plain_logits(cfg, values, b)[40:41]])
    assert close(found, wanted, "float32")
    for slot in slots:
        engine.close_sequence(slot)


def test_slots_and_pages_that_are_used_again_start_clean(models):
    """A cache of three pages and as many slots: every request takes pages that another wrote."""
    engine, cfg, values = engine_of(models, "mixed", "float32", 64 * 3)
    for round_number in range(4):
        requests = [tokens_for(cfg, length, 40 + 3 * round_number + index) for index, length in enumerate([60 + round_number, 40, 17])]
        together = run_batched(engine, requests, [len(request) - 6 for request in requests])
        for request, rows in zip(requests, together):
            assert close(rows, plain_logits(cfg, values, request)[len(request) - 7 :], "float32")
        engine.cache.check()


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_a_long_sequence_in_a_cache_of_four_pages(models, dtype):
    """600 tokens through a cache that holds 256 positions: every layer has a window, so pages that fall out of it are given back
    and taken again; in runs and single tokens against the plain statement of the whole sequence."""
    engine, cfg, values = engine_of(models, "edgy", dtype, 64 * 4)
    tokens = tokens_for(cfg, 600, 25)
    wanted = plain_logits(cfg, values, tokens)
    slot = engine.open_sequence()
    found, position = [], 0
    for count in [50, 1, 1, 64, 30, 1, 1, 1, 50, 50, 50, 64, 1, 50, 50, 50, 36] + [1] * 50:
        piece = tokens[position : position + count]
        found.append(engine.step([StepEntry(slot, piece, list(range(len(piece))))]).float().cpu().clone())
        position += len(piece)
        engine.cache.check()
        assert all(len(group.held[slot]) <= 3 for group in engine.cache.kv.values())
    assert position == 600
    engine.close_sequence(slot)
    assert close(torch.cat(found), wanted, dtype)


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
    compared = 0
    for prompt, result in zip(prompts, output):
        tokens = list(prompt)
        for _ in range(12):
            logits = plain_logits(cfg, values, tokens)[-1]
            best, second = torch.topk(logits, 2).values
            if float(best - second) < 1e-3 * float(logits.abs().max()):
                break                                                                # a close call proves nothing either way
            tokens.append(int(torch.argmax(logits)))
        made = len(tokens) - len(prompt)
        assert list(result.tokens[:made]) == tokens[len(prompt) :]
        compared += made
    assert compared >= 12


def test_trace_replay_of_a_tukulorn_folder(models, tmp_path):
    folder, cfg, values = models["odd"]
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
    assert close(torch.from_numpy(rows), torch.stack([wanted_a[0], wanted_a[65], wanted_b[29]]), "float32")
    rows = np.fromfile(out / "3.f32", dtype="<f4").reshape(2, cfg["vocab"])
    assert close(torch.from_numpy(rows), torch.stack([wanted_a[68], wanted_b[32]]), "float32")
    assert not (out / "4.f32").exists()


def test_the_command_line_on_a_tukulorn_folder(models, tmp_path):
    """`bin/tau` on a Tukulorn folder: greedy tokens in 32-bit equal those of `generate()`, with graphs and without, in chunks of
    prompt tokens; bfloat16 runs from the same folder; random weights are written for a Tukulorn config.json and read back."""
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
    config_path.write_text(json.dumps(tm.PEAKY))
    drawn = str(tmp_path / "drawn")
    records = run(["--random-weights", str(config_path), "--model", drawn, "--seed", "4", "--max-tokens", "5", "--stop-ids", "", "--prompt-ids", "1,2,3"])
    assert [len(record["tokens"]) for record in records if "tokens" in record] == [5]
