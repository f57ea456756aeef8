"""Small Tukulorn configurations and weights for the tests, made here from the config alone (names, shapes and scales are written
out by hand; nothing is taken from the library's own list of tensors)."""
from __future__ import annotations

import json
import os
from typing import Dict

import torch

from tau_rs_b200.weights.safetensors_io import write_safetensors


def dense(ff=72):
    return {"kind": "dense", "ff": ff}


def moe(experts=12, top=3, count=4, keep=2, ff=40, limit=0.8, scale=1.7):
    return {"kind": "moe", "router": {"experts": experts, "top": top, "groups": {"count": count, "keep": keep}, "scale": scale}, "expert": {"ff": ff, "limit": limit}}


def attention(heads=4, kv_heads=2, dim=16, vdim=24, scale=None, diff=0.3, coef=0.4, every=30, mlp="default"):
    return {"type": "attention",
            "mixer": {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "diff": diff, "scale": dim ** -0.5 if scale is None else scale,
                      "q_temp": {"coef": coef, "every": every}},
            "mlp": dense() if mlp == "default" else mlp}


def latent(heads=3, dim=24, rot_dim=8, vdim=20, kv_rank=40, window=37, base=5000.0, scale=None, mlp="default"):
    return {"type": "latent_attention",
            "mixer": {"heads": heads, "dim": dim, "rot_dim": rot_dim, "vdim": vdim, "kv_rank": kv_rank, "mask": {"size": window},
                      "rot": {"base": base, "dims": rot_dim}, "scale": (dim + rot_dim) ** -0.5 if scale is None else scale},
            "mlp": moe() if mlp == "default" else mlp}


def config(layers, width=96, vocab=211, eps=1e-5, loop=(0, 0, 1)) -> dict:
    return {"architecture": "Tukulorn", "layers": layers, "loop": None if loop is None else dict(zip(("start", "stop", "times"), loop)), "norm": {"eps": eps},
            "vocab": vocab, "width": width}


# Both mixers (the attention in both cache layouts) with both feed-forwards and none, windows shorter and longer than a page; the middle
# layers run three times.
MIXED = config([latent(), attention(mlp=moe(experts=6, top=2, count=3, keep=2, ff=24)), latent(heads=5, dim=16, rot_dim=16, vdim=32, kv_rank=64, window=100, mlp=dense(80)),
                attention(heads=6, kv_heads=3, dim=32, vdim=48, diff=0.6, coef=-0.2, every=7, mlp=None), latent(heads=2, dim=10, rot_dim=6, vdim=14, kv_rank=22, window=64, mlp=None)],
               loop=(1, 4, 3))
# Sizes that happen to be 1 or equal elsewhere, and nothing a multiple of 8: one head, a window of one position, one expert of one, groups
# of one expert, all groups kept, all experts chosen, a temperature that steps at every position, a loop that starts at the first layer.
ODD = config([latent(heads=1, dim=7, rot_dim=2, vdim=9, kv_rank=13, window=1, mlp=moe(experts=1, top=1, count=1, keep=1, ff=20, limit=7.0, scale=1.0)),
              attention(heads=1, kv_heads=1, dim=12, vdim=150, every=1, mlp=moe(experts=5, top=2, count=5, keep=3, ff=12, limit=0.3)),
              latent(heads=9, dim=5, rot_dim=4, vdim=11, kv_rank=30, window=1000, mlp=moe(experts=6, top=6, count=2, keep=2, ff=10, scale=0.5)),
              attention(heads=9, kv_heads=3, dim=10, vdim=6, diff=0.8, mlp=dense(ff=30))], width=100, vocab=77, eps=1e-6, loop=(0, 2, 2))
# No loop at all; wide latents, wide values, many experts and groups.
WIDE = config([latent(heads=10, dim=48, rot_dim=32, vdim=64, kv_rank=800, window=150, mlp=moe(experts=64, top=6, count=8, keep=3, ff=32)),
               attention(heads=2, kv_heads=1, dim=24, vdim=320, mlp=moe(experts=40, top=1, count=40, keep=4, ff=16)),
               attention(heads=4, kv_heads=2, dim=64, vdim=128, mlp=dense(96))], width=128, vocab=97, loop=None)
# Attention with a sharp softmax, so that single keys carry a query's weight: a key lost far back, at a page border or at the window's
# edge, or one seen beyond it, moves the logits by much more than rounding does.
PEAKY = config([attention(heads=3, kv_heads=1, dim=16, vdim=24, scale=0.9, coef=0.1, every=100, mlp=None), attention(heads=2, kv_heads=1, dim=16, vdim=32, scale=0.8, mlp=None)],
               width=64, vocab=97, loop=(0, 1, 2))
EDGY = config([latent(heads=4, dim=16, rot_dim=16, vdim=16, kv_rank=32, window=33, scale=1.2, mlp=None),
               latent(heads=2, dim=12, rot_dim=4, vdim=20, kv_rank=18, window=64, scale=1.0, mlp=None)], width=64, vocab=97, loop=(1, 2, 2))


def weights(cfg: dict, seed: int) -> Dict[str, torch.Tensor]:
    """Random weights of the scales that keep every branch alive, every value one that bfloat16 holds."""
    generator = torch.Generator().manual_seed(seed)
    width = cfg["width"]
    out: Dict[str, torch.Tensor] = {}

    def matrix(name, rows, columns, gain=1.0):
        out[name] = torch.randn(rows, columns, generator=generator) * gain / columns ** 0.5

    def vector(name, count, mean, spread):
        out[name] = mean + spread * torch.randn(count, generator=generator)

    out["embed"] = torch.randn(cfg["vocab"], width, generator=generator)
    matrix("head", cfg["vocab"], width)
    vector("final.norm", width, -0.1, 0.3)
    for index, layer in enumerate(cfg["layers"]):
        p, mixer, mlp = f"l{index}", layer["mixer"], layer["mlp"]
        for number in ("1", "2")[: 1 if mlp is None else 2]:
            vector(f"{p}.norm{number}", width, 0.0, 0.3)
            vector(f"{p}.ls{number}", width, 0.7, 0.3)
        heads, vdim, dim = mixer["heads"], mixer["vdim"], mixer["dim"]
        if layer["type"] == "attention":
            kv_heads = mixer["kv_heads"]
            for name, rows in (("q", heads * 2 * dim), ("k", kv_heads * 2 * dim), ("v", kv_heads * vdim), ("o", width)):
                matrix(f"{p}.mix.{name}", rows, width if name != "o" else heads * vdim)
                vector(f"{p}.mix.{name}.b", rows, 0.0, 0.3)
            for name in ("lq1", "lk1", "lq2", "lk2"):
                vector(f"{p}.mix.{name}", dim, 0.0, 0.25)
        else:
            rot, rank = mixer["rot_dim"], mixer["kv_rank"]
            matrix(f"{p}.mix.q", heads * (dim + rot), width)
            matrix(f"{p}.mix.dkv", rank + rot, width)
            vector(f"{p}.mix.dkv.norm", rank, 1.0, 0.2)
            matrix(f"{p}.mix.uk", heads * dim, rank)
            matrix(f"{p}.mix.uv", heads * vdim, rank)
            matrix(f"{p}.mix.g", heads, width, 1.5)
            matrix(f"{p}.mix.o", width, heads * vdim, 1.5)
        if mlp is not None and mlp["kind"] == "dense":
            matrix(f"{p}.mlp.gate", mlp["ff"], width)
            matrix(f"{p}.mlp.up", mlp["ff"], width)
            matrix(f"{p}.mlp.down", width, mlp["ff"], 1.5)
        elif mlp is not None:
            matrix(f"{p}.mlp.router", mlp["router"]["experts"], width, 1.5)
            for expert in range(mlp["router"]["experts"]):
                matrix(f"{p}.mlp.e{expert}.gate", mlp["expert"]["ff"], width)
                matrix(f"{p}.mlp.e{expert}.up", mlp["expert"]["ff"], width)
                matrix(f"{p}.mlp.e{expert}.down", width, mlp["expert"]["ff"])
    return {name: value.to(torch.bfloat16).float() for name, value in out.items()}


def write_model(folder: str, cfg: dict, seed: int, storage=torch.bfloat16, values=None) -> Dict[str, torch.Tensor]:
    os.makedirs(folder, exist_ok=True)
    values = weights(cfg, seed) if values is None else values
    write_safetensors(os.path.join(folder, "model.safetensors"), ((name, value.to(storage)) for name, value in values.items()))
    with open(os.path.join(folder, "config.json"), "w") as handle:
        json.dump(cfg, handle)
    return values
