"""Small Bikovik configurations and weights for the tests, made here from the config alone (names, shapes and scales are written out by
hand; nothing is taken from the library's own list of tensors)."""
from __future__ import annotations

import json
import os
from typing import Dict

import torch

from tau_rs_b200.weights.safetensors_io import write_safetensors


def dense(ff=72, limit=1.2):
    return {"kind": "dense", "ff": ff, "limit": limit}


def _entry(kind, mixer, mlp):
    return {"type": kind, "mixer": mixer, "mlp": dense() if mlp == "default" else mlp}


def attention(heads=4, kv_heads=2, dim=16, vdim=24, size=40, keep_first=5, rot_dims=8, base=5000.0, scale=None, v_mix=True, mlp="default"):
    mixer = {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "mask": {"size": size, "keep_first": keep_first},
             "rot": {"base": base, "dims": rot_dims}, "scale": dim ** -0.5 if scale is None else scale, "v_mix": v_mix}
    return _entry("attention", mixer, mlp)


def hgrn2(heads=3, dim=16, vdim=24, mlp="default"):
    return _entry("hgrn2", {"heads": heads, "dim": dim, "vdim": vdim}, mlp)


def retention(heads=3, dim=16, vdim=24, decay=None, rot_dims=8, base=3000.0, mlp="default"):
    decay = [1.0 - 2.0 ** (-2 - 1.3 * head) for head in range(heads)] if decay is None else decay
    return _entry("retention", {"heads": heads, "dim": dim, "vdim": vdim, "decay": decay, "rot": {"base": base, "dims": rot_dims}}, mlp)


def config(layers, width=96, vocab=211, eps=1e-5, scale=1.7, cap=4.0) -> dict:
    return {"architecture": "Bikovik", "embedding": {"scale": scale}, "layers": layers, "logit_softcap": cap, "norm": {"eps": eps}, "vocab": vocab, "width": width}


# Every mixer, every feed-forward and none; layers of a kind with different sizes, windows and kept positions; values mixed in three layers
# of which the first is not the first attention, one attention between them that does not mix.
MIXED = config([attention(v_mix=False, size=70, keep_first=9),
                hgrn2(),
                attention(),
                retention(),
                attention(heads=6, kv_heads=3, dim=8, vdim=16, size=65, keep_first=64, rot_dims=8, mlp=dense(40, 0.7)),
                retention(heads=2, dim=24, vdim=8, rot_dims=24, mlp=None),
                attention(heads=2, kv_heads=1, dim=32, vdim=40, size=17, keep_first=70, v_mix=False, mlp=None),
                hgrn2(heads=2, dim=24, vdim=8, mlp=None),
                attention(heads=4, kv_heads=1, dim=8, vdim=48, size=130, keep_first=1, mlp=dense(40, 3.0))])
# Sizes that happen to be 1 or equal elsewhere, and nothing a multiple of 8: one head, a window of one, no kept position, rotations of the
# whole head and of two elements, values wider than a warp's pass, decays of one and almost nothing, an embedding scale and limits of 1.
ODD = config([attention(heads=1, kv_heads=1, dim=12, vdim=150, size=1, keep_first=0, rot_dims=12, mlp=dense(30, 1.0)),
              hgrn2(heads=1, dim=20, vdim=70, mlp=dense(14, 0.3)),
              retention(heads=1, dim=10, vdim=34, decay=[1.0], rot_dims=2, mlp=dense(22, 2.0)),
              attention(heads=9, kv_heads=3, dim=10, vdim=50, size=37, keep_first=3, rot_dims=2, mlp=None),
              retention(heads=5, dim=6, vdim=13, decay=[0.05, 0.5, 0.9, 0.99, 1.0], rot_dims=6, mlp=None),
              hgrn2(heads=5, dim=6, vdim=5, mlp=None),
              attention(heads=3, kv_heads=3, dim=7, vdim=50, size=100, keep_first=1, rot_dims=6, mlp=dense(6, 1.0)),
              hgrn2(heads=2, dim=100, vdim=10, mlp=None)],
             width=100, vocab=77, eps=1e-6, scale=1.0, cap=30.0)
# Attention with sharp weights, so that single keys carry a query's result: a key at a window's edge or among the first ones that is lost or
# seen too long moves the logits by much more than rounding does.
PEAKY = config([attention(heads=3, kv_heads=1, dim=16, vdim=24, size=64, keep_first=3, scale=2.0, mlp=None),
                attention(heads=2, kv_heads=2, dim=16, vdim=12, size=100, keep_first=65, rot_dims=16, scale=2.0, mlp=None)], width=64, vocab=97, scale=1.3, cap=8.0)
# The same with keys and values as wide as ordinary heads (64 and 128), which the library keeps in another cache layout and serves on the
# tensor cores: several key heads side by side, one, and as many as heads.
HEADY = config([attention(heads=4, kv_heads=2, dim=64, vdim=64, size=90, keep_first=20, rot_dims=64, scale=0.4, mlp=None),
                attention(heads=4, kv_heads=1, dim=128, vdim=128, size=64, keep_first=1, rot_dims=64, scale=0.2, mlp=None),
                attention(heads=3, kv_heads=3, dim=128, vdim=128, size=200, keep_first=130, rot_dims=32, scale=0.2, v_mix=False, mlp=None)], width=64, vocab=97, scale=1.3)
# More key heads than the tensor-core kernel's query tile holds pieces for, and more value columns than the single-token kernel owns.
WIDE = config([attention(heads=8, kv_heads=8, dim=128, vdim=128, size=70, keep_first=10, rot_dims=128, mlp=None),
               attention(heads=48, kv_heads=2, dim=16, vdim=200, size=33, keep_first=2, rot_dims=8, v_mix=False, mlp=None)], width=64, vocab=97)
# States that forget slowly, so that one lost or restarted shows hundreds of tokens later.
LONG_MEMORY = config([hgrn2(heads=2, dim=32, vdim=16, mlp=None), retention(heads=4, dim=32, vdim=32, decay=[0.995, 0.999, 1.0, 0.998], rot_dims=32, base=1e6, mlp=None)],
                     width=64, vocab=53)
# One mechanism to a model.
ONLY = {
    "attention": config([attention(mlp=None)], width=64, vocab=61),
    "mixed_values": config([attention(mlp=None), attention(heads=3, kv_heads=3, dim=8, vdim=16, mlp=None)], width=64, vocab=61),
    "hgrn2": config([hgrn2(mlp=None)], width=64, vocab=61),
    "retention": config([retention(mlp=None)], width=64, vocab=61),
    "dense": config([hgrn2(heads=1, dim=8, vdim=8)], width=64, vocab=61),
}


def weights(cfg: dict, seed: int, slow_forgetting: bool = False) -> Dict[str, torch.Tensor]:
    """Random weights of the scales that keep every branch alive (gates and up values on both sides of the limits, logits inside the soft
    cap's bend), every value one that bfloat16 holds.  `slow_forgetting`: the forget gates stay close to one."""
    generator = torch.Generator().manual_seed(seed)
    width = cfg["width"]
    out: Dict[str, torch.Tensor] = {}

    def matrix(name, rows, columns, gain=1.0):
        out[name] = torch.randn(rows, columns, generator=generator) * gain / columns ** 0.5

    def vector(name, count, mean, spread):
        out[name] = mean + spread * torch.randn(count, generator=generator)

    def norm(name):
        vector(name, width, 1.0, 0.2)
        vector(f"{name}.b", width, 0.0, 0.2)
        out[f"{name}.alpha"] = 0.4 + 0.4 * torch.rand((), generator=generator)

    out["embed"] = torch.randn(cfg["vocab"], width, generator=generator)
    matrix("head", cfg["vocab"], width, 4.0)
    norm("final.norm")
    for index, layer in enumerate(cfg["layers"]):
        p, mixer, mlp = f"l{index}", layer["mixer"], layer["mlp"]
        heads, dim, vdim = mixer["heads"], mixer["dim"], mixer["vdim"]
        norm(f"{p}.norm1")
        if layer["type"] == "attention":
            kv_heads = mixer["kv_heads"]
            for name, rows in (("q", heads * dim), ("k", kv_heads * dim), ("v", kv_heads * vdim)):
                matrix(f"{p}.mix.{name}", rows, width, 1.3)
                vector(f"{p}.mix.{name}.b", rows, 0.0, 0.3)
            out[f"{p}.mix.talk"] = torch.eye(heads) + 0.4 * torch.randn(heads, heads, generator=generator) / heads ** 0.5
            if mixer["v_mix"]:
                out[f"{p}.mix.vmix"] = 0.3 + 0.3 * torch.rand((), generator=generator)
        elif layer["type"] == "hgrn2":
            matrix(f"{p}.mix.q", heads * dim, width, 2.0)
            matrix(f"{p}.mix.f", heads * dim, width, 2.0)
            vector(f"{p}.mix.f.b", heads * dim, 5.0 if slow_forgetting else 1.0, 1.0)
            out[f"{p}.mix.lower"] = 0.9 * torch.rand(heads * dim, generator=generator)
            matrix(f"{p}.mix.v", heads * vdim, width, 2.0)
            vector(f"{p}.mix.norm", vdim, 1.0, 0.2)
        else:
            for name, rows in (("q", heads * dim), ("k", heads * dim), ("v", heads * vdim), ("g", heads * vdim)):
                matrix(f"{p}.mix.{name}", rows, width, 2.0)
        matrix(f"{p}.mix.o", width, heads * vdim, 0.7)
        if mlp is not None:
            norm(f"{p}.norm2")
            matrix(f"{p}.mlp.gate", mlp["ff"], width, 2.0)
            matrix(f"{p}.mlp.up", mlp["ff"], width, 2.0)
            matrix(f"{p}.mlp.down", width, mlp["ff"])
    return {name: value.to(torch.bfloat16).float() for name, value in out.items()}


def write_model(folder: str, cfg: dict, seed: int, storage=torch.bfloat16, values=None, slow_forgetting: bool = False) -> Dict[str, torch.Tensor]:
    os.makedirs(folder, exist_ok=True)
    values = weights(cfg, seed, slow_forgetting) if values is None else values
    write_safetensors(os.path.join(folder, "model.safetensors"), ((name, value.to(storage)) for name, value in values.items()))
    with open(os.path.join(folder, "config.json"), "w") as handle:
        json.dump(cfg, handle)
    return values
