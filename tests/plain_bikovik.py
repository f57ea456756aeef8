"""Bikovik stated plainly: one function per mechanism, float64, whole sequences, masks instead of caches, loops over tokens instead of
carried state.

Shares nothing with the library.  `weights` maps tensor names to float64 tensors, `config` is the dictionary that a folder's
config.json holds.  Every function takes one sequence `[tokens, ...]` whose first row is position 0.
"""
from __future__ import annotations

import math

import torch

F = torch.float64


def unit_rms(x, eps):
    return x / torch.sqrt((x * x).mean(-1, keepdim=True) + eps)


def silu(z):
    return z * torch.sigmoid(z)


def dynamic_tanh(x, alpha, weight, bias):
    """No statistic of the row: every element passes tanh(alpha x) on its own."""
    return torch.tanh(alpha * x) * weight + bias


def rotate_halves(x, rot):
    """x [tokens, heads, dim]: element i of the first `dims` is paired with element i + dims / 2; the rest pass."""
    dims, base = rot["dims"], rot["base"]
    half = dims // 2
    frequency = torch.tensor([base ** (-2.0 * i / dims) for i in range(half)], dtype=F)
    angle = torch.arange(x.shape[0], dtype=F)[:, None] * frequency[None, :]
    cos, sin = torch.cos(angle)[:, None, :], torch.sin(angle)[:, None, :]
    a, b = x[..., :half], x[..., half:dims]
    return torch.cat([a * cos - b * sin, b * cos + a * sin, x[..., dims:]], dim=-1)


def visible_keys(tokens, size, keep_first):
    """[query, key]: the last `size` positions up to the query's own, and the sequence's first `keep_first`."""
    place = torch.arange(tokens)
    distance = place[:, None] - place[None, :]
    return (distance >= 0) & ((distance < size) | (place[None, :] < keep_first))


def talking_attention(q, k, v, scale, talk, visible):
    """q [tokens, heads, dim], k [tokens, kv_heads, dim], v [tokens, kv_heads, vdim]: every head's scores are a mix of all heads' scores,
    `sum_g talk[h, g] score_g`; then an ordinary softmax over the visible keys."""
    tokens, heads, _ = q.shape
    per = heads // k.shape[1]
    raw = torch.stack([q[:, head] @ k[:, head // per].T * scale for head in range(heads)])
    mixed = torch.einsum("hg,gij->hij", talk, raw)
    mixed = torch.where(visible[None], mixed, torch.full((), -math.inf, dtype=F))
    weight = torch.softmax(mixed, dim=-1)
    return torch.stack([weight[head] @ v[:, head // per] for head in range(heads)], dim=1)


def mixed_values(v, first, share):
    return v if first is None else (1.0 - share) * v + share * first


def attention_mixer(h, weights, prefix, mixer, first):
    """Returns (output, the values before mixing); `first` holds the values of the first layer that mixes, None in that layer itself."""
    tokens = h.shape[0]
    heads, kv_heads, dim, vdim = mixer["heads"], mixer["kv_heads"], mixer["dim"], mixer["vdim"]
    q, k, v = (h @ weights[f"{prefix}.{name}"].T + weights[f"{prefix}.{name}.b"] for name in ("q", "k", "v"))
    q = rotate_halves(q.reshape(tokens, heads, dim), mixer["rot"])
    k = rotate_halves(k.reshape(tokens, kv_heads, dim), mixer["rot"])
    mixed = mixed_values(v, first, weights[f"{prefix}.vmix"]) if mixer.get("v_mix") else v
    visible = visible_keys(tokens, mixer["mask"]["size"], mixer["mask"]["keep_first"])
    out = talking_attention(q, k, mixed.reshape(tokens, kv_heads, vdim), mixer["scale"], weights[f"{prefix}.talk"], visible)
    return out.reshape(tokens, heads * vdim) @ weights[f"{prefix}.o"].T, v


def forget_write_recurrence(q, f, v):
    """q, f [tokens, heads, dim], v [tokens, heads, vdim]: what a channel forgets is what it writes; the read-out sees the token itself."""
    tokens, heads, dim = q.shape
    state = torch.zeros(heads, dim, v.shape[-1], dtype=F)
    out = torch.zeros_like(v)
    for t in range(tokens):
        state = f[t][:, :, None] * state + (1.0 - f[t])[:, :, None] * v[t][:, None, :]
        out[t] = torch.einsum("hdv,hd->hv", state, q[t])
    return out


def forget_gate(pre, lower):
    return lower + (1.0 - lower) * torch.sigmoid(pre)


def hgrn2_mixer(h, weights, prefix, mixer, eps):
    tokens = h.shape[0]
    heads, dim, vdim = mixer["heads"], mixer["dim"], mixer["vdim"]
    q = silu(h @ weights[f"{prefix}.q"].T).reshape(tokens, heads, dim)
    f = forget_gate(h @ weights[f"{prefix}.f"].T + weights[f"{prefix}.f.b"], weights[f"{prefix}.lower"]).reshape(tokens, heads, dim)
    v = (h @ weights[f"{prefix}.v"].T).reshape(tokens, heads, vdim)
    out = unit_rms(forget_write_recurrence(q, f, v), eps) * weights[f"{prefix}.norm"]
    return out.reshape(tokens, heads * vdim) @ weights[f"{prefix}.o"].T


def decay_recurrence(q, k, v, decay):
    """q, k [tokens, heads, dim], v [tokens, heads, vdim], decay [heads]."""
    tokens, heads, dim = q.shape
    state = torch.zeros(heads, dim, v.shape[-1], dtype=F)
    out = torch.zeros_like(v)
    for t in range(tokens):
        state = decay[:, None, None] * state + k[t][:, :, None] * v[t][:, None, :]
        out[t] = torch.einsum("hdv,hd->hv", state, q[t])
    return out


def retention_mixer(h, weights, prefix, mixer, eps):
    tokens = h.shape[0]
    heads, dim, vdim = mixer["heads"], mixer["dim"], mixer["vdim"]
    q, k = (rotate_halves((h @ weights[f"{prefix}.{name}"].T).reshape(tokens, heads, dim), mixer["rot"]) for name in ("q", "k"))
    v = (h @ weights[f"{prefix}.v"].T).reshape(tokens, heads, vdim)
    read = decay_recurrence(q, k * dim ** -0.5, v, torch.tensor(mixer["decay"], dtype=F))
    gate = silu(h @ weights[f"{prefix}.g"].T)
    return (unit_rms(read, eps).reshape(tokens, heads * vdim) * gate) @ weights[f"{prefix}.o"].T


def clamped_activation(gate, up, limit):
    gate = torch.clamp(gate, max=limit)
    up = torch.clamp(up, min=-limit, max=limit)
    return gate * torch.sigmoid(1.702 * gate) * (up + 1.0)


def clamped_feed_forward(h, weights, prefix, limit):
    return clamped_activation(h @ weights[f"{prefix}.gate"].T, h @ weights[f"{prefix}.up"].T, limit) @ weights[f"{prefix}.down"].T


def soft_cap(logits, cap):
    return cap * torch.tanh(logits / cap)


def norm(x, weights, name):
    return dynamic_tanh(x, weights[f"{name}.alpha"], weights[name], weights[f"{name}.b"])


def forward(tokens, weights, config, return_layers=False):
    """Logits [tokens, vocab] of one sequence (and, if asked, the residual stream after every layer)."""
    eps = config["norm"]["eps"]
    x = weights["embed"][torch.as_tensor(tokens, dtype=torch.long)] * config["embedding"]["scale"]
    first, streams = None, []
    for index, layer in enumerate(config["layers"]):
        prefix, mixer = f"l{index}", layer["mixer"]
        h = norm(x, weights, f"{prefix}.norm1")
        if layer["type"] == "attention":
            mixed, own = attention_mixer(h, weights, f"{prefix}.mix", mixer, first)
            if mixer.get("v_mix") and first is None:
                first = own
        elif layer["type"] == "hgrn2":
            mixed = hgrn2_mixer(h, weights, f"{prefix}.mix", mixer, eps)
        elif layer["type"] == "retention":
            mixed = retention_mixer(h, weights, f"{prefix}.mix", mixer, eps)
        else:
            raise ValueError(layer["type"])
        x = x + mixed
        mlp = layer.get("mlp")
        if mlp is not None:
            x = x + clamped_feed_forward(norm(x, weights, f"{prefix}.norm2"), weights, f"{prefix}.mlp", mlp["limit"])
        streams.append(x)
    logits = soft_cap(norm(x, weights, "final.norm") @ weights["head"].T, config["logit_softcap"])
    return (logits, torch.stack(streams)) if return_layers else logits
