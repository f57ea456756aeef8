"""Tukulorn stated plainly: one function per mechanism, float64, whole sequences, masks instead of caches.

Shares nothing with the library.  `weights` maps tensor names to float64 tensors, `config` is the dictionary that a
folder's config.json holds.  Every function takes one sequence `[tokens, ...]` whose first row is position 0.
"""
from __future__ import annotations

import math

import torch

F = torch.float64


def unit_rms(x, eps):
    return x / torch.sqrt((x * x).mean(-1, keepdim=True) + eps)


def zero_centred_norm(x, weight, eps):
    return unit_rms(x, eps) * (1.0 + weight)


def sigmoid(z):
    return 1.0 / (1.0 + torch.exp(-z))


def rotate_pairs(x, rotary_dim, base):
    """`x` [tokens, ..., dim]: elements (2i, 2i+1) of the first `rotary_dim` turn by `position * base^(-2i / rotary_dim)`."""
    out = x.clone()
    positions = torch.arange(x.shape[0], dtype=F).view(-1, *([1] * (x.dim() - 2)))
    for i in range(rotary_dim // 2):
        angle = positions * base ** (-2.0 * i / rotary_dim)
        u, v = x[..., 2 * i], x[..., 2 * i + 1]
        out[..., 2 * i] = u * torch.cos(angle) - v * torch.sin(angle)
        out[..., 2 * i + 1] = v * torch.cos(angle) + u * torch.sin(angle)
    return out


def query_temperature(tokens, coef, every):
    """The factor of the query at each position."""
    return torch.tensor([1.0 + coef * math.log((p + 1) // every + 1) for p in range(tokens)], dtype=F)


def visible(tokens, window=None):
    """[i, j]: whether the token at position i sees the one at j."""
    distance = torch.arange(tokens).view(-1, 1) - torch.arange(tokens).view(1, -1)
    return (distance >= 0) if window is None else (distance >= 0) & (distance < window)


def softmax_over(scores, seen):
    return torch.softmax(scores.masked_fill(~seen, float("-inf")), dim=-1)


def map_difference(first, second, lam, diff, eps):
    return unit_rms(first - lam * second, eps) * (1.0 - diff)


def differential_attention(h, weights, prefix, mixer, eps):
    heads, kv_heads, dim, vdim = mixer["heads"], mixer["kv_heads"], mixer["dim"], mixer["vdim"]
    tokens = h.shape[0]

    def projected(name):
        return h @ weights[f"{prefix}.{name}"].T + weights[f"{prefix}.{name}.b"]

    q, k, v = projected("q").view(tokens, heads, 2, dim), projected("k").view(tokens, kv_heads, 2, dim), projected("v").view(tokens, kv_heads, vdim)
    q = q * query_temperature(tokens, mixer["q_temp"]["coef"], mixer["q_temp"]["every"]).view(-1, 1, 1, 1)

    def agreement(n):
        return math.exp(float((weights[f"{prefix}.lq{n}"] * weights[f"{prefix}.lk{n}"]).sum()))

    lam = agreement(1) - agreement(2) + mixer["diff"]
    seen = visible(tokens)
    results = []
    for head in range(heads):
        group = head // (heads // kv_heads)
        maps = [softmax_over(q[:, head, m] @ k[:, group, m].T * mixer["scale"], seen) @ v[:, group] for m in (0, 1)]
        results.append(map_difference(maps[0], maps[1], lam, mixer["diff"], eps))
    return torch.cat(results, dim=-1) @ weights[f"{prefix}.o"].T + weights[f"{prefix}.o.b"]


def latent_attention(h, weights, prefix, mixer, eps):
    heads, dim, rot, vdim, rank = mixer["heads"], mixer["dim"], mixer["rot_dim"], mixer["vdim"], mixer["kv_rank"]
    tokens = h.shape[0]
    q = (h @ weights[f"{prefix}.q"].T).view(tokens, heads, dim + rot)
    down = h @ weights[f"{prefix}.dkv"].T
    latent = unit_rms(down[:, :rank], eps) * weights[f"{prefix}.dkv.norm"]
    shared = rotate_pairs(down[:, rank:], rot, mixer["rot"]["base"])
    turned = rotate_pairs(q[:, :, dim:], rot, mixer["rot"]["base"])
    keys = (latent @ weights[f"{prefix}.uk"].T).view(tokens, heads, dim)
    values = (latent @ weights[f"{prefix}.uv"].T).view(tokens, heads, vdim)
    gates = sigmoid(h @ weights[f"{prefix}.g"].T)
    seen = visible(tokens, mixer["mask"]["size"])
    results = []
    for head in range(heads):
        scores = (q[:, head, :dim] @ keys[:, head].T + turned[:, head] @ shared.T) * mixer["scale"]
        results.append(softmax_over(scores, seen) @ values[:, head] * gates[:, head : head + 1])
    return torch.cat(results, dim=-1) @ weights[f"{prefix}.o"].T


def dense_feed_forward(h, weights, prefix):
    gate = h @ weights[f"{prefix}.gate"].T
    return (gate * sigmoid(gate) * (h @ weights[f"{prefix}.up"].T)) @ weights[f"{prefix}.down"].T


def clamped_expert(h, weights, prefix, limit):
    g = (h @ weights[f"{prefix}.gate"].T).clamp(max=limit)
    u = (h @ weights[f"{prefix}.up"].T).clamp(-limit, limit)
    return (g * sigmoid(1.702 * g) * (u + 1.0)) @ weights[f"{prefix}.down"].T


def choose_experts(scores, top, groups, keep):
    """`scores` of one token's experts -> the chosen experts' numbers, best first."""
    size = len(scores) // groups
    ranked = []
    for group in range(groups):
        members = sorted(scores[group * size : (group + 1) * size], reverse=True)
        ranked.append((sum(members[:2]), -group))
    allowed = {-number for _, number in sorted(ranked, reverse=True)[:keep]}
    candidates = [(score, -expert) for expert, score in enumerate(scores) if expert // size in allowed]
    return [-number for _, number in sorted(candidates, reverse=True)[:top]]


def routed_feed_forward(h, weights, prefix, mlp):
    router, limit = mlp["router"], mlp["expert"]["limit"]
    scores = sigmoid(h @ weights[f"{prefix}.router"].T)
    share = torch.zeros_like(scores)
    for token in range(h.shape[0]):
        row = scores[token].tolist()
        chosen = choose_experts(row, router["top"], router["groups"]["count"], router["groups"]["keep"])
        total = sum(row[expert] for expert in chosen) + 1e-20
        for expert in chosen:
            share[token, expert] = row[expert] / total * router["scale"]
    out = torch.zeros_like(h)
    for expert in range(router["experts"]):                            # every expert on every token, weighted by zero where not chosen
        out += share[:, expert : expert + 1] * clamped_expert(h, weights, f"{prefix}.e{expert}", limit)
    return out


MIXERS = {"attention": differential_attention, "latent_attention": latent_attention}


def layer(x, index, weights, config):
    eps, entry, p = config["norm"]["eps"], config["layers"][index], f"l{index}"
    mixed = MIXERS[entry["type"]](zero_centred_norm(x, weights[f"{p}.norm1"], eps), weights, f"{p}.mix", entry["mixer"], eps)
    x = x + weights[f"{p}.ls1"] * mixed
    mlp = entry["mlp"]
    if mlp is None:
        return x
    h = zero_centred_norm(x, weights[f"{p}.norm2"], eps)
    fed = dense_feed_forward(h, weights, f"{p}.mlp") if mlp["kind"] == "dense" else routed_feed_forward(h, weights, f"{p}.mlp", mlp)
    return x + weights[f"{p}.ls2"] * fed


def runs(config):
    """(layer, whether the embedding output joins before it) in the order in which the layers run."""
    count, loop = len(config["layers"]), config.get("loop") or {"start": 0, "stop": 0, "times": 1}
    order = [(index, False) for index in range(loop["start"])]
    for turn in range(loop["times"]):
        order += [(index, turn > 0 and index == loop["start"]) for index in range(loop["start"], loop["stop"])]
    return order + [(index, False) for index in range(loop["stop"], count)]


def forward(tokens, weights, config, return_layers=False):
    """Logits `[tokens, vocab]` of one sequence from its first token on (and the stream behind every run, if asked)."""
    embedded = weights["embed"][torch.as_tensor(tokens, dtype=torch.long)]
    x, results = embedded, []
    for index, joins in runs(config):
        x = layer(x + embedded if joins else x, index, weights, config)
        results.append(x)
    logits = zero_centred_norm(x, weights["final.norm"], config["norm"]["eps"]) @ weights["head"].T
    return (logits, results) if return_layers else logits
