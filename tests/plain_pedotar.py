"""Pedotar, plain and slow: whole sequences, no cache, float64, one function per mechanism.

Written from the design's equations alone; it shares no code with the package.  `weights` maps stored tensor names to
tensors, `config` is the model's config.json as a dict.  Angles are formed as the design forms them: the 32-bit
product of a position and a 32-bit frequency.
"""

from __future__ import annotations

import json
from pathlib import Path

import numpy as np
import torch

F = torch.float64


def read_model(folder):
    """(config, {name: tensor}) of a folder with config.json and model.safetensors (an 8-byte length, a JSON table of
    names, then the data)."""
    folder = Path(folder)
    config = json.loads((folder / "config.json").read_text())
    raw = (folder / "model.safetensors").read_bytes()
    size = int.from_bytes(raw[:8], "little")
    table = json.loads(raw[8:8 + size])
    body = raw[8 + size:]
    weights = {}
    for name, entry in table.items():
        if name == "__metadata__":
            continue
        begin, end = entry["data_offsets"]
        data = body[begin:end]
        if entry["dtype"] == "BF16":
            bits = np.frombuffer(data, dtype=np.uint16).astype(np.uint32) << 16
            values = torch.from_numpy(bits.view(np.float32).copy())
        elif entry["dtype"] == "F32":
            values = torch.from_numpy(np.frombuffer(data, dtype=np.float32).copy())
        else:
            raise ValueError(f"{name}: dtype {entry['dtype']}")
        weights[name] = values.reshape(entry["shape"]).to(F)
    return config, weights


def layer_norm(x, weight, bias, eps):
    centred = x - x.mean(-1, keepdim=True)
    variance = (centred * centred).mean(-1, keepdim=True)
    return centred / torch.sqrt(variance + eps) * weight.to(F) + bias.to(F)


def rms_norm(x, weight, eps):
    return x / torch.sqrt((x * x).mean(-1, keepdim=True) + eps) * weight.to(F)


def silu(z):
    return z / (1.0 + torch.exp(-z))


def softplus(z):
    return torch.where(z > 30.0, z, torch.log1p(torch.exp(torch.clamp(z, max=30.0))))


def rotate(x, dims, base, positions=None):
    """x [T, heads, dims]: the pair of channels (i, i + dims/2) turns by position * base^(-2i / dims)."""
    half = dims // 2
    frequencies = torch.tensor([float(base) ** (-2.0 * i / dims) for i in range(half)], dtype=torch.float32)
    if positions is None:
        positions = torch.arange(x.shape[0])
    angles = (positions.to(torch.float32)[:, None] * frequencies[None, :]).to(F)          # a 32-bit product, then exact
    cos, sin = torch.cos(angles)[:, None, :], torch.sin(angles)[:, None, :]
    u, v = x[..., :half], x[..., half:dims]
    return torch.cat([u * cos - v * sin, v * cos + u * sin], dim=-1)


def short_convolution(x, taps, bias):
    """y[t, c] = sum_j taps[c, j] x[t - (n - 1) + j, c] + bias[c], zeros before the first token."""
    count = taps.shape[1]
    padded = torch.cat([torch.zeros(count - 1, x.shape[1], dtype=F), x])
    out = bias.to(F).expand_as(x).clone()
    for j in range(count):
        out = out + padded[j:j + x.shape[0]] * taps[:, j].to(F)
    return out


def selective_scan(x, step, a, b, c, d, state=None):
    """x, step [T, inner], a [inner, N] (negative), b, c [T, N], d [inner]: the recurrence
    S <- exp(step a) S + (step x) b, read out as S c + d x.  Returns (read-out [T, inner], the state at the end)."""
    s = torch.zeros_like(a) if state is None else state.clone()
    out = torch.zeros_like(x)
    for t in range(x.shape[0]):
        s = torch.exp(step[t][:, None] * a) * s + (step[t] * x[t])[:, None] * b[t][None, :]
        out[t] = s @ c[t] + d * x[t]
    return out, s


def mixer_mamba(h, weights, p, m):
    inner, rank, n = m["inner"], m["dt_rank"], m["state"]
    both = h @ weights[p + "in"].to(F).T
    x, z = both[:, :inner], both[:, inner:]
    x = silu(short_convolution(x, weights[p + "conv"], weights[p + "conv.b"]))
    low = x @ weights[p + "x"].to(F).T
    step = softplus(low[:, :rank] @ weights[p + "dt"].to(F).T + weights[p + "dt.b"].to(F))
    b, c = low[:, rank:rank + n], low[:, rank + n:]
    y, _ = selective_scan(x, step, -torch.exp(weights[p + "A_log"].to(F)), b, c, weights[p + "D"].to(F))
    return (y * silu(z)) @ weights[p + "o"].to(F).T


def softmax_over(scores, seen):
    scores = torch.where(seen, scores, torch.full_like(scores, -float("inf")))
    scores = torch.exp(scores - scores.max(-1, keepdim=True).values)
    return scores / scores.sum(-1, keepdim=True)


def visible(tokens, chunk=None):
    """[T, T]: query i sees key j iff j <= i and, with a chunk, both lie in the same run of `chunk` positions."""
    i, j = torch.arange(tokens)[:, None], torch.arange(tokens)[None, :]
    seen = j <= i
    if chunk is not None:
        seen = seen & (i // chunk == j // chunk)
    return seen


def mixer_latent(h, weights, p, m, eps):
    """Keys and values come out of one latent per token; one rotated key part is shared by all heads."""
    tokens, heads, dim, r, v, rank = h.shape[0], m["heads"], m["dim"], m["rot_dim"], m["vdim"], m["kv_rank"]
    q = (h @ weights[p + "q"].to(F).T).view(tokens, heads, dim + r)
    down = h @ weights[p + "dkv"].to(F).T
    latent = rms_norm(down[:, :rank], weights[p + "dkv.norm"], eps)
    shared = down[:, rank:].view(tokens, 1, r)
    plain_q, turned_q = q[..., :dim], q[..., dim:]
    if r:
        turned_q, shared = rotate(turned_q, r, m["rot"]["base"]), rotate(shared, r, m["rot"]["base"])
    keys = (latent @ weights[p + "uk"].to(F).T).view(tokens, heads, dim)
    values = (latent @ weights[p + "uv"].to(F).T).view(tokens, heads, v)
    scores = torch.einsum("ihd,jhd->hij", plain_q, keys) + torch.einsum("ihd,jd->hij", turned_q, shared[:, 0])
    amounts = softmax_over(scores * m["scale"], visible(tokens)[None])
    return torch.einsum("hij,jhd->ihd", amounts, values).reshape(tokens, heads * v) @ weights[p + "o"].to(F).T


def talking_attention(q, k, v, scale, talk=None, chunk=None):
    """q [T, H, D], k [T, G, D], v [T, G, V] -> [T, H, V]; head h's weights over the keys are the combination
    sum_g talk[h, g] of all heads' softmax weights."""
    tokens, heads, _ = q.shape
    per_group = heads // k.shape[1]
    keys, values = k.repeat_interleave(per_group, 1), v.repeat_interleave(per_group, 1)
    amounts = softmax_over(torch.einsum("ihd,jhd->hij", q, keys) * scale, visible(tokens, chunk)[None])
    if talk is not None:
        amounts = torch.einsum("hg,gij->hij", talk.to(F), amounts)
    return torch.einsum("hij,jhd->ihd", amounts, values)


def mixer_attention(h, weights, p, m, eps):
    tokens, heads, groups = h.shape[0], m["heads"], m["kv_heads"]
    q = (h @ weights[p + "q"].to(F).T).view(tokens, heads, m["dim"])
    k = (h @ weights[p + "k"].to(F).T).view(tokens, groups, m["dim"])
    v = (h @ weights[p + "v"].to(F).T).view(tokens, groups, m["vdim"])
    q, k = rms_norm(q, weights[p + "q.norm"], eps), rms_norm(k, weights[p + "k.norm"], eps)
    out = talking_attention(q, k, v, m["scale"], weights[p + "talk"], m["mask"]["size"])
    return out.reshape(tokens, heads * m["vdim"]) @ weights[p + "o"].to(F).T


def gated_feed_forward(h, weights, p):
    gate, up = h @ weights[p + "gate"].to(F).T, h @ weights[p + "up"].to(F).T
    return (silu(gate) * up) @ weights[p + "down"].to(F).T


def layer_order(config):
    """(layer, opens a pass after the first) of every run of a layer."""
    count = len(config["layers"])
    loop = config.get("loop")
    if not loop:
        return [(i, False) for i in range(count)]
    inside = range(loop["start"], loop["stop"])
    order = [(i, False) for i in range(loop["start"])]
    for number in range(loop["times"]):
        order += [(i, number > 0 and i == loop["start"]) for i in inside]
    return order + [(i, False) for i in range(loop["stop"], count)]


def forward(config, weights, tokens, want_layers=False):
    """Logits [T, vocab] of one sequence; with want_layers also the residual after every run of a layer."""
    eps = config["norm"]["eps"]
    norm = lambda x, name: layer_norm(x, weights[name], weights[name + ".b"], eps)
    embedded = weights["embed"].to(F)[torch.as_tensor(list(tokens), dtype=torch.long)]
    x = embedded
    seen = []
    for index, reopens in layer_order(config):
        layer, prefix = config["layers"][index], f"l{index}."
        if reopens:
            x = x + embedded
        h = norm(x, prefix + "norm1")
        kind, m, p = layer["type"], layer["mixer"], prefix + "mix."
        if kind == "mamba1":
            y = mixer_mamba(h, weights, p, m)
        elif kind == "latent_attention":
            y = mixer_latent(h, weights, p, m, eps)
        elif kind == "attention":
            y = mixer_attention(h, weights, p, m, eps)
        else:
            raise ValueError(kind)
        x = x + norm(y, prefix + "norm1b")
        if layer.get("mlp") is not None:
            y = gated_feed_forward(norm(x, prefix + "norm2"), weights, prefix + "mlp.")
            x = x + norm(y, prefix + "norm2b")
        seen.append(x)
    logits = norm(x, "final.norm") @ weights["embed"].to(F).T
    return (logits, torch.stack(seen)) if want_layers else logits
