"""A plain, slow implementation of the Biravik design in float64: whole sequences, no cache, no batching, one function
per mechanism.  It shares no code with the package and is what the engine is compared with.

Notation: n tokens, width w.  A stored matrix W has shape [out, in]; the row vector x of a token is multiplied
as x @ W.T.
"""

from __future__ import annotations

import json
import math
from pathlib import Path

import numpy as np
import torch

F64 = torch.float64


# ------------------------------------------------------------------------------ reading a model folder
def read_model(folder):
    """(config, {name: float64 tensor}) of a folder with config.json and model.safetensors."""
    folder = Path(folder)
    config = json.loads((folder / "config.json").read_text())
    raw = (folder / "model.safetensors").read_bytes()
    size = int.from_bytes(raw[:8], "little")
    header = json.loads(raw[8:8 + size])
    body = raw[8 + size:]
    weights = {}
    for name, entry in header.items():
        if name == "__metadata__":
            continue
        begin, end = entry["data_offsets"]
        data = body[begin:end]
        if entry["dtype"] == "BF16":
            bits = np.frombuffer(data, dtype=np.uint16).astype(np.uint32) << 16
            values = torch.from_numpy(bits.view(np.float32).copy())
        elif entry["dtype"] == "F32":
            values = torch.from_numpy(np.frombuffer(data, dtype=np.float32).copy())
        elif entry["dtype"] == "I32":
            values = torch.from_numpy(np.frombuffer(data, dtype=np.int32).copy())
        else:
            raise ValueError(f"{name}: dtype {entry['dtype']}")
        weights[name] = values.reshape(entry["shape"]).to(F64)
    return config, weights


# ------------------------------------------------------------------------------ small pieces
def unit_rms(x, eps):
    """x divided by its root mean square over the last axis, eps inside the root."""
    return x / torch.sqrt((x * x).mean(dim=-1, keepdim=True) + eps)


def silu(z):
    return z / (1.0 + torch.exp(-z))


def sigmoid(z):
    return 1.0 / (1.0 + torch.exp(-z))


def post_norm(x, added, weight, alpha, eps):
    """What a sublayer leaves: the norm (weight stored around zero) of alpha times its input plus its result."""
    return unit_rms(alpha * x + added, eps) * (1.0 + weight)


# ------------------------------------------------------------------------------ positions
def rotary_table(rot):
    """(frequencies [dims / 2], factor on cos and sin) of a `rot` table {dims, base, scaling?}."""
    dims, base = int(rot["dims"]), float(rot["base"])
    half = dims // 2
    freq = torch.tensor([base ** (-2.0 * i / dims) for i in range(half)], dtype=F64)
    scaling = rot.get("scaling")
    if not scaling:
        return freq, 1.0
    factor, original = float(scaling["factor"]), float(scaling["original"])

    def turns_to_dim(turns):
        return dims * math.log(original / (2.0 * math.pi * turns)) / (2.0 * math.log(base))

    low = max(math.floor(turns_to_dim(float(scaling["fast"]))), 0)
    high = min(math.ceil(turns_to_dim(float(scaling["slow"]))), dims - 1)
    ramp = torch.tensor([min(max((i - low) / max(high - low, 0.001), 0.0), 1.0) for i in range(half)], dtype=F64)
    return freq / factor * ramp + freq * (1.0 - ramp), 0.1 * math.log(factor) + 1.0


def rotate_interleaved(x, positions, rot):
    """x [n, heads, d]: the first rot.dims of the last axis rotated in pairs (2i, 2i + 1) by position * frequency."""
    freq, magnitude = rotary_table(rot)
    dims = int(rot["dims"])
    angles = positions.to(F64)[:, None] * freq[None, :]
    cos, sin = (torch.cos(angles) * magnitude)[:, None, :], (torch.sin(angles) * magnitude)[:, None, :]
    out = x.clone()
    even, odd = x[..., 0:dims:2], x[..., 1:dims:2]
    out[..., 0:dims:2] = even * cos - odd * sin
    out[..., 1:dims:2] = odd * cos + even * sin
    return out


def query_temperature(positions, coef, every):
    """What a query is multiplied by at each position."""
    return 1.0 + float(coef) * torch.log(torch.floor((positions.to(F64) + 1.0) / float(every)) + 1.0)


def slopes(heads):
    """How much a head's score falls per position of distance."""
    return torch.tensor([2.0 ** (-8.0 * (h + 1) / heads) for h in range(heads)], dtype=F64)


def visible(n, size=None, keep_first=0):
    """[query, key]: whether the query sees the key; with a size, only the last `size` keys and the kept first ones."""
    i, j = torch.arange(n)[:, None], torch.arange(n)[None, :]
    seen = j <= i
    if size is not None:
        seen = seen & ((i - j < size) | (j < keep_first))
    return seen


def sink_softmax(scores, sinks):
    """scores [heads, n, n] with -inf where hidden; exp(sinks[h]) joins the denominator."""
    top = torch.maximum(scores.amax(dim=-1, keepdim=True), sinks[:, None, None])
    weights = torch.exp(scores - top)
    return weights / (weights.sum(dim=-1, keepdim=True) + torch.exp(sinks[:, None, None] - top))


def grouped_attention(q, k, v, scale, sinks, seen, bias=None):
    """q [n, H, d], k [n, G, d], v [n, G, e]; bias [H, n, n] is taken off the scaled scores."""
    n, heads = q.shape[:2]
    group = heads // k.shape[1]
    k, v = k.repeat_interleave(group, dim=1), v.repeat_interleave(group, dim=1)
    scores = torch.einsum("ihd,jhd->hij", q, k) * scale
    if bias is not None:
        scores = scores - bias
    scores = scores.masked_fill(~seen[None], float("-inf"))
    return torch.einsum("hij,jhe->ihe", sink_softmax(scores, sinks), v).reshape(n, -1)


# ------------------------------------------------------------------------------ mixers
def biased_attention(h, weights, prefix, mixer, eps):
    """Attention without rotation: a temperature on the queries and a bias that falls with the distance."""
    n = h.shape[0]
    heads, kv_heads, dim, vdim = (int(mixer[key]) for key in ("heads", "kv_heads", "dim", "vdim"))
    w = lambda name: weights[prefix + name]
    positions = torch.arange(n)
    q = unit_rms((h @ w("q").T).reshape(n, heads, dim), eps) * w("q.norm")
    k = unit_rms((h @ w("k").T).reshape(n, kv_heads, dim), eps) * w("k.norm")
    v = (h @ w("v").T).reshape(n, kv_heads, vdim)
    if mixer.get("q_temp"):
        q = q * query_temperature(positions, mixer["q_temp"]["coef"], mixer["q_temp"]["every"])[:, None, None]
    distance = (positions[:, None] - positions[None, :]).to(F64)
    mixed = grouped_attention(q, k, v, float(mixer["scale"]), w("sink"), visible(n),
                              slopes(heads)[:, None, None] * distance)
    return (mixed * sigmoid(h @ w("g").T)) @ w("o").T


def lightning(h, weights, prefix, mixer, eps):
    """Linear attention with a fixed decay per head and silu on everything that enters the recurrence."""
    n = h.shape[0]
    heads, dim, vdim = (int(mixer[key]) for key in ("heads", "dim", "vdim"))
    w = lambda name: weights[prefix + name]
    q = silu(h @ w("q").T).reshape(n, heads, dim)
    k = silu(h @ w("k").T).reshape(n, heads, dim)
    v = silu(h @ w("v").T).reshape(n, heads, vdim)
    decay = torch.tensor([float(d) for d in mixer["decay"]], dtype=F64)[:, None, None]
    state = torch.zeros(heads, dim, vdim, dtype=F64)
    out = torch.zeros(n, heads, vdim, dtype=F64)
    for t in range(n):
        state = decay * state + k[t][:, :, None] * v[t][:, None, :]
        out[t] = torch.einsum("hkv,hk->hv", state, q[t])
    out = unit_rms(out.reshape(n, heads * vdim), eps) * w("norm")
    return (out * sigmoid(h @ w("g").T)) @ w("o").T


def side_by_side(h, weights, prefix, mixer, eps):
    return float(mixer["left_scale"]) * biased_attention(h, weights, prefix + "left.", mixer["left"], eps) \
        + float(mixer["right_scale"]) * lightning(h, weights, prefix + "right.", mixer["right"], eps)


def key_value_attention(h, weights, prefix, mixer, eps):
    """Windowed attention whose values are the keys' raw projections (neither normed nor rotated)."""
    n = h.shape[0]
    heads, kv_heads, dim = (int(mixer[key]) for key in ("heads", "kv_heads", "dim"))
    w = lambda name: weights[prefix + name]
    positions = torch.arange(n)
    raw = (h @ w("k").T).reshape(n, kv_heads, dim)
    q = unit_rms((h @ w("q").T).reshape(n, heads, dim), eps) * w("q.norm")
    k = unit_rms(raw, eps) * w("k.norm")
    if mixer.get("rot"):
        q, k = rotate_interleaved(q, positions, mixer["rot"]), rotate_interleaved(k, positions, mixer["rot"])
    mask = mixer.get("mask") or {}
    seen = visible(n, int(mask["size"]), int(mask.get("keep_first", 0))) if mask.get("size") else visible(n)
    mixed = grouped_attention(q, k, raw, float(mixer["scale"]), w("sink"), seen)
    return (mixed * sigmoid(h @ w("g").T)) @ w("o").T


def wkv(h, weights, prefix, mixer, eps):
    """Time mixing with a matrix state per head and a decay per head and key channel."""
    n = h.shape[0]
    heads, dim = int(mixer["heads"]), int(mixer["dim"])
    w = lambda name: weights[prefix + name]
    before = torch.cat([torch.zeros(1, h.shape[1], dtype=F64), h[:-1]], dim=0)
    mix = lambda name: h + (before - h) * w("mu." + name)
    r, k, v = ((mix(name) @ w(name).T).reshape(n, heads, dim) for name in ("r", "k", "v"))
    gate = silu(mix("g") @ w("g").T)
    decay = torch.exp(-torch.exp(torch.tanh(mix("w") @ w("w1").T) @ w("w2").T + w("w0"))).reshape(n, heads, dim)
    bonus = w("u").reshape(heads, dim)
    state = torch.zeros(heads, dim, dim, dtype=F64)                           # [head, key channel, value channel]
    out = torch.zeros(n, heads, dim, dtype=F64)
    for t in range(n):
        outer = k[t][:, :, None] * v[t][:, None, :]
        out[t] = torch.einsum("hkv,hk->hv", state + bonus[:, :, None] * outer, r[t])
        state = decay[t][:, :, None] * state + outer
    out = unit_rms(out, eps).reshape(n, heads * dim) * w("norm")
    return (out * gate) @ w("o").T


MIXERS = {"parallel": side_by_side, "attention": key_value_attention, "wkv": wkv}


# ------------------------------------------------------------------------------ feed-forwards
def dense_mlp(h, weights, prefix):
    return torch.relu(h @ weights[prefix + "up"].T) ** 2 @ weights[prefix + "down"].T


def gated_expert(h, weights, prefix):
    return (silu(h @ weights[prefix + "gate"].T) * (h @ weights[prefix + "up"].T)) @ weights[prefix + "down"].T


def route(h, weights, prefix, router):
    """(chosen experts [n, top], their weights [n, top]): the softmax is over the chosen logits alone."""
    logits = h @ weights[prefix + "router"].T
    picked, chosen = logits.topk(int(router["top"]), dim=-1)
    return chosen, torch.softmax(picked, dim=-1)


def mixture(h, weights, prefix, mlp):
    chosen, share = route(h, weights, prefix, mlp["router"])
    out = torch.zeros_like(h)
    for t in range(h.shape[0]):
        for expert, weight in zip(chosen[t].tolist(), share[t].tolist()):
            out[t] += weight * gated_expert(h[t:t + 1], weights, f"{prefix}e{expert}.")[0]
    return out


# ------------------------------------------------------------------------------ the model
def layer(x, index, config, weights, read=lambda h: h):
    """`read`: what a sublayer makes of the residual as it reads it (a rounding, to see how much of one the model magnifies)."""
    spec = config["layers"][index]
    eps, alpha = float(config["norm"]["eps"]), float(config["postln_alpha"])
    prefix = f"l{index}."
    mixed = MIXERS[spec["type"]](read(x), weights, prefix + "mix.", spec["mixer"], eps)
    x = post_norm(x, mixed, weights[prefix + "norm1"], alpha, eps)
    mlp = spec.get("mlp")
    if mlp is None:
        return x
    fed = dense_mlp(read(x), weights, prefix + "mlp.") if mlp["kind"] == "dense" \
        else mixture(read(x), weights, prefix + "mlp.", mlp)
    return post_norm(x, fed, weights[prefix + "norm2"], alpha, eps)


def forward(config, weights, ids, trace=None, read=lambda h: h):
    """Logits [n, vocab] of one sequence; `trace`, a list, receives the residual stream after every layer."""
    ids = torch.as_tensor(ids, dtype=torch.long)
    x = weights["embed"][ids] * float((config.get("embedding") or {}).get("scale", 1.0))
    for index in range(len(config["layers"])):
        x = layer(x, index, config, weights, read)
        if trace is not None:
            trace.append(x.clone())
    return (unit_rms(x, float(config["norm"]["eps"])) * (1.0 + weights["final.norm"])) @ weights["head"].T
