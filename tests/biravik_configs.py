"""Tiny Biravik configurations for the tests, and model folders with weights that make every mechanism matter.  The
configurations differ from one another in every size, in the order and kinds of layers and in the constants; some take
values that make two sizes equal or 1, some leave optional keys out."""

from __future__ import annotations

import math
from pathlib import Path

import torch


def _left(heads, kv_heads, dim, vdim, scale, temperature=None):
    left = {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "scale": scale}
    if temperature:
        left["q_temp"] = {"coef": temperature[0], "every": temperature[1]}
    return left


def _right(dim, vdim, decays):
    return {"heads": len(decays), "dim": dim, "vdim": vdim, "decay": list(decays)}


def _parallel(left, right, left_scale, right_scale):
    return {"type": "parallel", "mixer": {"left": left, "right": right, "left_scale": left_scale, "right_scale": right_scale}}


def _attention(heads, kv_heads, dim, scale, window=None, keep_first=0, rot=None):
    mixer = {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": dim, "scale": scale}
    if window:
        mixer["mask"] = {"size": window, "keep_first": keep_first}
    if rot:
        mixer["rot"] = {"dims": rot[0], "base": rot[1]}
        if len(rot) > 2:
            mixer["rot"]["scaling"] = dict(zip(("factor", "original", "fast", "slow"), rot[2]))
    return {"type": "attention", "mixer": mixer}


def _wkv(heads, dim, rank):
    return {"type": "wkv", "mixer": {"heads": heads, "dim": dim, "decay_rank": rank}}


def _dense(ff):
    return {"kind": "dense", "ff": ff}


def _moe(experts, top, ff):
    return {"kind": "moe", "expert": {"ff": ff}, "router": {"experts": experts, "top": top}}


def _layer(mixer, mlp):
    return dict(mixer, mlp=mlp)


BIRAVIK_A = {   # every mixer and feed-forward; grouped heads everywhere, widths that all differ
    "architecture": "Biravik", "vocab": 211, "width": 96, "norm": {"eps": 1e-6}, "embedding": {"scale": 3.0},
    "postln_alpha": 1.4,
    "layers": [
        _layer(_parallel(_left(6, 3, 32, 20, 0.2, (0.4, 24)), _right(24, 40, (0.6, 0.95, 0.995)), 0.7, 1.2), _dense(160)),
        _layer(_attention(4, 2, 24, 0.25, window=19, keep_first=5, rot=(16, 500.0, (3.0, 64, 16.0, 1.0))), _moe(6, 3, 40)),
        _layer(_wkv(3, 20, 5), _moe(5, 2, 24)),
        _layer(_attention(3, 1, 16, 0.2, rot=(8, 10000.0)), None),
    ],
}

BIRAVIK_B = {   # sizes that are equal or 1: one head each, one expert chosen, no temperature, no rotation, no mask
    "architecture": "Biravik", "vocab": 130, "width": 64, "norm": {"eps": 1e-5}, "embedding": {"scale": 1.0},
    "postln_alpha": 1.0,
    "layers": [
        _layer(_parallel(_left(1, 1, 16, 16, 0.25), _right(16, 16, (0.9,)), 1.0, 1.0), _moe(2, 1, 64)),
        _layer(_attention(1, 1, 16, 0.3), _dense(64)),
        _layer(_wkv(1, 64, 1), _moe(3, 3, 16)),
    ],
}

BIRAVIK_C = {   # heads of 64 channels with narrower and wider values; widths that are no multiples of 8
    "architecture": "Biravik", "vocab": 150, "width": 100, "norm": {"eps": 1e-5}, "embedding": {"scale": 8.0},
    "postln_alpha": 2.5,
    "layers": [
        _layer(_parallel(_left(4, 2, 64, 32, 0.15, (0.2, 10)), _right(20, 12, (0.5, 0.9, 0.99, 1.0)), 1.1, 0.6), _dense(52)),
        _layer(_parallel(_left(5, 1, 64, 128, 0.12, (0.5, 7)), _right(36, 36, (0.999,)), 0.9, 0.8), None),
        _layer(_attention(6, 2, 64, 0.13, window=37, keep_first=3, rot=(64, 250000.0, (2.0, 40, 8.0, 1.0))), _moe(12, 4, 36)),
        _layer(_parallel(_left(3, 3, 64, 64, 0.14), _right(20, 64, (0.97, 0.8)), 0.5, 1.5), _dense(44)),
    ],
}

BIRAVIK_D = {   # heads of 128 channels: values of 64, of 128 and of 32 beside them
    "architecture": "Biravik", "vocab": 97, "width": 128, "norm": {"eps": 1e-6}, "embedding": {"scale": 0.5},
    "postln_alpha": 0.8,
    "layers": [
        _layer(_parallel(_left(4, 2, 128, 64, 0.09, (0.35, 50)), _right(128, 64, (0.99, 0.9)), 0.85, 1.05), _moe(5, 2, 48)),
        _layer(_attention(4, 1, 128, 0.08, window=70, keep_first=9, rot=(32, 10000.0, (4.0, 128, 32.0, 1.0))), _dense(200)),
        _layer(_parallel(_left(2, 1, 128, 128, 0.1, (0.6, 33)), _right(64, 128, (0.98,)), 1.3, 0.4), _dense(48)),
        _layer(_parallel(_left(2, 2, 128, 32, 0.1), _right(100, 20, (0.7, 0.995)), 1.0, 1.0), None),
    ],
}

ALL = {"A": BIRAVIK_A, "B": BIRAVIK_B, "C": BIRAVIK_C, "D": BIRAVIK_D}
PAGE_SIZES = {"A": 8, "B": 16, "C": 4, "D": 16}


def make_folder(tmp_path, config: dict, seed: int, dtype: str, sharpen: float = 2.0) -> Path:
    """config.json + model.safetensors.  The random weights of the package's writer are rescaled so that norm weights,
    sinks, gates, decays, blends, router and attention scores are far from their neutral values and a mixer's result is
    about as large as the residual it is added to: a lost state, a missed or extra key at a window's edge, a sink, a bias or
    a temperature left out then changes the logits well beyond the tolerances.  `sharpen` multiplies the attention scores
    (through the q and k norm weights)."""
    from libmir_b200.weights import load_tensor, read_catalog, write_file, write_model_folder
    folder = write_model_folder(Path(tmp_path), config, seed=seed, dtype=dtype)
    tensors = {name: load_tensor(entry) for name, entry in read_catalog(folder).items()}
    generator = torch.Generator().manual_seed(seed + 1000)
    normal = lambda shape, deviation: torch.randn(shape, generator=generator) * deviation
    for name, tensor in list(tensors.items()):
        kind, shape = tensor.dtype, tensor.shape
        last = name.split(".")[-1]
        if ".mu." in name:
            new = torch.rand(shape, generator=generator)
        elif last in ("norm1", "norm2") or name == "final.norm":
            new = normal(shape, 0.25)                             # stored around zero
        elif name.endswith("q.norm") or name.endswith("k.norm"):
            new = (1.0 + normal(shape, 0.25)) * sharpen ** 0.5
        elif last == "norm":
            new = 1.0 + normal(shape, 0.25)
        elif last == "sink":
            new = 1.0 + normal(shape, 1.0)
        elif last == "w0":
            new = normal(shape, 1.0) - 0.5
        elif last == "u":
            new = normal(shape, 0.5)
        elif len(shape) == 2:
            gain = {"router": 2.0, "g": 1.5, "w1": 0.5, "embed": 1.0}.get(last, 1.0)
            new = normal(shape, gain / math.sqrt(shape[1]) if name != "embed" else 1.0)
        else:
            continue
        tensors[name] = new.to(kind)
    write_file(folder / "model.safetensors", tensors)
    return folder


def random_config(rng) -> dict:
    """A configuration drawn at random: any layer order, head counts and widths that are no multiples of 8 (or of 4), with
    and without temperature, rotation, scaling, mask, kept tokens and feed-forward."""
    def parallel():
        dim = int(rng.choice([4, 12, 20, 32, 64, 96, 128]))
        kv_heads = int(rng.integers(1, 4))
        vdim = int(rng.choice([dim, 4, 6, 12, 32, 40, 64, 128]))
        temperature = (float(rng.uniform(0.05, 0.8)), int(rng.integers(1, 60))) if rng.random() < 0.8 else None
        left = _left(kv_heads * int(rng.integers(1, 5)), kv_heads, dim, vdim, float(rng.uniform(0.05, 0.3)), temperature)
        decays = [float(1.0 - 2.0 ** -rng.uniform(0.5, 11.0)) for _ in range(int(rng.integers(1, 6)))]
        right = _right(int(rng.choice([4, 12, 20, 32, 36, 64, 100, 128])), int(rng.choice([4, 6, 12, 20, 32, 64])), decays)
        return _parallel(left, right, float(rng.uniform(0.3, 1.5)), float(rng.uniform(0.3, 1.5)))

    def attention():
        dim = int(rng.choice([4, 12, 16, 24, 64, 80, 128]))
        kv_heads = int(rng.integers(1, 4))
        rot = None
        if rng.random() < 0.8:
            rot = (int(rng.choice([d for d in (2, 4, 6, 8, 16, 32, 64, 128) if d <= dim])),
                   float(rng.choice([50.0, 10000.0, 500000.0])))
            if rng.random() < 0.7:
                rot += ((float(rng.uniform(1.5, 8.0)), int(rng.integers(20, 200)), float(rng.uniform(8.0, 32.0)), 1.0),)
        window = int(rng.integers(1, 80)) if rng.random() < 0.8 else None
        keep = int(rng.integers(0, 12)) if rng.random() < 0.7 else 0
        return _attention(kv_heads * int(rng.integers(1, 5)), kv_heads, dim, float(rng.uniform(0.05, 0.3)), window, keep, rot)

    def wkv():
        return _wkv(int(rng.integers(1, 5)), int(rng.choice([4, 12, 20, 32, 48, 64, 100])), int(rng.integers(1, 20)))

    layers = []
    for _ in range(int(rng.integers(1, 6))):
        mixer = (parallel, attention, wkv)[int(rng.choice(3, p=[0.5, 0.3, 0.2]))]()
        kind = rng.random()
        experts = int(rng.integers(1, 10))
        mlp = None if kind < 0.2 else (_dense(int(rng.choice([40, 64, 100, 130]))) if kind < 0.6 else
                                       _moe(experts, int(rng.integers(1, experts + 1)), int(rng.choice([16, 20, 40]))))
        layers.append(_layer(mixer, mlp))
    return {"architecture": "Biravik", "vocab": int(rng.integers(30, 300)), "width": int(rng.choice([48, 52, 64, 72, 100, 136, 50])),
            "norm": {"eps": float(rng.choice([1e-5, 1e-6, 1e-4]))}, "embedding": {"scale": float(rng.uniform(0.5, 10.0))},
            "postln_alpha": float(rng.uniform(0.7, 3.0)), "layers": layers}
