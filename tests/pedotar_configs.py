"""Tiny Pedotar configurations for the tests, and model folders with weights that make every mechanism matter.
The configurations differ from one another in every size, in the kinds and order of layers, in the loop, head counts,
runs of positions, rotations and state sizes; some take values that make two sizes equal or 1, some have sizes that are
no multiples of 8, some have heads that the tensor-core kernels take (64 and 128 channels)."""

from __future__ import annotations

import math
from pathlib import Path

import torch


def scan(inner, state, dt_rank, conv):
    return {"type": "mamba1", "mixer": {"inner": inner, "state": state, "dt_rank": dt_rank, "conv": conv}}


def latent(heads, dim, rot_dim, vdim, kv_rank, scale, base=10000.0):
    return {"type": "latent_attention", "mixer": {"heads": heads, "dim": dim, "rot_dim": rot_dim, "vdim": vdim,
                                                  "kv_rank": kv_rank, "scale": scale, "rot": {"dims": rot_dim, "base": base}}}


def mixed(heads, kv_heads, dim, vdim, scale, size):
    return {"type": "attention", "mixer": {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "scale": scale,
                                           "mask": {"size": size}}}


def _layer(mixer, ff=None):
    return dict(mixer, mlp=None if ff is None else {"kind": "dense", "ff": ff})


PEDOTAR_A = {   # every kind of layer inside and outside the loop; grouped heads, value heads narrower and wider than keys
    "architecture": "Pedotar", "vocab": 203, "width": 80, "norm": {"eps": 1e-5}, "loop": {"start": 1, "stop": 4, "times": 2},
    "layers": [
        _layer(mixed(4, 2, 24, 40, 0.3, 19), 72),
        _layer(scan(88, 16, 8, 4)),
        _layer(latent(3, 16, 8, 24, 48, 0.2, 700.0), 56),
        _layer(mixed(6, 3, 16, 8, 0.25, 33)),
        _layer(scan(64, 10, 3, 3), 40),
    ],
}

PEDOTAR_B = {   # sizes that are 1 or equal, widths that are no multiples of 8, no loop
    "architecture": "Pedotar", "vocab": 61, "width": 52, "norm": {"eps": 1e-6},
    "layers": [
        _layer(scan(20, 1, 1, 1), 30),
        _layer(mixed(1, 1, 12, 12, 0.5, 1), 52),
        _layer(latent(1, 6, 2, 10, 14, 0.4, 100.0)),
        _layer(scan(52, 7, 5, 2)),
        _layer(mixed(3, 1, 10, 6, 0.4, 5)),
    ],
}

PEDOTAR_C = {   # heads of 64 channels (tensor cores in bfloat16), as many key heads as query heads; the loop at the end
    "architecture": "Pedotar", "vocab": 151, "width": 104, "norm": {"eps": 1e-5}, "loop": {"start": 1, "stop": 3, "times": 2},
    "layers": [
        _layer(scan(160, 12, 6, 4)),
        _layer(mixed(5, 5, 64, 64, 0.12, 50), 88),
        _layer(latent(4, 32, 16, 32, 96, 0.15, 250000.0), 64),
    ],
}

PEDOTAR_D = {   # heads of 128 channels in groups; the whole model repeated; a wide state
    "architecture": "Pedotar", "vocab": 97, "width": 128, "norm": {"eps": 1e-6}, "loop": {"start": 0, "stop": 3, "times": 2},
    "layers": [
        _layer(mixed(12, 3, 128, 128, 0.09, 70), 96),
        _layer(scan(136, 40, 16, 4), 64),
        _layer(latent(2, 64, 32, 64, 128, 0.1, 5000.0)),
    ],
}

PEDOTAR_E = {   # recurrent layers only: nothing is kept in pages
    "architecture": "Pedotar", "vocab": 77, "width": 64, "norm": {"eps": 1e-5}, "loop": {"start": 1, "stop": 2, "times": 4},
    "layers": [_layer(scan(96, 8, 4, 4)), _layer(scan(32, 20, 2, 2), 48)],
}

ALL = {"A": PEDOTAR_A, "B": PEDOTAR_B, "C": PEDOTAR_C, "D": PEDOTAR_D, "E": PEDOTAR_E}
PAGE_SIZES = {"A": 8, "B": 4, "C": 16, "D": 16, "E": 16}


def make_folder(tmp_path, config: dict, seed: int, dtype: str, sharpen: float = 2.0, edit=None) -> Path:
    """config.json + model.safetensors.  The random weights of the package's writer are rescaled so that norm weights
    and biases, the heads' mixing, step sizes, decays and attention scores are far from their neutral values: a key
    missed or seen at the edge of a run, a state that is lost, a norm or a pass left out then changes the logits well
    beyond the tolerances.  `sharpen` multiplies the scores; `edit(tensors)` may change the table of tensors before it
    is written."""
    from libmir_b200.weights import load_tensor, read_catalog, write_file, write_model_folder
    folder = write_model_folder(Path(tmp_path), config, seed=seed, dtype=dtype)
    tensors = {name: load_tensor(entry) for name, entry in read_catalog(folder).items()}
    generator = torch.Generator().manual_seed(seed + 1000)
    normal = lambda shape, deviation: torch.randn(shape, generator=generator) * deviation
    for name, tensor in list(tensors.items()):
        kind = tensor.dtype
        parts = name.split(".")
        last = parts[-1]
        if last in ("norm1", "norm2", "norm1b", "norm2b") or name == "final.norm" or name.endswith("dkv.norm"):
            new = 1.0 + normal(tensor.shape, 0.25)
        elif name.endswith("q.norm") or name.endswith("k.norm"):
            new = (1.0 + normal(tensor.shape, 0.25)) * sharpen ** 0.5
        elif name.endswith("dt.b"):
            new = -2.5 + normal(tensor.shape, 0.8)             # step sizes of a few hundredths to a few tenths
        elif last == "b":
            new = normal(tensor.shape, 0.3)
        elif last == "A_log":
            new = torch.log(0.05 + torch.rand(tensor.shape, generator=generator) * 4.0)
        elif last == "D":
            new = 1.0 + normal(tensor.shape, 0.4)
        elif last == "conv":
            new = normal(tensor.shape, 1.0 / math.sqrt(tensor.shape[1]))
        elif last == "talk":
            new = torch.eye(tensor.shape[0]) + normal(tensor.shape, 0.5)
        elif name == "embed":
            new = tensor.float() * 25.0
        elif tensor.dim() == 2:                                # projections: results about as large as their inputs
            new = tensor.float() * (50.0 / math.sqrt(tensor.shape[1]))
            if last in ("q", "dkv") and f"{name[:-len(last)]}dkv" in tensors:
                new = new * sharpen ** 0.5
        else:
            continue
        tensors[name] = new.to(kind)
    if edit is not None:
        edit(tensors)
    write_file(folder / "model.safetensors", tensors)
    return folder


def random_config(rng) -> dict:
    """A configuration drawn at random: any order of layers, head counts and widths that are no multiples of 8 (or of
    4), with and without feed-forwards and loop, runs of positions from one on."""
    def mixer():
        kind = rng.integers(0, 3)
        if kind == 0:
            return scan(int(rng.choice([12, 40, 64, 72, 100])), int(rng.choice([1, 4, 9, 16, 24, 33, 64])),
                        int(rng.integers(1, 20)), int(rng.integers(1, 6)))
        if kind == 1:
            return latent(int(rng.integers(1, 7)), int(rng.choice([4, 6, 16, 32, 40])), int(rng.choice([2, 4, 8, 16, 32])),
                          int(rng.choice([4, 12, 16, 24, 64])), int(rng.choice([10, 16, 40, 64, 128])),
                          float(rng.uniform(0.05, 0.4)), float(rng.choice([50.0, 10000.0, 500000.0])))
        kv_heads = int(rng.integers(1, 5))
        dim = int(rng.choice([4, 10, 16, 24, 32, 64, 64, 128]))
        vdim = dim if rng.random() < 0.6 else int(rng.choice([4, 6, 16, 24, 64, 128]))
        return mixed(kv_heads * int(rng.integers(1, 5)), kv_heads, dim, vdim, float(rng.uniform(0.05, 0.4)),
                     int(rng.integers(1, 90)))

    layers = [_layer(mixer(), int(rng.choice([40, 64, 100, 30])) if rng.random() < 0.6 else None)
              for _ in range(int(rng.integers(1, 5)))]
    config = {"architecture": "Pedotar", "vocab": int(rng.integers(30, 300)),
              "width": int(rng.choice([48, 52, 64, 72, 100, 136, 50])),
              "norm": {"eps": float(rng.choice([1e-5, 1e-6, 1e-4]))}, "layers": layers}
    if rng.random() < 0.7:
        start = int(rng.integers(0, len(layers)))
        config["loop"] = {"start": start, "stop": int(rng.integers(start, len(layers) + 1)), "times": int(rng.integers(1, 4))}
    return config
