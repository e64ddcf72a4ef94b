"""Biravik without a GPU: configuration -> model description, tensor names and shapes, what the cache manager is asked for,
configuration errors; fixed points of the plain implementation itself, and that every mechanism shows in its logits."""

import copy
import math

import numpy as np
import pytest
import torch

import plain_biravik as plain
from biravik_configs import ALL, BIRAVIK_A, BIRAVIK_B, BIRAVIK_C, make_folder, random_config

from libmir_b200.cache import CacheManager
from libmir_b200.config.spec import CacheBundle, FixedState, PagedKv, QueryTemperature, YarnScaling
from libmir_b200.errors import ConfigError
from libmir_b200.models.decoder import DecoderModel
from libmir_b200.parts.base import BuildEnv
from libmir_b200.registry import architecture_of, build_spec
from libmir_b200.weights import catalog_shapes, parameter_specs

F64 = torch.float64


def test_the_class_is_chosen_by_the_configuration():
    assert architecture_of(BIRAVIK_A) == "Biravik"
    assert build_spec(BIRAVIK_A, None).architecture == "Biravik"


def test_description_and_tensor_names():
    spec = build_spec(BIRAVIK_A, None)
    assert [layer.mixer.kind for layer in spec.layers] == ["side_by_side", "softmax_attention", "wkv", "softmax_attention"]
    assert all(layer.arrangement == "post_norm" and layer.residual_alpha == 1.4 for layer in spec.layers)
    assert spec.embedding.multiplier == 3.0 and spec.final_norm.offset == 1.0 and not spec.head.tied
    assert spec.layers[3].feed_forward is None and spec.layers[3].feed_forward_norm is None
    assert spec.layers[0].feed_forward.activation == "relu2" and spec.layers[0].feed_forward.intermediate_size == 160
    pair = spec.layers[0].mixer
    assert pair.scales == (0.7, 1.2) and [name for name, _ in pair.branches] == ["left", "right"]
    left, right = (branch for _, branch in pair.branches)
    assert (left.heads, left.kv_heads, left.head_dim, left.value_dim, left.scale) == (6, 3, 32, 20, 0.2)
    assert left.position is None and left.sinks and left.gate and left.qk_norm and left.window is None
    assert left.temperature == QueryTemperature(0.4, 24.0)
    assert left.slopes == tuple(2.0 ** (-8.0 * h / 6) for h in range(1, 7))
    assert (right.heads, right.key_dim, right.value_dim, right.decays) == (3, 24, 40, (0.6, 0.95, 0.995))
    assert right.activated and right.norm_span == "all" and right.norm_weight and right.gate == "sigmoid" and right.key_scale == 1.0
    attention = spec.layers[1].mixer
    assert attention.values_from_keys and attention.window == 19 and attention.keep_first == 5 and not attention.slopes
    assert attention.position.layout == "interleaved" and attention.position.rotary_dim == 16
    assert attention.position.scaling == YarnScaling(3.0, 64.0, 16.0, 1.0)
    experts = spec.layers[1].feed_forward
    assert (experts.experts, experts.top, experts.expert_size, experts.score, experts.correction) == (6, 3, 40, "softmax", False)
    assert spec.layers[3].mixer.window is None and spec.layers[3].mixer.position.scaling is None
    plain_left = build_spec(BIRAVIK_B, None).layers[0].mixer.branches[0][1]
    assert plain_left.temperature is None and plain_left.slopes == (2.0 ** -8,)
    assert build_spec(BIRAVIK_B, None).layers[1].mixer.position is None
    shapes = {name: tuple(param.shape) for name, param in parameter_specs(BIRAVIK_A).items()}
    assert shapes["embed"] == (211, 96) and shapes["final.norm"] == (96,) and shapes["head"] == (211, 96)
    assert shapes["l0.norm1"] == (96,) and shapes["l0.norm2"] == (96,) and "l3.norm2" not in shapes
    assert shapes["l0.mix.left.q"] == (192, 96) and shapes["l0.mix.left.k"] == (96, 96) and shapes["l0.mix.left.v"] == (60, 96)
    assert shapes["l0.mix.left.q.norm"] == (32,) and shapes["l0.mix.left.k.norm"] == (32,) and shapes["l0.mix.left.sink"] == (6,)
    assert shapes["l0.mix.left.g"] == (120, 96) and shapes["l0.mix.left.o"] == (96, 120)
    assert shapes["l0.mix.right.q"] == (72, 96) and shapes["l0.mix.right.v"] == (120, 96)
    assert shapes["l0.mix.right.norm"] == (120,) and shapes["l0.mix.right.g"] == (120, 96) and shapes["l0.mix.right.o"] == (96, 120)
    assert not any(name.endswith(".out") for name in shapes)      # (branches with factors have no norms of their own)
    assert shapes["l1.mix.q"] == (96, 96) and shapes["l1.mix.k"] == (48, 96) and "l1.mix.v" not in shapes
    assert shapes["l1.mix.g"] == (96, 96) and shapes["l1.mix.sink"] == (4,)
    assert shapes["l1.mlp.router"] == (6, 96) and shapes["l1.mlp.e5.down"] == (96, 40) and "l1.mlp.correction" not in shapes
    assert shapes["l2.mix.w1"] == (5, 96) and shapes["l2.mix.u"] == (3, 20) and shapes["l2.mix.mu.w"] == (96,)
    assert "l3.mlp.up" not in shapes


def test_what_the_cache_manager_is_asked_for():
    plan = DecoderModel(build_spec(BIRAVIK_A, None), BuildEnv(torch.float32, torch.device("cpu"))).cache_plan()
    assert plan[0].requirement == CacheBundle(PagedKv(3, 32, None, 20), (FixedState((3, 40, 24), "float32"),))
    assert plan[1].requirement == PagedKv(2, 24, 19, None, 5)
    assert plan[2].requirement == CacheBundle(None, (FixedState((3, 20, 20), "float32"), FixedState((96,), "float32")))
    assert plan[3].requirement == PagedKv(1, 16, None, None, 0)
    manager = CacheManager(plan, page_size=8, num_pages=10, max_requests=2)
    assert sorted(manager.state_entries) == [0, 2]


def test_random_weights_have_the_configurations_names(tmp_path):
    folder = make_folder(tmp_path, BIRAVIK_C, seed=1, dtype="bfloat16")
    catalog = dict(catalog_shapes(folder))
    assert set(catalog) == set(parameter_specs(BIRAVIK_C))
    config, weights = plain.read_model(folder)
    logits = plain.forward(config, weights, [1, 2, 3, 4, 5])
    assert logits.shape == (5, 150) and torch.isfinite(logits).all()


def test_the_rank_of_the_decay_comes_from_the_checkpoint():
    catalog = {"l2.mix.w1": (11, 96)}
    assert build_spec(BIRAVIK_A, catalog).layers[2].mixer.decay_rank == 11


def test_configurations_drawn_at_random_are_described():
    rng = np.random.default_rng(3)
    for _ in range(30):
        config = random_config(rng)
        spec = build_spec(config, None)
        assert len(spec.layers) == len(config["layers"]) == len(spec.schedule)
        DecoderModel(spec, BuildEnv(torch.float32, torch.device("cpu"))).cache_plan()


@pytest.mark.parametrize("change,text", [
    (lambda c: c["layers"][0].update(type="mamba"), "type"),
    (lambda c: c["layers"][1]["mlp"].update(kind="routed"), "kind"),
    (lambda c: c["layers"][1]["mlp"]["router"].update(top=7), "router"),
    (lambda c: c["layers"][1]["mixer"].pop("kv_heads"), "kv_heads"),
    (lambda c: c["layers"][1]["mixer"].update(vdim=20), "vdim"),
    (lambda c: c["layers"][1]["mixer"].update(heads=3), "kv_heads"),
    (lambda c: c["layers"][1]["mixer"]["rot"].update(dims=26), "rot.dims"),
    (lambda c: c["layers"][1]["mixer"]["rot"]["scaling"].pop("slow"), "slow"),
    (lambda c: c["layers"][1]["mixer"]["mask"].update(size=0), "size"),
    (lambda c: c["layers"][0]["mixer"]["left"].pop("scale"), "scale"),
    (lambda c: c["layers"][0]["mixer"]["left"]["q_temp"].update(every=0), "every"),
    (lambda c: c["layers"][0]["mixer"]["right"].update(decay=[0.5]), "decay"),
    (lambda c: c["layers"][0]["mixer"].pop("right_scale"), "right_scale"),
    (lambda c: c["layers"][0]["mixer"].pop("left"), "left"),
    (lambda c: c.pop("postln_alpha"), "postln_alpha"),
    (lambda c: c.pop("width"), "width"),
    (lambda c: c.pop("norm"), "norm"),
])
def test_configuration_errors_name_what_is_wrong(change, text):
    config = copy.deepcopy(BIRAVIK_A)
    change(config)
    with pytest.raises(ConfigError) as error:
        build_spec(config, None)
    assert text in str(error.value)


def test_combinations_that_the_parts_do_not_know_are_refused():
    from dataclasses import replace
    from libmir_b200.registry import build_part
    env = BuildEnv(torch.float32, torch.device("cpu"))
    left = build_spec(BIRAVIK_A, None).layers[0].mixer.branches[0][1]
    keys = build_spec(BIRAVIK_A, None).layers[1].mixer
    right = build_spec(BIRAVIK_A, None).layers[0].mixer.branches[1][1]
    for spec in (replace(left, slopes=(0.5,)), replace(left, window=8, keep_first=2), replace(keys, value_head_dim=12),
                 replace(keys, own_kv=False), replace(right, gate="relu"), replace(right, norm_span="group")):
        with pytest.raises(ValueError):
            build_part(spec, env)
    assert not build_part(left, env).plain and not build_part(keys, env).plain


def test_every_mechanism_shows_in_the_logits(tmp_path):
    """With the tests' weights, changing or leaving out any one mechanism moves the plain implementation's logits by far
    more than the engine's tolerance, so that a comparison with it would notice."""
    folder = make_folder(tmp_path, BIRAVIK_A, seed=3, dtype="float32")
    config, weights = plain.read_model(folder)
    ids = np.random.default_rng(0).integers(0, config["vocab"], 90).tolist()
    want = plain.forward(config, weights, ids)

    def moved(change_config=None, change_weights=None):
        c, w = copy.deepcopy(config), dict(weights)
        if change_config:
            change_config(c)
        if change_weights:
            change_weights(w)
        other = plain.forward(c, w, ids)
        return float((((other - want) ** 2).mean(-1).sqrt() / (want ** 2).mean(-1).sqrt()).median())
    mixer = lambda c, i: c["layers"][i]["mixer"]
    cases = {
        "alpha": (lambda c: c.update(postln_alpha=1.5), None),
        "temperature": (lambda c: mixer(c, 0)["left"].pop("q_temp"), None),
        "temperature's step": (lambda c: mixer(c, 0)["left"]["q_temp"].update(every=25), None),
        "left factor": (lambda c: mixer(c, 0).update(left_scale=1.0), None),
        "right factor": (lambda c: mixer(c, 0).update(right_scale=1.0), None),
        "decay": (lambda c: mixer(c, 0)["right"].update(decay=[0.6, 0.95, 0.98]), None),
        "window": (lambda c: mixer(c, 1)["mask"].update(size=20), None),
        "kept tokens": (lambda c: mixer(c, 1)["mask"].update(keep_first=4), None),
        "scaling": (lambda c: mixer(c, 1)["rot"].pop("scaling"), None),
        "rotation": (lambda c: mixer(c, 3).pop("rot"), None),
        "left sink": (None, lambda w: w.update({"l0.mix.left.sink": w["l0.mix.left.sink"] - 40.0})),
        "sink": (None, lambda w: w.update({"l1.mix.sink": w["l1.mix.sink"] - 40.0})),
        "left gate": (None, lambda w: w.update({"l0.mix.left.g": w["l0.mix.left.g"] * 0.0})),
        "lightning norm": (None, lambda w: w.update({"l0.mix.right.norm": w["l0.mix.right.norm"] * 0.0 + 1.0})),
        "blend": (None, lambda w: w.update({"l2.mix.mu.w": w["l2.mix.mu.w"] * 0.0})),
        "bonus": (None, lambda w: w.update({"l2.mix.u": w["l2.mix.u"] * 0.0})),
        "norm behind the mixer": (None, lambda w: w.update({"l1.norm1": w["l1.norm1"] * 0.0})),
    }
    for name, change in cases.items():
        assert moved(*change) > 1e-3, f"{name}: {moved(*change):.2e}"
    # the slope: another exponent
    original = plain.slopes
    try:
        plain.slopes = lambda heads: original(heads) * 0.0
        assert moved() > 1e-2
    finally:
        plain.slopes = original


def test_plain_implementation_fixed_points():
    x = torch.tensor([[3.0, 4.0]], dtype=F64)
    # the norm behind the sum: alpha x + y = (6, 10) with alpha 2, y (0, 2); root mean square sqrt(68)
    got = plain.post_norm(x, torch.tensor([[0.0, 2.0]], dtype=F64), torch.tensor([0.0, 1.0], dtype=F64), 2.0, 0.0)
    assert torch.allclose(got, torch.tensor([[6.0, 20.0]], dtype=F64) / math.sqrt(68.0))
    # the temperature steps where position + 1 is a multiple of `every`
    steps = plain.query_temperature(torch.tensor([0, 8, 9, 18, 19]), 0.5, 10)
    assert torch.allclose(steps, 1.0 + 0.5 * torch.log(torch.tensor([1.0, 1.0, 2.0, 2.0, 3.0], dtype=F64)))
    assert torch.allclose(plain.slopes(4), torch.tensor([0.25, 0.0625, 0.015625, 0.00390625], dtype=F64))
    assert plain.slopes(1)[0] == 2.0 ** -8
    # a window of two with one kept token: position 3 sees 0, 2 and 3
    assert plain.visible(4, 2, 1)[3].tolist() == [True, False, True, True]
    assert plain.visible(4, 2, 0)[3].tolist() == [False, False, True, True]
    assert plain.visible(3)[1].tolist() == [True, True, False]
    # a sink of a score's size takes half
    weights = plain.sink_softmax(torch.tensor([[[0.7]]], dtype=F64), torch.tensor([0.7], dtype=F64))
    assert torch.allclose(weights, torch.tensor([[[0.5]]], dtype=F64))
    # the bias falls from the score after the scale: one head (slope 2^-8) at distance 3
    q, k, v = torch.zeros(4, 1, 2, dtype=F64), torch.zeros(4, 1, 2, dtype=F64), torch.eye(4, dtype=F64)[:, None, :]
    distance = (torch.arange(4)[:, None] - torch.arange(4)[None, :]).to(F64)
    out = plain.grouped_attention(q, k, v, 0.5, torch.tensor([-1e4], dtype=F64), plain.visible(4),
                                  plain.slopes(1)[:, None, None] * distance)
    assert torch.allclose(out[3] / out[3, 3], torch.exp(-torch.tensor([3.0, 2.0, 1.0, 0.0], dtype=F64) / 256.0))
    # values are the keys as projected, before their norm: one token alone, its gate open, no sink
    eye, two = torch.eye(2, dtype=F64), torch.full((2,), 2.0, dtype=F64)
    w = {"p.q": eye, "p.k": eye * 3.0, "p.g": eye * 100.0, "p.o": eye, "p.q.norm": two, "p.k.norm": two,
         "p.sink": torch.tensor([-1e4], dtype=F64)}
    out = plain.key_value_attention(x, w, "p.", {"heads": 1, "kv_heads": 1, "dim": 2, "scale": 1.0}, 0.0)
    assert torch.allclose(out, 3.0 * x)
    # lightning attention: two tokens, one head, no other scale; one norm over all heads, a sigmoid gate
    wr = {"r.q": eye, "r.k": eye, "r.v": eye, "r.g": eye, "r.o": eye, "r.norm": two}
    h = torch.tensor([[1.0, 0.0], [1.0, 1.0]], dtype=F64)
    a = plain.silu(h)
    state = 0.5 * torch.outer(a[0], a[0]) + torch.outer(a[1], a[1])
    o = state.T @ a[1]
    want = o / torch.sqrt((o * o).mean()) * 2.0 * plain.sigmoid(h[1])
    assert torch.allclose(plain.lightning(h, wr, "r.", {"heads": 1, "dim": 2, "vdim": 2, "decay": [0.5]}, 0.0)[1], want)
    # the chosen experts' weights: a softmax over their logits alone
    chosen, share = plain.route(torch.tensor([[1.0, 2.0]], dtype=F64), {"m.router": torch.tensor([[0.0, 0.0], [1.0, 0.0], [0.0, 1.0]], dtype=F64)},
                                "m.", {"experts": 3, "top": 2})
    assert chosen[0].tolist() == [2, 1] and torch.allclose(share[0], torch.softmax(torch.tensor([2.0, 1.0], dtype=F64), -1))
    assert torch.equal(plain.dense_mlp(torch.tensor([[-2.0, 3.0]], dtype=F64), {"d.up": eye, "d.down": eye}, "d."),
                       torch.tensor([[0.0, 9.0]], dtype=F64))


def test_every_configuration_of_the_tests_runs_through_the_plain_implementation(tmp_path):
    for name, config in ALL.items():
        folder = make_folder(tmp_path / name, config, seed=1, dtype="float32")
        _, weights = plain.read_model(folder)
        assert torch.isfinite(plain.forward(config, weights, list(range(1, 30)))).all()
