"""Pedotar without a GPU: configuration -> model description, tensor names and shapes, the schedule of a repeated run
of layers, what the cache manager is asked for and when it gives pages of runs of positions back, configuration errors,
the padding of the selective scan's weights, fixed points of the plain implementation itself."""

import copy
import math

import pytest
import torch

import plain_pedotar as plain
from pedotar_configs import ALL, PEDOTAR_A, PEDOTAR_B, PEDOTAR_C, PEDOTAR_D, PEDOTAR_E, make_folder

from libmir_b200.cache import CacheManager
from libmir_b200.config.spec import PagedKv, SelectiveScanSpec, SoftmaxAttentionSpec, split_requirement
from libmir_b200.errors import ConfigError
from libmir_b200.models.decoder import CacheEntryPlan, DecoderModel
from libmir_b200.parts import BuildEnv, SelectiveScan, SoftmaxAttention
from libmir_b200.registry import architecture_of, build_spec
from libmir_b200.weights import parameter_specs

F64 = torch.float64
META = BuildEnv(torch.float32, torch.device("meta"))


def test_the_class_is_chosen_by_the_configuration():
    assert architecture_of(PEDOTAR_A) == "Pedotar"
    assert build_spec(PEDOTAR_A, None).architecture == "Pedotar"


def test_description_of_the_layers():
    spec = build_spec(PEDOTAR_A, None)
    assert all(layer.arrangement == "sandwich" for layer in spec.layers) and spec.head.tied and spec.head.scale == 1.0
    mixed, scan, latent, other, last = (layer.mixer for layer in spec.layers)
    assert (mixed.heads, mixed.kv_heads, mixed.head_dim, mixed.value_dim, mixed.scale) == (4, 2, 24, 40, 0.3)
    assert mixed.chunk == 19 and mixed.head_mix and mixed.window is None and mixed.position is None
    assert mixed.qk_norm and mixed.qk_norm_weight and mixed.qk_norm_span == "head" and not mixed.qkv_bias and not mixed.out_bias
    assert (scan.inner, scan.state, scan.dt_rank, scan.conv_taps) == (88, 16, 8, 4)
    assert (latent.heads, latent.head_dim, latent.rotary_dim, latent.value_dim, latent.kv_rank, latent.q_rank) == (3, 16, 8, 24, 48, 0)
    assert not latent.gate and latent.position.layout == "half" and latent.position.theta == 700.0 and latent.norm_eps == 1e-5
    assert other.chunk == 33 and (last.inner, last.state, last.conv_taps) == (64, 10, 3)
    for layer in spec.layers:
        norms = [layer.mixer_norm, layer.mixer_out_norm]
        if layer.feed_forward is not None:
            norms += [layer.feed_forward_norm, layer.feed_forward_out_norm]
        else:
            assert layer.feed_forward_norm is None and layer.feed_forward_out_norm is None
        assert all(norm.kind == "layer_norm" and norm.eps == 1e-5 and norm.size == 80 for norm in norms)
    assert spec.layers[0].feed_forward.kind == "swiglu" and spec.layers[0].feed_forward.intermediate_size == 72
    assert spec.layers[1].feed_forward is None


def test_a_repeated_run_of_layers_adds_the_embedding_before_every_pass_but_the_first():
    spec = build_spec(PEDOTAR_A, None)
    assert [(entry.layer, entry.opens_pass) for entry in spec.schedule] == \
        [(0, None), (1, 0), (2, None), (3, None), (1, 1), (2, None), (3, None), (4, None)]
    assert spec.loop.passes == 2 and spec.loop.step_tensor is None and spec.loop.add_embedding
    model = DecoderModel(spec, META)
    assert [model.pass_adds(entry) for entry in spec.schedule] == [False] * 4 + [True] + [False] * 3
    assert [entry.layer for entry in build_spec(PEDOTAR_B, None).schedule] == [0, 1, 2, 3, 4]
    assert [entry.layer for entry in build_spec(PEDOTAR_C, None).schedule] == [0, 1, 2, 1, 2]
    assert [entry.layer for entry in build_spec(PEDOTAR_E, None).schedule] == [0, 1, 1, 1, 1]
    assert build_spec(PEDOTAR_B, None).loop is None
    empty = dict(PEDOTAR_A, loop={"start": 2, "stop": 2, "times": 3})
    assert [entry.layer for entry in build_spec(empty, None).schedule] == [0, 1, 2, 3, 4]


def test_the_block_before_a_pass_adds_the_embedding_itself():
    """Only where nobody looks at the residual in between."""
    spec = build_spec(PEDOTAR_A, None)
    model, rows = DecoderModel(spec, META), object()
    opens = [model.rows_before(index + 1, model.blocks[entry.layer], rows) for index, entry in enumerate(spec.schedule)]
    assert opens == [None, None, None, rows, None, None, None, None]
    model.after_entry = lambda index, residual: None
    assert model.rows_before(4, model.blocks[3], rows) is None


def test_tensor_names_and_shapes():
    shapes = {name: tuple(param.shape) for name, param in parameter_specs(PEDOTAR_A).items()}
    assert shapes["embed"] == (203, 80) and "head" not in shapes
    assert shapes["final.norm"] == (80,) and shapes["final.norm.b"] == (80,)
    for norm in ("norm1", "norm1b", "norm2", "norm2b"):
        assert shapes[f"l0.{norm}"] == (80,) and shapes[f"l0.{norm}.b"] == (80,)
    assert "l1.norm2" not in shapes and "l1.norm2b" not in shapes and shapes["l1.norm1b.b"] == (80,)
    assert shapes["l0.mix.q"] == (96, 80) and shapes["l0.mix.k"] == (48, 80) and shapes["l0.mix.v"] == (80, 80)
    assert shapes["l0.mix.q.norm"] == (24,) and shapes["l0.mix.k.norm"] == (24,) and shapes["l0.mix.talk"] == (4, 4)
    assert shapes["l0.mix.o"] == (80, 160) and "l0.mix.q.b" not in shapes
    assert shapes["l0.mlp.gate"] == (72, 80) and shapes["l0.mlp.up"] == (72, 80) and shapes["l0.mlp.down"] == (80, 72)
    assert shapes["l1.mix.in"] == (176, 80) and shapes["l1.mix.conv"] == (88, 4) and shapes["l1.mix.conv.b"] == (88,)
    assert shapes["l1.mix.x"] == (40, 88) and shapes["l1.mix.dt"] == (88, 8) and shapes["l1.mix.dt.b"] == (88,)
    assert shapes["l1.mix.A_log"] == (88, 16) and shapes["l1.mix.D"] == (88,) and shapes["l1.mix.o"] == (80, 88)
    assert shapes["l2.mix.q"] == (72, 80) and shapes["l2.mix.dkv"] == (56, 80) and shapes["l2.mix.dkv.norm"] == (48,)
    assert shapes["l2.mix.uk"] == (48, 48) and shapes["l2.mix.uv"] == (72, 48) and shapes["l2.mix.o"] == (80, 72)
    assert "l2.mix.g" not in shapes and "l2.mix.dq" not in shapes
    assert not any(name.endswith(("qkv_proj.weight", "sinks")) for name in shapes)


@pytest.mark.parametrize("change,needle", [
    (lambda c: c.pop("width"), "width"),
    (lambda c: c["norm"].pop("eps"), "eps"),
    (lambda c: c["layers"][0].update(type="attention_9"), "attention_9"),
    (lambda c: c["layers"][0]["mixer"].pop("scale"), "scale"),
    (lambda c: c["layers"][0]["mixer"].update(kv_heads=3), "kv_heads"),
    (lambda c: c["layers"][0]["mixer"].pop("mask"), "mask"),
    (lambda c: c["layers"][0]["mixer"]["mask"].update(size=0), "size"),
    (lambda c: c["layers"][1]["mixer"].pop("dt_rank"), "dt_rank"),
    (lambda c: c["layers"][1]["mixer"].update(conv=0), "conv"),
    (lambda c: c["layers"][2]["mixer"]["rot"].update(dims=6), "rot.dims"),
    (lambda c: c["layers"][2]["mixer"].pop("kv_rank"), "kv_rank"),
    (lambda c: c["layers"][0]["mlp"].update(kind="other"), "other"),
    (lambda c: c["loop"].update(stop=9), "loop"),
])
def test_configuration_errors_name_what_is_wrong(change, needle):
    config = copy.deepcopy(PEDOTAR_A)
    change(config)
    with pytest.raises(ConfigError) as error:
        build_spec(config, None)
    assert needle in str(error.value)


# ------------------------------------------------------------------------------ cache
def test_what_the_cache_manager_is_asked_for():
    plan = DecoderModel(build_spec(PEDOTAR_A, None), META).cache_plan()
    assert len(plan) == 8 and all(item.writes for item in plan)          # every run of a layer has a cache of its own
    paged, states = split_requirement(plan[0].requirement)
    assert (paged.kv_heads, paged.head_dim, paged.value_dim, paged.window, paged.chunk) == (2, 24, 40, None, 19) and not states
    paged, states = split_requirement(plan[1].requirement)
    assert paged is None and [state.shape for state in states] == [(88, 16), (3, 88)]
    paged, states = split_requirement(plan[2].requirement)
    assert (paged.kv_heads, paged.head_dim, paged.value_dim, paged.chunk) == (1, 56, 0, None) and not states
    manager = CacheManager(plan, page_size=8, num_pages=40, max_requests=2)
    assert len(manager.groups) == 3 and sorted(manager.state_entries) == [1, 4, 7]
    assert [group.chunk for group in manager.groups] == [19, None, 33] and [group.releases for group in manager.groups] == [True, False, True]


@pytest.mark.parametrize("chunk,page", [(16, 4), (19, 4), (5, 8), (1, 2), (8, 8)])
def test_pages_of_runs_that_are_over_are_given_back_and_no_others(chunk, page):
    requirement = PagedKv(1, 4, None, None, 0, chunk)
    manager = CacheManager([CacheEntryPlan(0, requirement, 0, True)], page_size=page, num_pages=60, max_requests=1)
    sequence = manager.admit("a")
    length = 0
    for portion in (3, 1, 1, 7, 2, 11, 1, 1, 1, 30, 2):
        manager.grow(sequence, length + portion)
        table = sequence.tables[0]
        for position in range(length, length + portion):               # whatever these queries see is there
            for key in range(position // chunk * chunk, position + 1):
                assert table[key // page] >= 0, (position, key)
        length += portion
        manager.commit(sequence, length)
        manager.check()
        first_seen = length // chunk * chunk                             # by the next query
        for block, held in enumerate(table):
            assert (held >= 0) == ((block + 1) * page > first_seen), (length, block)
    assert manager.groups[0].pool.high_water <= manager.peak_pages(length, manager.groups[0], 30)
    manager.release("a")
    assert manager.groups[0].pool.available == 60


def test_prefixes_are_not_remembered_where_runs_of_positions_give_pages_back():
    plan = [CacheEntryPlan(0, PagedKv(1, 4, chunk=8), 0, True)]
    assert CacheManager(plan, 4, 8, 1, prefix_cache=True).prefix is None
    plan = [CacheEntryPlan(0, PagedKv(1, 4), 0, True)]
    assert CacheManager(plan, 4, 8, 1, prefix_cache=True).prefix is not None


# ------------------------------------------------------------------------------ parts
def test_mixed_heads_take_plain_scores_only():
    for change in (dict(sinks=True), dict(fixed_sink=0.0), dict(gate=True), dict(softcap=3.0), dict(window=8, keep_first=2)):
        with pytest.raises(ValueError):
            SoftmaxAttention(SoftmaxAttentionSpec(hidden_size=8, heads=2, kv_heads=1, head_dim=4, head_mix=True, **change), META)


def test_the_scans_weights_are_padded_to_eights_without_changing_anything():
    """Bound weights of odd sizes give what the stored ones give: the packed products in float64, zeros elsewhere."""
    spec = SelectiveScanSpec(hidden_size=10, inner=13, state=5, dt_rank=3, conv_taps=2)
    part = SelectiveScan(spec, BuildEnv(torch.float32, torch.device("cpu")))
    assert (part.channels, part.rank, part.columns) == (16, 8, 8)
    generator = torch.Generator().manual_seed(0)
    tensors = {name: torch.randn(param.shape, generator=generator) for name, param in part.parameters().items()}
    part.bind(tensors)
    h, x, low = (torch.randn(4, width, generator=generator) for width in (10, 13, 3))
    packed = h @ part.w_in.T
    assert torch.allclose(packed[:, :13], h @ tensors["in"][:13].T) and torch.allclose(packed[:, 16:29], h @ tensors["in"][13:].T)
    assert (packed[:, 13:16] == 0).all() and (packed[:, 29:] == 0).all()
    wide = torch.cat([x, torch.zeros(4, 3)], 1)
    second = wide @ part.w_x.T
    want = x @ tensors["x"].T
    assert torch.allclose(second[:, :3], want[:, :3]) and torch.allclose(second[:, 8:13], want[:, 3:8], atol=1e-6)
    assert torch.allclose(second[:, 16:21], want[:, 8:], atol=1e-6) and (second[:, 21:] == 0).all()
    step = torch.cat([low, torch.zeros(4, 5)], 1) @ part.w_dt.T
    assert torch.allclose(step[:, :13], low @ tensors["dt"].T, atol=1e-6)
    assert torch.allclose(part.rates[:13], -torch.exp(tensors["A_log"]) / math.log(2.0)) and (part.rates[13:] == 0).all()
    assert (part.w_conv[13:] == 0).all() and (part.conv_bias[13:] == 0).all() and (part.w_o[:, 13:] == 0).all()


# ------------------------------------------------------------------------------ the plain implementation
def test_fixed_points_of_the_plain_implementation():
    x = torch.arange(12, dtype=F64).view(4, 3)
    assert torch.equal(plain.short_convolution(x, torch.tensor([[0.0, 1.0]] * 3), torch.zeros(3)), x)
    shifted = plain.short_convolution(x, torch.tensor([[1.0, 0.0]] * 3), torch.zeros(3))
    assert torch.equal(shifted[1:], x[:-1]) and (shifted[0] == 0).all()
    # without decay (a = 0) and with unit steps the state sums its inputs
    ones = torch.ones(4, 3, dtype=F64)
    y, state = plain.selective_scan(x, ones, torch.zeros(3, 1, dtype=F64), torch.ones(4, 1, dtype=F64), torch.ones(4, 1, dtype=F64),
                                    torch.zeros(3, dtype=F64))
    assert torch.equal(y, x.cumsum(0)) and torch.equal(state[:, 0], x.sum(0))
    # two halves of a sequence, the state carried over, are the whole
    a = -torch.rand(3, 2, dtype=F64)
    b, c, d = torch.randn(4, 2, dtype=F64), torch.randn(4, 2, dtype=F64), torch.randn(3, dtype=F64)
    whole, end = plain.selective_scan(x, ones * 0.3, a, b, c, d)
    first, middle = plain.selective_scan(x[:2], ones[:2] * 0.3, a, b[:2], c[:2], d)
    second, last = plain.selective_scan(x[2:], ones[2:] * 0.3, a, b[2:], c[2:], d, middle)
    assert torch.allclose(torch.cat([first, second]), whole) and torch.allclose(last, end)
    # a rotation keeps lengths; position 0 does not turn
    v = torch.randn(5, 2, 6, dtype=F64)
    turned = plain.rotate(v, 6, 50.0)
    assert torch.allclose(turned.norm(dim=-1), v.norm(dim=-1)) and torch.equal(turned[0], v[0])
    # heads mixed by the identity are heads that are not mixed; a run of one position sees itself alone
    q, k, v = torch.randn(7, 4, 3, dtype=F64), torch.randn(7, 2, 3, dtype=F64), torch.randn(7, 2, 5, dtype=F64)
    assert torch.allclose(plain.talking_attention(q, k, v, 0.7, torch.eye(4)), plain.talking_attention(q, k, v, 0.7))
    assert torch.allclose(plain.talking_attention(q, k, v, 0.7, None, 1), v.repeat_interleave(2, 1))
    assert plain.visible(6, 4).tolist()[5] == [False] * 4 + [True] * 2
    z = torch.tensor([-40.0, -1.0, 0.0, 1.0, 35.0], dtype=F64)
    assert torch.allclose(plain.softplus(z), torch.nn.functional.softplus(z))


@pytest.mark.parametrize("name", sorted(ALL))
def test_a_prefix_of_a_sequence_has_the_logits_of_the_sequence(tmp_path, name):
    """Causality of the plain implementation, on folders that the writer made."""
    folder = make_folder(tmp_path, ALL[name], seed=1, dtype="float32")
    config, weights = plain.read_model(folder)
    ids = [(7 * i + 3) % config["vocab"] for i in range(40)]
    whole = plain.forward(config, weights, ids)
    assert torch.allclose(plain.forward(config, weights, ids[:23]), whole[:23], atol=1e-9)
    assert whole.shape == (40, config["vocab"]) and torch.isfinite(whole).all()
