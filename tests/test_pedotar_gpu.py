"""Pedotar on the GPU against the plain implementation (tests/plain_pedotar.py): every mechanism's kernel alone, then
whole models through the engine's step function, cache manager and scheduler: prompts whole, token by token, in
portions down to two tokens, in batches of unequal requests, with pages and slots that change hands, with keys far
away, at page borders and on either side of the edge of a run of positions, in long decoding, and greedy generation
through the entry point."""

import json
import math

import numpy as np
import pytest
import torch

import plain_pedotar as plain
from helpers import TOL, Trace, random_ids, run_trace
from pedotar_configs import ALL, PAGE_SIZES, latent, make_folder, mixed, random_config, scan

pytestmark = pytest.mark.gpu
F64 = torch.float64
BF16 = torch.bfloat16
DTYPES = [(torch.float32, 2e-6), (torch.bfloat16, 8e-3)]


def device():
    return torch.device("cuda", 0)


def close(got, want, tol, what=""):
    got = got.detach().double().cpu() if isinstance(got, torch.Tensor) else torch.as_tensor(got, dtype=F64)
    want = want.detach().double().cpu() if isinstance(want, torch.Tensor) else torch.as_tensor(want, dtype=F64)
    error = (got - want).abs().max().item()
    bound = tol * max(1.0, want.abs().max().item())
    assert math.isfinite(error) and error <= bound, f"{what}: max |diff| {error:.3e} > {bound:.3e}"


def relative_error(got, want):
    got, want = np.asarray(got, dtype=np.float64), np.asarray(want, dtype=np.float64)
    return np.sqrt(((got - want) ** 2).mean(-1)) / np.sqrt((want ** 2).mean(-1))


def close_logits(got, want, dtype, what=""):
    """Logits [positions, vocab] of a whole model, judged by each position's relative root-mean-square error: 2e-4 in
    float32, the helpers' tolerance in bfloat16 at nine positions in ten and twice that at all of them."""
    relative = relative_error(got, want)
    assert np.isfinite(relative).all(), f"{what}: not finite"
    if dtype == "float32":
        assert relative.max() <= 2e-4, f"{what}: {relative.max():.3e} at position {int(relative.argmax())}"
    else:
        assert np.quantile(relative, 0.9) <= TOL[dtype] and relative.max() <= 2 * TOL[dtype], \
            f"{what}: 90% {np.quantile(relative, 0.9):.3e}, max {relative.max():.3e} at {int(relative.argmax())}"


def on_device(tensor, dtype=None):
    return tensor.to(device=device(), dtype=dtype or tensor.dtype).contiguous()


def ints(values):
    return torch.as_tensor(np.asarray(values, dtype=np.int32), device=device())


# ------------------------------------------------------------------------------ whole models
def load(folder, dtype, page_size, pages, requests=4, graphs=False):
    from libmir_b200 import CacheConfig, CudaConfig, Library, RuntimeConfig, SchedulerConfig
    runtime = RuntimeConfig(kv_cache=CacheConfig(block_size=page_size, block_count=pages),
                            scheduler=SchedulerConfig(max_batch_requests=requests),
                            cuda=CudaConfig(decode_graphs=graphs), dtype=dtype)
    return Library(runtime).load(folder)


def reference(folder, ids):
    config, weights = plain.read_model(folder)
    return plain.forward(config, weights, list(ids)).numpy()


def feed(model, name, ids, cuts):
    """Feed `ids` in portions of the given sizes (the last repeated), wanting every position; returns logits [n, V]."""
    from libmir_b200 import StepEntry
    model.admit(name)
    out, cursor, turn = [], 0, 0
    while cursor < len(ids):
        size = min(cuts[min(turn, len(cuts) - 1)], len(ids) - cursor)
        result = model.step([StepEntry(name, ids[cursor:cursor + size], range(size))])
        out.append(result.logits.float().cpu().numpy().copy())
        cursor += size
        turn += 1
    model.release(name)
    return np.concatenate(out)


@pytest.mark.parametrize("name", ["A", "B", "E"])
def test_the_residual_after_every_run_of_a_layer(tmp_path, name):
    """One prompt in 32-bit: the residual after each run of a layer (a repeated layer counts every time) against the
    plain implementation's, so that a fault shows at the run that has it."""
    from libmir_b200 import StepEntry
    config = ALL[name]
    folder = make_folder(tmp_path, config, seed=2, dtype="float32")
    ids = random_ids(np.random.default_rng(1), config["vocab"], 60)
    plain_config, weights = plain.read_model(folder)
    _, want = plain.forward(plain_config, weights, ids, want_layers=True)
    model = load(folder, "float32", PAGE_SIZES[name], 40)
    seen = []
    model.decoder.after_entry = lambda index, residual: seen.append(residual.cpu())
    model.admit("x")
    model.step([StepEntry("x", ids, [0])])
    model.decoder.after_entry = None
    assert len(seen) == want.shape[0] == len(plain.layer_order(config))
    for run, (got, expected) in enumerate(zip(seen, want)):
        close(got, expected, 2e-5, f"after layer run {run}")


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("name", sorted(ALL))
def test_whole_prompts_token_by_token_and_portions(tmp_path, name, dtype):
    """A prompt whole; the same token by token from its first token (150 single steps: long decoding, windows that
    pass over decoded tokens, the first tokens of a sequence); in portions of changing size down to two tokens; and
    most of it whole with the rest decoded."""
    config = ALL[name]
    folder = make_folder(tmp_path, config, seed=3, dtype=dtype)
    ids = random_ids(np.random.default_rng(7), config["vocab"], 150)
    want = reference(folder, ids)
    model = load(folder, dtype, PAGE_SIZES[name], 60)
    whole = feed(model, "whole", ids, [len(ids)])
    close_logits(whole, want, dtype, f"{name}/{dtype} whole")
    single = feed(model, "single", ids, [1])
    close_logits(single, want, dtype, f"{name}/{dtype} token by token")
    portions = feed(model, "portions", ids, [2, 3, 1, 7, 2, 16, 5, 2, 33, 1, 2, 9])
    close_logits(portions, want, dtype, f"{name}/{dtype} portions")
    late = feed(model, "late", ids, [118, 1])
    close_logits(late, want, dtype, f"{name}/{dtype} prompt then decoding")
    if dtype == "float32":
        # 32-bit results do not depend on the cut at all: attention reduces a query's keys in an order that depends on
        # its position alone, products and norms reduce in one fixed order, an expert pair's row does not depend on
        # which tile it shares with whom
        assert np.array_equal(whole, single) and np.array_equal(whole, portions) and np.array_equal(whole, late)
    for group in model.cache_stats()["groups"]:
        assert group["free"] == group["pages"]


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("name", ["A", "C", "D"])
def test_batches_of_unequal_requests_with_pages_and_slots_that_change_hands(tmp_path, name, dtype):
    """Up to three live requests of unequal lengths, portions of some beside single tokens of others, requests that
    sit a step out, in a pool so small that pages and slots are used again; every request against itself alone."""
    from libmir_b200 import StepEntry
    config = ALL[name]
    folder = make_folder(tmp_path, config, seed=5, dtype=dtype)
    rng = np.random.default_rng(11)
    lengths = [70, 31, 96, 18, 55, 40, 77]
    requests = [random_ids(rng, config["vocab"], n) for n in lengths]
    want = [reference(folder, ids) for ids in requests]
    page = PAGE_SIZES[name]
    model = load(folder, dtype, page, 3 * (-(-96 // page)) + 2, requests=3)
    queue, live, got = list(range(len(requests))), {}, {i: [] for i in range(len(requests))}
    while queue or live:
        while queue and len(live) < 3:
            index = queue.pop(0)
            model.admit(f"r{index}")
            live[index] = 0
        entries, ended = [], []
        for index in list(live):
            cursor, ids = live[index], requests[index]
            if len(live) > 1 and rng.random() < 0.25:
                continue
            decode_from = max(2, len(ids) - 20)
            size = 1 if cursor >= decode_from else min(int(rng.integers(2, 19)), decode_from - cursor)
            entries.append(StepEntry(f"r{index}", ids[cursor:cursor + size], range(size)))
            live[index] = cursor + size
            if live[index] == len(ids):
                ended.append(index)
        if not entries:
            continue
        result = model.step(entries)
        logits, at = result.logits.float().cpu().numpy(), 0
        for entry in entries:
            got[int(entry.request_id[1:])].append(logits[at:at + len(entry.tokens)].copy())
            at += len(entry.tokens)
        for index in ended:
            model.release(f"r{index}")
            del live[index]
        model.cache.check()
    if dtype == "float32":
        for index in range(len(requests)):
            close_logits(np.concatenate(got[index]), want[index], dtype, f"{name}/{dtype} request {index} in a mixed batch")
    else:       # (the share of positions is taken over all requests: the shortest has eighteen)
        close_logits(np.concatenate([np.concatenate(got[index]) for index in range(len(requests))]), np.concatenate(want),
                     dtype, f"{name}/{dtype} requests in mixed batches")
    stats = model.cache_stats()
    for group in stats["groups"]:
        assert group["free"] == group["pages"] and group["reused"] > 0


