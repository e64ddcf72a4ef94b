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
    float32, the helpers' tolerance in bfloat16 at nine positions in ten and five times that at all of them (a layer norm
    of a narrow row with little spread multiplies what rounding left in it)."""
    relative = relative_error(got, want)
    assert np.isfinite(relative).all(), f"{what}: not finite"
    if dtype == "float32":
        assert relative.max() <= 2e-4, f"{what}: {relative.max():.3e} at position {int(relative.argmax())}"
    else:
        assert np.quantile(relative, 0.9) <= TOL[dtype] and relative.max() <= 5 * TOL[dtype], \
            f"{what}: 90% {np.quantile(relative, 0.9):.3e}, max {relative.max():.3e} at {int(relative.argmax())}"


def on_device(tensor, dtype=None):
    return tensor.to(device=device(), dtype=dtype or tensor.dtype).contiguous()


def ints(values):
    return torch.as_tensor(np.asarray(values, dtype=np.int32), device=device())


# ------------------------------------------------------------------------------ norms around a sublayer
@pytest.mark.parametrize("dtype,tol", DTYPES)
@pytest.mark.parametrize("width", [50, 96, 1028, 4608])
def test_a_branch_is_normed_and_added_and_the_new_residual_normed_for_its_reader(dtype, tol, width):
    from libmir_b200 import kernels
    generator = torch.Generator().manual_seed(width)
    normal = lambda *shape: torch.randn(*shape, generator=generator)
    tokens = 9
    x, y, extra = normal(tokens, width) * 2.0 + 0.5, normal(tokens, width) * 30.0 - 4.0, normal(tokens, width)
    weight, bias, next_weight, next_bias = (normal(width) for _ in range(4))
    for rows in (None, extra):
        want = x.double() + plain.layer_norm(y.double(), weight, bias, 1e-5)
        if rows is not None:
            want = want + rows.double()
        residual, out = on_device(x), torch.empty(tokens, width, dtype=dtype, device=device())
        kernels.add_layer_norm(residual, on_device(y), on_device(weight), on_device(bias), 1e-5,
                               on_device(rows) if rows is not None else None, on_device(next_weight), on_device(next_bias),
                               1e-6, out)
        close(residual, want, 2e-6, "the residual")
        close(out, plain.layer_norm(want, next_weight, next_bias, 1e-6), 4 * tol, "its norm")
        alone = on_device(x)
        kernels.add_layer_norm(alone, on_device(y), on_device(weight), on_device(bias), 1e-5,
                               on_device(rows) if rows is not None else None)
        assert torch.equal(alone, residual)


# ------------------------------------------------------------------------------ recurrence
def batch_of(portions, slots, begins):
    """(row_of_token, query_starts, state_slots, positions) of rows that bring `portions` tokens from `begins` on."""
    rows = np.repeat(np.arange(len(portions)), portions)
    positions = np.concatenate([np.arange(b, b + n) for b, n in zip(begins, portions)])
    return ints(rows), ints(np.concatenate([[0], np.cumsum(portions)])), ints(slots), ints(positions)


PORTIONS = ([1, 2], [2, 1], [1, 1], [3, 1], [1, 5], [40, 2], [7, 66], [1, 1], [2, 70])


@pytest.mark.parametrize("dtype,tol", DTYPES)
@pytest.mark.parametrize("taps,channels", [(1, 64), (2, 64), (3, 72), (4, 272), (5, 64), (4, 30), (2, 12)])
def test_short_convolution_with_a_bias_in_the_activations_type(dtype, tol, taps, channels):
    """Two requests in portions of 1, 2, 3 and more tokens, in state slots 2 and 0: 16-byte pieces up to four taps, the
    general kernel for other sizes; the same bits in 32-bit results of the two."""
    from libmir_b200 import kernels
    generator = torch.Generator().manual_seed(taps + channels)
    lengths = [sum(p[r] for p in PORTIONS) for r in range(2)]
    inputs = [torch.randn(n, channels, generator=generator).to(dtype) for n in lengths]
    weight = (torch.randn(channels, taps, generator=generator) * 0.7).to(dtype)
    bias = torch.randn(channels, generator=generator)
    want = [plain.silu(plain.short_convolution(x.double(), weight.double(), bias)) for x in inputs]
    width = channels + 16
    for out_dtype in {dtype, torch.float32}:
        tail = torch.zeros(3, taps - 1, channels, device=device())
        got, cursors = [[], []], [0, 0]
        for portions in PORTIONS:
            rows = torch.full((sum(portions), width), 77.0, dtype=dtype)
            at = 0
            for r, count in enumerate(portions):
                rows[at:at + count, 8:8 + channels] = inputs[r][cursors[r]:cursors[r] + count]
                at += count
            rows = rows.to(device())
            batch = batch_of(portions, [2, 0], cursors)
            out = torch.empty(sum(portions), channels, dtype=out_dtype, device=device())
            kernels.short_conv_silu(rows[:, 8:8 + channels], weight.to(device()), tail, *batch, out, bias=on_device(bias),
                                    single_tokens_only=all(n == 1 for n in portions))
            at = 0
            for r, count in enumerate(portions):
                got[r].append(out[at:at + count].cpu())
                cursors[r] += count
                at += count
        for r in range(2):
            close(torch.cat(got[r]), want[r], tol if out_dtype == dtype else 2e-6, f"request {r}")
        assert torch.all(tail[1] == 0), "the state of a slot nobody used was written"
        for r, slot in ((0, 2), (1, 0)):
            if taps > 1:
                assert torch.equal(tail[slot].cpu(), inputs[r][-(taps - 1):].float()), "the last inputs are kept"


@pytest.mark.parametrize("dtype,tol", DTYPES)
@pytest.mark.parametrize("channels,n", [(64, 16), (40, 1), (200, 24), (8, 7), (72, 4), (64, 33), (32, 64), (16, 100), (8, 256)])
def test_selective_scan_carries_its_state_between_portions(dtype, tol, channels, n):
    """Two requests in portions, in state slots 2 and 0; step sizes from almost nothing to large ones (a state that
    stays, a state that is forgotten at once); the state after it in 32-bit, other slots untouched, and in 32-bit the
    same bits as token by token."""
    from libmir_b200 import kernels
    generator = torch.Generator().manual_seed(channels * 300 + n)
    normal = lambda *shape: torch.randn(*shape, generator=generator)
    columns = -(-n // 8) * 8
    lengths = [sum(p[r] for p in PORTIONS) for r in range(2)]
    x = [normal(t, channels).to(dtype) for t in lengths]
    z = [normal(t, channels).to(dtype) for t in lengths]
    raw = [normal(t, channels) * 3.0 - 2.0 for t in lengths]
    b, c = ([torch.cat([normal(t, n), torch.full((t, columns - n), 55.0)], 1).to(dtype) for t in lengths] for _ in range(2))
    bias, skip = normal(channels) - 1.0, normal(channels)
    a = -torch.rand(channels, n, generator=generator) * 3.0 - 0.01
    rates = (a.double() / math.log(2.0)).float()
    want, final = [], []
    for r in range(2):
        y, s = plain.selective_scan(x[r].double(), plain.softplus(raw[r].double() + bias.double()), a.double(),
                                    b[r][:, :n].double(), c[r][:, :n].double(), skip.double())
        want.append(y * plain.silu(z[r].double()))
        final.append(s)

    def run(cuts):
        state = torch.zeros(3, channels, n, device=device())
        got, cursors = [[], []], [0, 0]
        for portions in cuts:
            take = lambda source: torch.cat([source[r][cursors[r]:cursors[r] + portions[r]] for r in range(2)]).to(device())
            wide = torch.cat([take(x), take(z)], 1)              # column ranges of wider rows
            low = torch.cat([take(b), take(c)], 1)
            _, starts, slots, positions = batch_of(portions, [2, 0], cursors)
            out = torch.empty(sum(portions), channels, dtype=dtype, device=device())
            kernels.selective_scan(wide[:, :channels], take(raw), on_device(bias), low[:, :columns], low[:, columns:],
                                   wide[:, channels:], on_device(rates), on_device(skip), state, starts, slots, positions, out)
            for r, rows in enumerate(out.split(portions)):
                got[r].append(rows.cpu())
                cursors[r] += portions[r]
        return [torch.cat(rows) for rows in got], state
    got, state = run(PORTIONS)
    for r, slot in ((0, 2), (1, 0)):
        close(got[r], want[r], 4 * tol, f"request {r}")
        close(state[slot], final[r], 5e-6, f"the state of request {r}")
    assert torch.all(state[1] == 0)
    shorter = min(lengths)
    again, _ = run([[1, 1]] * shorter)
    for r in range(2):
        assert torch.equal(again[r], got[r][:shorter]), "token by token"


# ------------------------------------------------------------------------------ latent attention
@pytest.mark.parametrize("dtype,tol", DTYPES)
@pytest.mark.parametrize("heads,dim,rot,rank", [(3, 16, 8, 48), (1, 5, 2, 10), (5, 40, 64, 160)])
def test_the_latent_is_normed_and_queries_and_shared_key_rotated_in_one_launch(dtype, tol, heads, dim, rot, rank):
    from libmir_b200 import kernels
    generator = torch.Generator().manual_seed(rank)
    tokens, per_head = 7, dim + rot
    offset = heads * per_head + 3
    packed = torch.randn(tokens, offset + rank + rot, generator=generator).to(dtype)
    norm = 1.0 + 0.3 * torch.randn(rank, generator=generator)
    positions, slots = [5, 6, 0, 1, 4000, 9, 2], [3, 0, 8, -1, 5, 6, 2]
    frequencies = torch.tensor([700.0 ** (-2.0 * i / rot) for i in range(rot // 2)], dtype=torch.float32)
    rows = on_device(packed)
    q = rows[:, :heads * per_head].unflatten(1, (heads, per_head))
    folded = torch.full((tokens, heads, rank + rot), 7.0, dtype=dtype, device=device())
    pages = torch.full((9, 1, rank + rot), 77.0, dtype=dtype, device=device())
    kernels.latent_prepare(rows, 0, 0, offset, rank, rot, None, on_device(norm), 1e-5, ints(positions), ints(slots),
                           on_device(frequencies), 1.0, False, None, pages, (q[:, :, dim:], folded[:, :, rank:]))
    source = packed.double()
    at = torch.tensor(positions)
    turned = plain.rotate(source[:, :heads * per_head].view(tokens, heads, per_head)[..., dim:], rot, 700.0, at)
    close(folded[:, :, rank:], turned, tol, "rotated queries")
    assert (folded[:, :, :rank] == 7.0).all()
    latent_rows = plain.rms_norm(source[:, offset:offset + rank], norm, 1e-5)
    shared = plain.rotate(source[:, offset + rank:].view(tokens, 1, rot), rot, 700.0, at)[:, 0]
    written = [t for t in range(tokens) if slots[t] >= 0]
    close(pages[[slots[t] for t in written], 0], torch.cat([latent_rows, shared], 1)[written], 2 * tol, "cache rows")
    assert (pages[[s for s in range(9) if s not in slots]] == 77.0).all()


def pool_of(keys, values, page, rng, dtype):
    """Scatter each request's keys and values into a shuffled pool of pages; garbage elsewhere.  Returns the pool
    tensors and the block table [requests, width]."""
    needs = [-(-k.shape[0] // page) for k in keys]
    total = sum(needs) + 5
    order = rng.permutation(total)
    width = max(needs)
    table = np.full((len(keys), width), -1, dtype=np.int32)
    k_pool = torch.full((total * page, keys[0].shape[1], keys[0].shape[2]), 1e4, dtype=torch.float32)
    v_pool = torch.full((total * page, values[0].shape[1], values[0].shape[2]), 1e4, dtype=torch.float32)
    at = 0
    for r, (k, v) in enumerate(zip(keys, values)):
        for p in range(needs[r]):
            page_id = int(order[at]); at += 1
            table[r, p] = page_id
            n = min(page, k.shape[0] - p * page)
            k_pool[page_id * page:page_id * page + n] = k[p * page:p * page + n]
            v_pool[page_id * page:page_id * page + n] = v[p * page:p * page + n]
    return on_device(k_pool, dtype), on_device(v_pool, dtype), ints(table)


# ------------------------------------------------------------------------------ attention with mixed heads
MIXED_CASES = [
    # dtype, heads, kv_heads, dim, vdim, page, window, chunk, path
    (torch.float32, 4, 2, 24, 40, 8, None, 37, "reference"),
    (torch.float32, 3, 1, 10, 6, 4, None, 50, "reference"),
    (torch.float32, 5, 5, 64, 16, 16, 29, None, "reference"),
    (BF16, 6, 3, 32, 16, 16, None, 110, "split"),
    (BF16, 7, 7, 8, 200, 8, None, 130, "split"),
    (BF16, 9, 1, 256, 64, 16, None, None, "split"),
    (BF16, 7, 7, 64, 64, 16, None, 90, "tiles"),
    (BF16, 1, 1, 64, 128, 4, None, 64, "tiles"),
    (BF16, 12, 3, 128, 128, 16, None, 50, "tiles"),
    (BF16, 32, 8, 128, 64, 32, None, 101, "tiles"),
    (BF16, 32, 8, 128, 128, 16, None, 150, "tiles"),
    (BF16, 6, 2, 128, 128, 8, 140, None, "tiles"),
    (BF16, 24, 1, 128, 128, 16, None, None, "tiles"),
    (BF16, 16, 4, 128, 128, 32, None, 128, "tiles"),
    (BF16, 16, 2, 64, 64, 8, 77, None, "tiles"),
    (BF16, 20, 20, 128, 128, 8, None, None, "tiles"),
    (BF16, 4, 4, 64, 64, 16, None, 1, "tiles"),
]


@pytest.mark.parametrize("dtype,heads,kv_heads,dim,vdim,page,window,chunk,path", MIXED_CASES)
def test_mixed_heads_where_keys_at_the_edges_of_a_run_stand_out(dtype, heads, kv_heads, dim, vdim, page, window, chunk, path):
    """Three requests of unequal lengths in a shuffled pool.  For queries in the middle and at the end of runs of
    positions, the first key that is seen, the one before it (more strongly: it must not be seen) and the keys on either
    side of a page border stand out: a run that is one token off, or a page read from the wrong place, changes the
    result.  Portions that start in mid-request and single tokens, the tile kernels with all weights in memory and in
    slabs, the split-key kernels, and the reference kernel."""
    from libmir_b200 import kernels
    rng = np.random.default_rng(dim + page)
    generator = torch.Generator().manual_seed(dim * 3 + page)
    lengths = [300, 19, 131]
    scale = 1.0 / math.sqrt(dim)
    talk = torch.randn(heads, heads, generator=generator) * 0.7
    qs, ks, vs, wants = [], [], [], []
    for n in lengths:
        q = torch.randn(n, heads, dim, generator=generator)
        k = torch.randn(n, kv_heads, dim, generator=generator)
        v = torch.randn(n, kv_heads, vdim, generator=generator)
        edge = (n - 1) // chunk * chunk if chunk else 0
        for query in {n - 1, n - 2, edge, max(0, edge - 1), n // 2}:
            direction = q[query, 0] / q[query, 0].norm()
            inside = query // chunk * chunk if chunk else (max(0, query - window + 1) if window else 0)
            k[inside, 0] = direction * 4.0
            if inside > 0:
                k[inside - 1, 0] = direction * 12.0              # just outside: must not be seen
            border = (query // page) * page
            if inside < border:
                k[border, 0] += direction * 3.0
                k[border - 1, 0] += direction * 2.0
        q, k, v = (t.to(dtype).double() for t in (q, k, v))
        if window:
            seen = plain.visible(n) & (torch.arange(n)[None, :] > torch.arange(n)[:, None] - window)
            weights = plain.softmax_over(torch.einsum("ihd,jhd->hij", q, k.repeat_interleave(heads // kv_heads, 1)) * scale, seen[None])
            want = torch.einsum("hg,gij,jhd->ihd", talk.double(), weights, v.repeat_interleave(heads // kv_heads, 1))
        else:
            want = plain.talking_attention(q, k, v, scale, talk, chunk)
        qs.append(q); ks.append(k); vs.append(v); wants.append(want.reshape(n, heads * vdim))
    k_pool, v_pool, table = pool_of(ks, vs, page, rng, dtype)
    mix = on_device(talk)
    tol = 2e-5 if dtype == torch.float32 else 2e-2
    scratch = lambda shape, kind: torch.empty(tuple(shape), dtype=kind, device=device())
    packed = lambda rows_of: on_device(torch.cat([torch.cat([qs[r][a:b].reshape(b - a, -1) for r, a, b in rows_of]),
                                                  torch.zeros(sum(b - a for _, a, b in rows_of), 8, dtype=F64)], 1), dtype)
    takes = dtype == BF16 and kernels.mixed_prefill_takes(heads, dim, vdim)
    assert takes == (path == "tiles") and (dtype == torch.float32 or kernels.mixed_decode_takes(heads, kv_heads, dim, vdim))
    for portions in ([(0, 150, 300), (1, 0, 19), (2, 64, 131)], [(0, 298, 300), (1, 17, 19), (2, 0, 131)]):
        rows = packed(portions)
        want = torch.cat([wants[r][a:b] for r, a, b in portions])
        counts = [b - a for _, a, b in portions]
        out = torch.zeros(sum(counts), heads * vdim, dtype=dtype, device=device())
        kernels.paged_attention_mixed(rows, out, k_pool, v_pool, table, ints(np.repeat(np.arange(3), counts)),
                                      ints(np.concatenate([np.arange(a, b) for _, a, b in portions])), page, heads, kv_heads,
                                      dim, vdim, scale, mix, window, chunk)
        close(out, want, tol, "reference kernel")
        if takes:
            starts = ints(np.concatenate([[0], np.cumsum(counts)]))
            for slab in (kernels.MIXED_SLAB_BYTES, 1):           # (1: a slab of one tile at a time)
                before, kernels.MIXED_SLAB_BYTES = kernels.MIXED_SLAB_BYTES, slab
                try:
                    for tensor_cores in (False, True) if dim == vdim == 128 else (False,):
                        out.fill_(float("nan"))
                        kernels.mixed_prefill_attention(rows, out, k_pool, v_pool, table, starts, ints(lengths), page, heads,
                                                        kv_heads, dim, vdim, scale, mix, window, chunk, sum(counts),
                                                        max(lengths), scratch, tensor_cores=tensor_cores)
                        close(out, want, tol, f"tile kernels, tcgen05 {tensor_cores}, slab {slab}")
                    assert kernels.mixed_attention_error() == 0
                finally:
                    kernels.MIXED_SLAB_BYTES = before
    if dtype == BF16:
        singles = [(r, n - 1, n) for r, n in enumerate(lengths)]
        want = torch.cat([wants[r][a:b] for r, a, b in singles])
        for longest in (300, 512):                               # (a captured step's tables are wider than its requests)
            out = torch.full((3, heads * vdim), float("nan"), dtype=dtype, device=device())
            kernels.mixed_decode_attention(packed(singles), out, k_pool, v_pool, table, ints([n - 1 for n in lengths]), page,
                                           heads, kv_heads, dim, vdim, scale, mix, window, chunk, longest, scratch)
            close(out, want, tol, "split keys")


def test_runs_of_positions_without_mixed_heads_in_the_reference_kernel():
    """The kernel of plain softmax attention knows runs of positions too."""
    from libmir_b200 import kernels
    generator = torch.Generator().manual_seed(3)
    n, heads, dim, chunk, page = 90, 2, 24, 13, 8
    q, k, v = (torch.randn(n, heads, dim, generator=generator, dtype=F64).float().double() for _ in range(3))
    k_pool, v_pool, table = pool_of([k], [v], page, np.random.default_rng(0), torch.float32)
    out = torch.zeros(n, heads * dim, device=device())
    kernels.paged_attention_generic(on_device(q.reshape(n, -1).float()), out, k_pool, v_pool, table, ints([0] * n),
                                    ints(range(n)), page, heads, heads, dim, 0.3, None, chunk=chunk)
    close(out, plain.talking_attention(q, k, v, 0.3, None, chunk).reshape(n, -1), 2e-5)


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
        # its position alone, products, norms and the recurrence reduce in one fixed order
        assert np.array_equal(whole, single) and np.array_equal(whole, portions) and np.array_equal(whole, late)
    for group in model.cache_stats()["groups"]:
        assert group["free"] == group["pages"]


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("name", ["A", "C", "E"])
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


def test_far_tokens_decide_the_logits_in_prompt_and_in_decoding(tmp_path):
    """Sharp latent attention and a slow recurrence: the last positions depend on tokens hundreds of positions back, over
    many pages; whole, with the last tokens decoded one by one, and in portions."""
    config = {"architecture": "Pedotar", "vocab": 90, "width": 64, "norm": {"eps": 1e-5}, "layers": [
        dict(latent(2, 16, 8, 24, 40, 0.25), mlp=None), dict(scan(48, 8, 4, 4), mlp=None)]}

    def slow(tensors):
        tensors["l1.mix.A_log"] = torch.full_like(tensors["l1.mix.A_log"], math.log(0.02))
        tensors["l1.mix.D"] = torch.zeros_like(tensors["l1.mix.D"])
    ids = random_ids(np.random.default_rng(4), 90, 700)
    for dtype in ("float32", "bfloat16"):
        folder = make_folder(tmp_path / dtype, config, seed=6, dtype=dtype, sharpen=7.0, edit=slow)
        plain_config, weights = plain.read_model(folder)
        want = plain.forward(plain_config, weights, ids).numpy()
        shorter = plain.forward(plain_config, weights, ids[300:]).numpy()
        assert relative_error(shorter[-20:], want[-20:]).min() > 3 * TOL["bfloat16"]      # the early tokens matter
        model = load(folder, dtype, 16, 50)
        close_logits(feed(model, "whole", ids, [700]), want, dtype, f"far tokens, whole, {dtype}")
        close_logits(feed(model, "late", ids, [650, 1]), want, dtype, f"far tokens, decoded, {dtype}")
        close_logits(feed(model, "cut", ids, [15, 17, 300, 2, 31]), want, dtype, f"far tokens, portions, {dtype}")


@pytest.mark.parametrize("dim,page", [(24, 8), (64, 4), (128, 16)])
def test_the_edges_of_a_run_and_the_mixture_of_heads_show_in_the_logits(tmp_path, dim, page):
    """Two layers with runs of 37 and 21 positions: the plain implementation with runs one token longer or shorter, or
    without the heads' mixture, gives other logits, and the engine gives the configured ones, in a prompt and in decoding
    (heads of 24 channels: the reference and the split-key kernels, 64 and 128: the tile kernels in bfloat16)."""
    def model_config(first, second):
        return {"architecture": "Pedotar", "vocab": 80, "width": 64, "norm": {"eps": 1e-5}, "layers": [
            dict(mixed(4, 2, dim, dim, 1.0 / dim, first), mlp=None), dict(mixed(2, 2, dim, dim, 1.0 / dim, second), mlp=None)]}
    config = model_config(37, 21)
    ids = random_ids(np.random.default_rng(dim), 80, 120)
    for dtype in ("float32", "bfloat16"):
        folder = make_folder(tmp_path / dtype, config, seed=8, dtype=dtype, sharpen=6.0)
        _, weights = plain.read_model(folder)
        want = plain.forward(config, weights, ids).numpy()
        for first, second in ((38, 21), (36, 21), (37, 22), (37, 20)):
            moved = plain.forward(model_config(first, second), weights, ids).numpy()
            assert np.median(relative_error(moved, want)[45:]) > 0.05        # a run one token off is seen
        unmixed = dict(weights)
        for name in ("l0.mix.talk", "l1.mix.talk"):
            unmixed[name] = torch.eye(weights[name].shape[0], dtype=F64)
        assert np.median(relative_error(plain.forward(config, unmixed, ids).numpy(), want)) > 0.2
        model = load(folder, dtype, page, 80)
        for label, cuts in (("whole", [120]), ("decoded", [30, 1]), ("portions", [36, 2, 19, 2, 1, 22])):
            close_logits(feed(model, label, ids, cuts), want, dtype, f"{label}/{dtype}")


def test_runs_that_are_over_give_their_pages_back(tmp_path):
    """A request whose only paged mixer sees runs of 16 positions never holds more pages than a run and a portion."""
    config = {"architecture": "Pedotar", "vocab": 50, "width": 64, "norm": {"eps": 1e-5},
              "layers": [dict(mixed(2, 1, 16, 16, 0.25, 16), mlp=None)]}
    folder = make_folder(tmp_path, config, seed=1, dtype="float32")
    ids = random_ids(np.random.default_rng(1), 50, 130)
    model = load(folder, "float32", 4, 8)                       # 32 tokens of pages for a request of 130
    got = feed(model, "x", ids, [7, 12, 1, 1, 16, 2, 9, 1])
    close_logits(got, reference(folder, ids), "float32")
    stats = model.cache_stats()["groups"][0]
    assert stats["free"] == stats["pages"] and stats["high_water"] <= 8 and stats["chunk"] == 16


def test_the_designs_kernels_run_in_bfloat16(tmp_path):
    """Prompts run the tile kernels for mixed heads, single tokens the split-key ones; the recurrence, the norms between
    sublayers and the latent's preparation are one launch each per layer run; the reference kernels do not run."""
    from libmir_b200 import kernels
    for name in ("C", "D"):
        config = ALL[name]
        folder = make_folder(tmp_path / name, config, seed=3, dtype="bfloat16")
        ids = random_ids(np.random.default_rng(2), config["vocab"], 90)
        model = load(folder, "bfloat16", 16, 40)
        kernels.launch_counts(reset=True)
        feed(model, "x", ids, [88, 1])
        counts = kernels.launch_counts()
        assert counts.get("paged_attention_mixed", 0) == 0 and counts.get("paged_attention_generic", 0) == 0, counts
        order = [config["layers"][index] for index, _ in plain.layer_order(config)]
        runs = {kind: sum(layer["type"] == kind for layer in order) for kind in ("mamba1", "latent_attention", "attention")}
        steps = 3
        form = "_tc" if name == "D" else ""                     # heads of 128 channels: tcgen05, of 64: mma.sync
        assert counts["mixed_weights" + form] == counts["mixed_values" + form] == counts["mixed_row_sums" + form] \
            == runs["attention"], counts
        assert counts["mixed_decode_scores"] == counts["mixed_decode_values"] == 2 * runs["attention"], counts
        assert counts["selective_scan"] == steps * runs["mamba1"] and counts["latent_prepare"] == steps * runs["latent_attention"]
        assert counts["latent_attention"] == steps * runs["latent_attention"], counts
        sublayers = sum(1 + (layer["mlp"] is not None) for layer in order)
        # one norm ahead of the first layer and one before the head; all others inside the additions to the residual
        assert counts["add_layer_norm"] == steps * sublayers and counts["layer_norm"] == 2 * steps, counts
        assert counts.get("add_rows", 0) == 0, counts           # what opens a pass is added there too


@pytest.mark.parametrize("graphs", [False, True])
@pytest.mark.parametrize("name", ["A", "B"])
def test_greedy_generation_through_the_scheduler(tmp_path, name, graphs):
    """Model.generate_batch (scheduler, sampler, decode steps as captured graphs or not) against the plain
    implementation choosing greedily; float32, so that equal choices are expected wherever the best two logits are
    not closer than the tolerance."""
    from libmir_b200 import GenerationOverrides, GenerationRequest
    config = ALL[name]
    folder = make_folder(tmp_path, config, seed=9, dtype="float32")
    plain_config, weights = plain.read_model(folder)
    rng = np.random.default_rng(2)
    prompts = [random_ids(rng, config["vocab"], n) for n in (5, 23, 1)]
    model = load(folder, "float32", PAGE_SIZES[name], 48, graphs=graphs)
    outputs = model.generate_batch([GenerationRequest(p, GenerationOverrides(max_tokens=12, ignore_eos=True))
                                    for p in prompts])
    for prompt, output in zip(prompts, outputs):
        assert len(output.token_ids) == 12
        ids = list(prompt)
        for token in output.token_ids:
            logits = plain.forward(plain_config, weights, ids)[-1]
            best = int(torch.argmax(logits))
            assert token == best or float(logits[best] - logits[token]) < 1e-4, \
                f"{name}: the engine chose {token}, the plain implementation {best}"
            ids.append(token)
    if graphs:
        assert model.runner._graphs is not None and len(model.runner._graphs.graphs) > 0


@pytest.mark.parametrize("name", ["C", "D"])
def test_decode_steps_replayed_from_captured_graphs_in_bfloat16(tmp_path, name):
    """Two requests decoded together through captured graphs in bfloat16 (heads of 64 and 128 channels, runs of
    positions that begin and end among the decoded tokens, states that are carried by replays): the teacher-forced logits
    of every step against the plain implementation."""
    from libmir_b200 import StepEntry, kernels
    from libmir_b200.sampling import RequestSampler
    config = ALL[name]
    folder = make_folder(tmp_path, config, seed=8, dtype="bfloat16")
    rng = np.random.default_rng(5)
    requests = {"a": random_ids(rng, config["vocab"], 100), "b": random_ids(rng, config["vocab"], 87)}
    want = {key: reference(folder, ids) for key, ids in requests.items()}
    prompt = {"a": 21, "b": 8}
    model = load(folder, "bfloat16", PAGE_SIZES[name], 80, graphs=True)
    got = {key: [] for key in requests}
    for key, ids in requests.items():
        model.admit(key)
        result = model.step([StepEntry(key, ids[:prompt[key]], range(prompt[key]))])
        got[key].append(result.logits.float().cpu().numpy().copy())
    for step in range(79):
        entries = [StepEntry(key, [ids[prompt[key] + step]], [0]) for key, ids in requests.items()]
        result = model.step(entries, [RequestSampler() for _ in entries])
        logits = result.logits.float().cpu().numpy()
        for row, key in enumerate(requests):
            got[key].append(logits[row:row + 1].copy())
    assert model.runner._graphs is not None and len(model.runner._graphs.graphs) > 0
    everything = np.concatenate([np.concatenate(got[key]) for key in requests])
    wanted = np.concatenate([want[key][:prompt[key] + 79] for key in requests])
    close_logits(everything, wanted, "bfloat16", "decode steps from captured graphs")
    assert kernels.tensor_core_linear_error() == 0 and kernels.decode_attention_error() == 0


def test_trace_runner_picks_the_design_by_its_configuration(tmp_path):
    """bin/trace_run as a user runs it: the model class comes from config.json; prompts in portions, decoded tokens,
    a pool that holds less than all requests together."""
    config = ALL["A"]
    folder = make_folder(tmp_path / "model", config, seed=4, dtype="bfloat16")
    (folder / "config.json").write_text(json.dumps(dict(config, vocab_size=config["vocab"])))   # (helpers read this key)
    rng = np.random.default_rng(3)
    requests = {f"q{i}": random_ids(rng, config["vocab"], n) for i, n in enumerate((100, 64, 37))}
    want = {name: reference(folder, ids) for name, ids in requests.items()}
    for dtype, extra in (("bfloat16", []), ("float32", []), ("bfloat16", ["--decode-graphs"])):
        trace = Trace()
        for name, ids in requests.items():
            trace.step([(name, ids[:len(ids) - 10], [0, len(ids) - 11])])
            for position in range(len(ids) - 10, len(ids)):
                trace.step([(name, ids[position:position + 1], [0])], end=[name] if position == len(ids) - 1 else [])
        results = run_trace(folder, dtype, trace, tmp_path / f"out-{dtype}-{len(extra)}", max_tokens=128,
                            extra_args=["--page-size", "8"] + extra)
        got = np.stack([results[index][row] for index, rows in enumerate(trace.expect) for row in range(len(rows))])
        wanted = np.stack([want[name][position] for rows in trace.expect for name, position in rows])
        close_logits(got, wanted, dtype, f"trace {dtype} {extra}")


def test_generate_command_line(tmp_path):
    """bin/generate on a model folder of the design: two prompts as one batch, greedy, against the plain
    implementation."""
    import subprocess
    import sys
    from helpers import ROOT
    config = ALL["D"]
    folder = make_folder(tmp_path / "model", config, seed=12, dtype="float32")
    plain_config, weights = plain.read_model(folder)
    command = [sys.executable, str(ROOT / "bin" / "generate"), str(folder), "--dtype", "float32", "--block-size", "8",
               "--block-count", "64", "--max-tokens", "6", "--ignore-eos"]
    done = subprocess.run(command + ["--prompt-ids", "5,9,80,33;7", "--json"], capture_output=True, text=True, timeout=600)
    assert done.returncode == 0, done.stderr[-3000:]
    outputs = [json.loads(line) for line in done.stdout.splitlines() if line.startswith("{")]
    assert len(outputs) == 2
    for prompt, output in zip(([5, 9, 80, 33], [7]), outputs):
        ids = list(prompt)
        for token in output["token_ids"]:
            logits = plain.forward(plain_config, weights, ids)[-1]
            best = int(torch.argmax(logits))
            assert token == best or float(logits[best] - logits[token]) < 1e-4
            ids.append(token)


@pytest.mark.parametrize("seed", range(8))
def test_configurations_drawn_at_random(tmp_path, seed):
    """Sizes nobody chose: a prompt whole, token by token, in portions and as a prompt followed by decoding, in both
    dtypes, against the plain implementation (32-bit: every position within 2e-4 of its logits' root mean square and
    the same bits under every cut; bfloat16: nine positions in ten within the tolerance)."""
    rng = np.random.default_rng(900 + seed)
    config = random_config(rng)
    page = int(rng.choice([4, 8, 16]))
    ids = random_ids(rng, config["vocab"], 100)
    for dtype in ("float32", "bfloat16"):
        folder = make_folder(tmp_path / dtype, config, seed=seed, dtype=dtype)
        want = reference(folder, ids)
        model = load(folder, dtype, page, 80)
        outputs = [feed(model, "whole", ids, [len(ids)]), feed(model, "single", ids, [1]),
                   feed(model, "portions", ids, [2, 5, 1, 33, 3, 16, 2, 7]), feed(model, "late", ids, [80, 1])]
        for got in outputs:
            relative = relative_error(got, want)
            assert np.isfinite(relative).all(), json.dumps(config)
            if dtype == "float32":
                assert relative.max() <= 2e-4, f"{relative.max():.3e} at {int(relative.argmax())}: {json.dumps(config)}"
            else:
                assert np.quantile(relative, 0.9) <= TOL[dtype], f"{np.quantile(relative, 0.9):.3e}: {json.dumps(config)}"
        if dtype == "float32":
            assert all(np.array_equal(outputs[0], other) for other in outputs[1:]), json.dumps(config)
        model.unload()
