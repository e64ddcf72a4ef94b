"""Biravik on the GPU against the plain implementation (tests/plain_biravik.py): every mechanism's kernel alone, then whole
models through the engine's step function, cache manager and scheduler: prompts whole, token by token, in portions down to
two tokens, in batches of unequal requests, with pages and state slots that change hands, with keys far away, at page
borders and at windows' edges, in long decoding, and greedy generation through the entry point."""

import json
import math

import numpy as np
import pytest
import torch

import plain_biravik as plain
from biravik_configs import ALL, PAGE_SIZES, make_folder, random_config
from helpers import TOL, Trace, random_ids, run_trace

pytestmark = pytest.mark.gpu
F64, BF16 = torch.float64, torch.bfloat16


def device():
    return torch.device("cuda", 0)


def close(got, want, tol, what=""):
    got = got.detach().double().cpu() if isinstance(got, torch.Tensor) else torch.as_tensor(got, dtype=F64)
    want = want.detach().double().cpu() if isinstance(want, torch.Tensor) else torch.as_tensor(want, dtype=F64)
    error = (got - want).abs().max().item()
    bound = tol * max(1.0, want.abs().max().item())
    assert math.isfinite(error) and error <= bound, f"{what}: max |diff| {error:.3e} > {bound:.3e}"


def relative_error(got, want):
    """Of every position: root mean square of the difference over that of the logits."""
    got, want = np.asarray(got, dtype=np.float64), np.asarray(want, dtype=np.float64)
    return np.sqrt(((got - want) ** 2).mean(-1)) / np.sqrt((want ** 2).mean(-1))


def close_logits(got, want, dtype, what=""):
    """Logits [positions, vocab] of a whole model.  float32: every position within 2e-4 of its logits' root mean square.
    bfloat16: nine positions in ten within the tolerance and all but three in a hundred within five times it: where two
    experts' scores lie closer together than the rounding of the router's input, the engine and the 64-bit implementation
    may choose differently at that one token, and where a recurrent head reads almost nothing out of a young state its
    norm magnifies the projections' rounding.  A lost state or a missed key is an error of order one at most positions."""
    relative = relative_error(got, want)
    assert np.isfinite(relative).all(), f"{what}: not finite"
    if dtype == "float32":
        assert relative.max() <= 2e-4, f"{what}: {relative.max():.3e} at position {int(relative.argmax())}"
        return
    assert np.quantile(relative, 0.9) <= TOL[dtype] and (relative <= 5 * TOL[dtype]).mean() >= 0.97, \
        f"{what}: relative error of positions: 90% {np.quantile(relative, 0.9):.3e}, max {relative.max():.3e}"


def on_device(tensor, dtype=None):
    return tensor.to(device=device(), dtype=dtype or tensor.dtype).contiguous()


def batch_description(portions, slots, starts_at=None):
    """Device tensors describing packed rows: portions = tokens per request row; positions count from starts_at."""
    starts = np.concatenate([[0], np.cumsum(portions)]).astype(np.int32)
    row_of_token = np.repeat(np.arange(len(portions)), portions).astype(np.int32)
    first = starts_at or [0] * len(portions)
    positions = np.concatenate([np.arange(f, f + n) for f, n in zip(first, portions)]) if len(portions) else []
    to = lambda a: torch.as_tensor(np.asarray(a, dtype=np.int32), device=device())
    return to(row_of_token), to(starts), to(slots), to(positions)


DTYPES = [(torch.float32, 2e-6), (BF16, 8e-3)]


# ------------------------------------------------------------------------------ kernels alone
@pytest.mark.parametrize("rows,width", [(1, 8), (5, 100), (130, 192), (3, 50), (7, 2050), (2, 4096), (1, 9000), (2, 16384)])
@pytest.mark.parametrize("branches", [1, 2, 4])
def test_norm_behind_the_sum(rows, width, branches):
    """x <- rmsnorm(alpha x + sum of scaled branches) * w, and its copy in bfloat16: the same bits as a cast."""
    from libmir_b200 import kernels
    torch.manual_seed(width)
    x, weight = torch.randn(rows, width) * 2.0, 1.0 + torch.randn(width) * 0.3
    results = [torch.randn(rows, width) * (3.0 + b) for b in range(branches)]
    scales = [1.3, 0.7, -0.4, 2.0][:branches]
    total = 1.7 * x.double() + sum(s * r.double() for s, r in zip(scales, results))
    want = plain.unit_rms(total, 1e-5) * weight.double()
    got, rounded = on_device(x), torch.full((rows, width), 7.0, dtype=BF16, device=device())
    kernels.norm_scaled_sum([on_device(r) for r in results], scales, got, on_device(weight), 1.7, 1e-5, rounded=rounded)
    close(got, want, 2e-6, f"{rows} x {width}")
    assert torch.equal(rounded, got.to(BF16))
    again = on_device(x)
    kernels.norm_scaled_sum([on_device(r) for r in results], scales, again, on_device(weight), 1.7, 1e-5)
    assert torch.equal(again, got)
    for accumulate in (False, True):
        out = on_device(x)
        kernels.scaled_sum([on_device(r) for r in results], scales, out, accumulate=accumulate)
        close(out, total - (1.7 - accumulate) * x.double(), 2e-6, "scaled sum")


@pytest.mark.parametrize("dtype,tol", DTYPES)
@pytest.mark.parametrize("heads,kv_heads,dim,rotary,scaled", [(4, 2, 24, 16, True), (1, 1, 16, 0, False), (6, 2, 64, 64, True),
                                                              (4, 1, 128, 32, True), (3, 3, 20, 20, False), (2, 1, 128, 0, False)])
def test_values_are_the_keys_as_projected(dtype, tol, heads, kv_heads, dim, rotary, scaled):
    """Packed rows [q | k | gate]: q and k normed and rotated in interleaved pairs (with a factor on cos and sin), the keys'
    columns as they were projected go to the value pages, bit for bit; the gate's columns are left alone; a token without a
    place in the pool leaves nothing there."""
    from libmir_b200 import kernels
    from libmir_b200.config.spec import YarnScaling
    from libmir_b200.parts.rope import inverse_frequencies, yarn_magnitude
    torch.manual_seed(dim + heads)
    tokens, eps = 11, 1e-5
    rot, table, magnitude = None, None, 1.0
    if rotary:
        rot = {"dims": rotary, "base": 700.0}
        scaling = None
        if scaled:
            rot["scaling"] = {"factor": 4.0, "original": 64, "fast": 16.0, "slow": 1.0}
            scaling = YarnScaling(4.0, 64.0, 16.0, 1.0)
        table, magnitude = on_device(inverse_frequencies(rotary, 700.0, scaling)), yarn_magnitude(scaling)
        close(table, plain.rotary_table(rot)[0], 1e-6, "frequencies")
        assert math.isclose(magnitude, plain.rotary_table(rot)[1], rel_tol=1e-12) and (magnitude != 1.0) == scaled
    positions = torch.tensor([0, 1, 2, 3, 500, 501, 77, 9, 10, 11, 4096], dtype=torch.int32)
    slots = torch.tensor([5, 6, 7, 40, 41, 63, 0, 1, 2, -1, 20], dtype=torch.int32)
    packed = torch.randn(tokens, (heads + kv_heads) * dim + heads * dim).to(dtype)
    q_norm, k_norm = 1.0 + torch.randn(dim) * 0.3, 1.0 + torch.randn(dim) * 0.3
    raw = packed[:, heads * dim:(heads + kv_heads) * dim].reshape(tokens, kv_heads, dim)
    q = plain.unit_rms(packed[:, :heads * dim].double().reshape(tokens, heads, dim), eps) * q_norm.double()
    k = plain.unit_rms(raw.double(), eps) * k_norm.double()
    if rot:
        q, k = plain.rotate_interleaved(q, positions, rot), plain.rotate_interleaved(k, positions, rot)
    k_pool = torch.zeros(64, kv_heads, dim, dtype=dtype, device=device())
    v_pool = torch.zeros(64, kv_heads, dim, dtype=dtype, device=device())
    rows = on_device(packed)
    kernels.qk_rope_store(rows, on_device(positions), on_device(slots), table, on_device(q_norm), on_device(k_norm), k_pool,
                          v_pool, heads, kv_heads, dim, rotary, eps, interleaved=True, magnitude=magnitude,
                          values_from_keys=True)
    angle_tol = max(tol, 5e-4 if rotary else 0.0)                 # (angles are 32-bit products: 4096 * frequency)
    close(rows[:, :heads * dim], q.reshape(tokens, -1), angle_tol, "queries")
    assert torch.equal(rows[:, (heads + kv_heads) * dim:].cpu(), packed[:, (heads + kv_heads) * dim:])
    kept = slots >= 0
    close(k_pool[slots[kept].long()], k[kept], angle_tol, "keys")
    assert torch.equal(v_pool[slots[kept].long()].cpu(), raw[kept])
    mask = torch.ones(64, dtype=torch.bool)
    mask[slots[kept].long()] = False
    assert float(k_pool[mask].abs().max()) == 0.0 and float(v_pool[mask].abs().max()) == 0.0


@pytest.mark.parametrize("dtype,tol", DTYPES)
@pytest.mark.parametrize("heads,kv_heads,dim,vdim,every,half_split", [(6, 2, 32, 20, 24, False), (4, 2, 64, 32, 1, False),
                                                                      (4, 4, 128, 64, 256, False), (1, 1, 12, 12, 7, False),
                                                                      (4, 2, 64, 64, 10, True), (3, 1, 20, 20, 10, True)])
def test_temperature_on_the_queries(dtype, tol, heads, kv_heads, dim, vdim, every, half_split):
    """Queries times 1 + coef ln(floor((p + 1) / every) + 1) behind their norm, on either side of its steps; keys without it;
    values of another width than the keys into their own pages.  With a half-split rotation too."""
    from libmir_b200 import kernels
    torch.manual_seed(dim)
    positions = torch.tensor([0, every - 2 if every > 1 else 1, every - 1, every, 2 * every - 1, 2 * every, 5 * every - 1, 70000],
                             dtype=torch.int32).clamp(min=0)
    tokens = positions.numel()
    slots = torch.arange(tokens, dtype=torch.int32) + 3
    packed = torch.randn(tokens, (heads + kv_heads) * dim + kv_heads * vdim + heads * vdim).to(dtype)
    q_norm, k_norm = 1.0 + torch.randn(dim) * 0.3, 1.0 + torch.randn(dim) * 0.3
    q = plain.unit_rms(packed[:, :heads * dim].double().reshape(tokens, heads, dim), 1e-6) * q_norm.double()
    k = plain.unit_rms(packed[:, heads * dim:(heads + kv_heads) * dim].double().reshape(tokens, kv_heads, dim), 1e-6) * k_norm.double()
    v = packed[:, (heads + kv_heads) * dim:(heads + kv_heads) * dim + kv_heads * vdim].reshape(tokens, kv_heads, vdim)
    q = q * plain.query_temperature(positions, 0.4, every)[:, None, None]
    table, rotary = None, 0
    if half_split:
        positions_gpu = positions.clamp(max=1000)                # (keep the angles' rounding out of this test)
        q = q / plain.query_temperature(positions, 0.4, every)[:, None, None]
        q = q * plain.query_temperature(positions_gpu, 0.4, every)[:, None, None]
        positions, rotary = positions_gpu, dim
        freq = torch.tensor([100.0 ** (-2.0 * i / dim) for i in range(dim // 2)], dtype=F64)
        table = on_device(freq.float())

        def turn(x):
            angle = positions.double()[:, None] * freq[None, :]
            cos, sin = torch.cos(angle)[:, None], torch.sin(angle)[:, None]
            a, b = x[..., :dim // 2], x[..., dim // 2:]
            return torch.cat([a * cos - b * sin, b * cos + a * sin], dim=-1)
        q, k = turn(q), turn(k)
    rows = on_device(packed)
    k_pool = torch.zeros(32, kv_heads, dim, dtype=dtype, device=device())
    v_pool = torch.zeros(32, kv_heads, vdim, dtype=dtype, device=device())
    kernels.qk_rope_store(rows, on_device(positions), on_device(slots), table, on_device(q_norm), on_device(k_norm), k_pool,
                          v_pool, heads, kv_heads, dim, rotary, 1e-6, value_dim=vdim, temperature=(0.4, every))
    bound = max(tol, 2e-4 if half_split else 0.0)
    close(rows[:, :heads * dim], q.reshape(tokens, -1), bound, "queries")
    close(k_pool[slots.long()], k, bound, "keys")
    assert torch.equal(v_pool[slots.long()].cpu(), v)
    tail = (heads + kv_heads) * dim + kv_heads * vdim
    assert torch.equal(rows[:, tail:].cpu(), packed[:, tail:])


def plain_recurrence(q, k, v, decays, state):
    """q, k [n, heads, dim], v [n, heads, vdim], state [heads, dim, vdim] float64: the read-outs and the last state."""
    out = torch.zeros(v.shape, dtype=F64)
    for t in range(q.shape[0]):
        state = decays[:, None, None] * state + k[t][:, :, None] * v[t][:, None, :]
        out[t] = torch.einsum("hkv,hk->hv", state, q[t])
    return out, state


@pytest.mark.parametrize("dtype", [torch.float32, BF16])
@pytest.mark.parametrize("heads,dim,vdim", [(2, 64, 40), (3, 20, 12), (1, 128, 64), (4, 6, 6), (2, 100, 20), (1, 256, 8)])
def test_lightning_recurrence_with_activated_inputs(dtype, heads, dim, vdim):
    """silu of q, k and v enters, in every form of the recurrence's kernel: a whole prompt, a portion that goes on from a
    carried state and a single token in one batch, then single tokens; with and without the inputs prepared by a kernel of
    its own (the same bits).  Slots that no row names stay as they were."""
    from libmir_b200 import kernels
    torch.manual_seed(heads * dim)
    decays = torch.tensor([0.5, 0.9, 0.99, 0.999][:heads], dtype=F64)
    slots, lengths, starts = [4, 0, 2], [70, 33, 1], [0, 517, 9]
    ld = heads * (2 * dim + vdim) + 8
    state0 = torch.randn(6, heads, vdim, dim) * 0.5
    state0[4] = 0.0
    state = on_device(state0)
    for phase in range(2):
        if phase == 1:
            starts, lengths = [s + n for s, n in zip(starts, lengths)], [1, 1, 1]
        tokens = sum(lengths)
        packed = torch.randn(tokens, ld).to(dtype)
        cut = lambda t: (t[:, :heads * dim], t[:, heads * dim:2 * heads * dim], t[:, 2 * heads * dim:2 * heads * dim + heads * vdim])
        q, k, v = (plain.silu(part.double()) for part in cut(packed))
        _, query_starts, slot_tensor, positions = batch_description(lengths, slots, starts)
        before = state.cpu().double()
        want, want_state, cursor = [], before.clone(), 0
        for slot, n in zip(slots, lengths):
            rows = slice(cursor, cursor + n)
            o, s = plain_recurrence(q[rows].reshape(n, heads, dim), k[rows].reshape(n, heads, dim),
                                    v[rows].reshape(n, heads, vdim), decays, before[slot].transpose(1, 2))
            want.append(o.reshape(n, heads * vdim))
            want_state[slot] = s.transpose(1, 2)
            cursor += n
        gpu = cut(on_device(packed))
        scratch = torch.full((kernels.retention_prepared_floats(tokens, heads, dim),), float("nan"), device=device())
        outputs = []
        for prepared in (None, scratch):
            here, out = state.clone(), torch.full((tokens, heads * vdim), 5.0, device=device())
            kernels.retention_scan(*gpu, None, on_device(decays.float()), 1.0, here, query_starts, slot_tensor, positions, out,
                                   heads, dim, vdim, prepared=prepared, activated=True)
            outputs.append((out, here))
        assert torch.equal(outputs[0][0], outputs[1][0]) and torch.equal(outputs[0][1], outputs[1][1])
        out, state = outputs[0]
        close(out, torch.cat(want), 3e-5, f"read-outs, phase {phase}")
        close(state, want_state, 3e-5, f"states, phase {phase}")
        for untouched in (1, 3, 5):
            assert torch.equal(state[untouched].cpu(), before[untouched].float())


@pytest.mark.parametrize("dtype,tol", DTYPES)
def test_norm_over_all_heads_with_a_sigmoid_gate(dtype, tol):
    """One root mean square over all heads' columns, a weight per column, a sigmoid gate; narrow and wide rows."""
    from libmir_b200 import kernels
    torch.manual_seed(2)
    for tokens, width in ((1, 8), (9, 60), (70, 320), (4, 511), (5, 512), (3, 2050), (130, 1024)):
        o, weight = torch.randn(tokens, width) * 3.0, 1.0 + torch.randn(width) * 0.3
        packed = torch.randn(tokens, width + 24).to(dtype)
        want = plain.unit_rms(o.double(), 1e-5) * weight.double() * plain.sigmoid(packed[:, 16:16 + width].double())
        out = torch.zeros(tokens, width, dtype=dtype, device=device())
        kernels.gated_head_norm(on_device(o), on_device(packed)[:, 16:16 + width], on_device(weight), out, 1, width, 1e-5, True)
        close(out, want, tol, f"{tokens} x {width}")


@pytest.mark.parametrize("experts,top", [(8, 2), (5, 5), (3, 1), (40, 7)])
def test_softmax_over_the_chosen_logits_alone(experts, top):
    """Also where the logits lie so far apart that a softmax over all of them underflows."""
    from libmir_b200 import kernels
    torch.manual_seed(experts)
    logits = torch.randn(33, experts) * 4.0
    logits[5] = torch.arange(experts).float() * -300.0           # all but one probability underflow
    logits[6] = logits[5].flip(0)
    ids = torch.zeros(33, top, dtype=torch.int32, device=device())
    weights = torch.zeros(33, top, device=device())
    kernels.moe_route(on_device(logits), None, False, ids, weights, None, experts, top, 1, 1, 1.0, score="softmax",
                      group_score="max")
    picked, chosen = logits.double().topk(top, dim=-1)
    assert torch.equal(ids.cpu().long(), chosen)
    close(weights, torch.softmax(picked, -1), 2e-6, "weights")


def plain_attention(q, k, v, scale, sinks, slopes, gate, first, window=None, keep=0):
    """q [n, H, d] at positions first .. first + n - 1 over keys [m, G, d] and values [m, G, e], float64."""
    n, heads, _ = q.shape
    keys = k.shape[0]
    group = heads // k.shape[1]
    k, v = k.double().repeat_interleave(group, 1), v.double().repeat_interleave(group, 1)
    i, j = torch.arange(first, first + n)[:, None], torch.arange(keys)[None, :]
    scores = torch.einsum("ihd,jhd->hij", q.double(), k) * scale
    if slopes is not None:
        scores = scores - slopes.double()[:, None, None] * (i - j).double()
    seen = j <= i
    if window:
        seen = seen & ((i - j < window) | (j < keep))
    weights = plain.sink_softmax(scores.masked_fill(~seen[None], float("-inf")), sinks.double())
    out = torch.einsum("hij,jhe->ihe", weights, v).reshape(n, -1)
    return out * plain.sigmoid(gate.double())


def scatter_into_pool(ks, vs, page, rng, dtype):
    """Each request's keys and values into shuffled pages of one pool (garbage elsewhere); the pools and the table."""
    blocks = [-(-k.shape[0] // page) for k in ks]
    total = sum(blocks) + 3
    order = rng.permutation(total)
    k_pool = (torch.randn(total * page, *ks[0].shape[1:]) * 40.0).to(dtype)
    v_pool = (torch.randn(total * page, *vs[0].shape[1:]) * 40.0).to(dtype)
    table = torch.full((len(ks), max(blocks)), -1, dtype=torch.int32)
    cursor = 0
    for r, (k, v) in enumerate(zip(ks, vs)):
        for block in range(blocks[r]):
            physical = int(order[cursor]); cursor += 1
            table[r, block] = physical
            rows = slice(block * page, min(k.shape[0], (block + 1) * page))
            k_pool[physical * page: physical * page + rows.stop - rows.start] = k[rows]
            v_pool[physical * page: physical * page + rows.stop - rows.start] = v[rows]
    return k_pool, v_pool, table


# which kernels a case runs: the reference kernel, the mma.sync kernels, the tcgen05 kernels
BIASED_CASES = [
    # dtype, heads, kv_heads, dim, vdim, page, path
    (torch.float32, 6, 2, 32, 20, 8, "reference"), (torch.float32, 1, 1, 16, 16, 4, "reference"),
    (BF16, 3, 3, 20, 12, 4, "reference"), (BF16, 4, 2, 64, 40, 16, "reference"),
    (BF16, 4, 2, 64, 32, 8, "mma"), (BF16, 6, 1, 64, 64, 16, "mma"), (BF16, 5, 5, 64, 128, 4, "mma"),
    (BF16, 4, 2, 128, 32, 16, "mma"), (BF16, 4, 1, 128, 64, 8, "mma"), (BF16, 4, 2, 128, 128, 16, "mma"),
    (BF16, 4, 2, 128, 64, 16, "tcgen05"), (BF16, 12, 1, 128, 64, 32, "tcgen05"), (BF16, 3, 3, 128, 64, 8, "tcgen05"),
    (BF16, 8, 2, 128, 128, 16, "tcgen05"), (BF16, 24, 1, 128, 128, 8, "tcgen05"),
]


@pytest.mark.parametrize("dtype,heads,kv_heads,dim,vdim,page,path", BIASED_CASES)
def test_attention_with_a_linear_bias_and_values_of_their_own_width(dtype, heads, kv_heads, dim, vdim, page, path):
    """Per request one query is made to look at one chosen key (its query and that key scaled so that this score stands
    out): the first token, either side of a page border, hundreds of tokens back (where the bias has taken off a known
    part of it), the newest.  Requests run as a whole prompt, a portion that starts in mid-request, a two-token portion
    and single decoded tokens, in one batch through the kernels the engine would choose."""
    from libmir_b200 import kernels
    rng = np.random.default_rng(dim + heads)
    torch.manual_seed(dim * heads + vdim)
    scale = 0.9 / math.sqrt(dim)
    slopes = plain.slopes(heads)
    # (context length, first token of the step's portion, the key the last query looks at)
    plans = [(300, 0, 0), (300, 283, 7), (97, 95, 2 * page - 1), (130, 129, 2 * page), (290, 289, 3), (64, 63, 63), (1, 0, 0)]
    order = sorted(plans, key=lambda plan: plan[0] - plan[1] != 1)               # single tokens lead the batch
    qs, ks, vs = [], [], []
    for length, first, target in order:
        q, k = torch.randn(length, heads, dim), torch.randn(length, kv_heads, dim)
        direction = torch.randn(dim)
        direction /= direction.norm()
        k[target] = direction * 6.0
        # every head's score of the chosen key is about 36 after its bias
        lift = 36.0 + slopes.float()[:, None] * (length - 1 - target)
        q[-1] = direction * (lift / 6.0) / scale + torch.randn(heads, dim) * 0.1
        qs.append(q.to(dtype)); ks.append(k.to(dtype)); vs.append(torch.randn(length, kv_heads, vdim).to(dtype))
    sinks = torch.randn(heads) * 1.5 + 1.0
    k_pool, v_pool, table = scatter_into_pool(ks, vs, page, rng, dtype)
    q_rows = torch.cat([q[first:].reshape(length - first, -1) for q, (length, first, _) in zip(qs, order)])
    tokens = q_rows.shape[0]
    gate = (torch.randn(tokens, heads * vdim) * 2.0).to(dtype)
    packed = torch.cat([q_rows, torch.randn(tokens, 24).to(dtype), gate], dim=1)
    portions = [length - first for length, first, _ in order]
    row_of_token, starts, _, positions = batch_description(portions, [0] * len(portions), [first for _, first, _ in order])
    contexts = torch.tensor([length for length, _, _ in order], dtype=torch.int32, device=device())
    edges = starts.tolist()
    want = torch.cat([plain_attention(q[first:], k, v, scale, sinks, slopes, gate[a:b], first)
                      for q, k, v, (_, first, _), a, b in zip(qs, ks, vs, order, edges, edges[1:])])
    rows = on_device(packed)
    gate_view = rows[:, heads * dim + 24:]
    out = torch.full((tokens, heads * vdim), 9.0, dtype=dtype, device=device())
    pools = (on_device(k_pool), on_device(v_pool))
    table, sinks_gpu, slopes_gpu = on_device(table), on_device(sinks), on_device(slopes.float())
    tol = 1e-5 if dtype == torch.float32 else 2e-2
    if path == "reference":
        kernels.paged_attention_generic(rows, out, *pools, table, row_of_token, positions, page, heads, kv_heads, dim, scale,
                                        None, value_dim=vdim, sinks=sinks_gpu, gate=gate_view, slopes=slopes_gpu)
        close(out, want, tol, "reference kernel")
        return
    singles = sum(1 for n in portions if n == 1)
    extras = dict(sinks=sinks_gpu, slopes=slopes_gpu, value_dim=vdim)
    for partition, contexts_in_one in ((64, False), (128, False), (256, False), (384, True)):
        if path == "tcgen05" and partition == 64:
            continue
        out.fill_(9.0)
        count = 1 if contexts_in_one else -(-300 // partition)
        floats = kernels.decode_attention_scratch_floats(singles, heads, vdim, count)
        scratch = torch.full((max(floats, 1),), float("nan"), device=device())
        with kernels.option("decode_tensor_cores", int(path == "tcgen05")):
            kernels.decode_attention(rows[:singles], out[:singles], *pools, table[:singles], positions, page, heads, kv_heads,
                                     dim, scale, None, partition, count, scratch if floats else None,
                                     gate=gate_view[:singles], **extras)
        kernels.prefill_attention(rows, out, *pools, table[singles:], starts[singles:], contexts[singles:], page, heads,
                                  kv_heads, dim, scale, None, tensor_cores=path == "tcgen05", gate=gate_view, **extras)
        close(out, want, tol, f"{path} kernels, partitions of {partition} keys")
    # what the engine plans for these rows fits the kernel it then runs
    partition, count, floats = kernels.decode_attention_plan(singles, heads, kv_heads, dim, page, 300, value_dim=vdim)
    out[:singles].fill_(9.0)
    kernels.decode_attention(rows[:singles], out[:singles], *pools, table[:singles], positions, page, heads, kv_heads, dim,
                             scale, None, partition, count, torch.empty(max(floats, 1), device=device()) if floats else None,
                             gate=gate_view[:singles], **extras)
    close(out[:singles], want[:singles], tol, f"{path}, the engine's own plan")
    assert kernels.decode_attention_error() == 0 and kernels.prefill_attention_error() == 0


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


@pytest.mark.parametrize("name", sorted(ALL))
def test_the_residual_stream_after_every_layer(tmp_path, name):
    """One prompt in 32-bit: the residual after each layer against the plain implementation's, so that a fault shows at the
    layer that has it."""
    from libmir_b200 import StepEntry
    config = ALL[name]
    folder = make_folder(tmp_path, config, seed=2, dtype="float32")
    ids = random_ids(np.random.default_rng(1), config["vocab"], 60)
    plain_config, weights = plain.read_model(folder)
    want, seen = [], []
    plain.forward(plain_config, weights, ids, want)
    model = load(folder, "float32", PAGE_SIZES[name], 40)
    model.decoder.after_entry = lambda index, residual: seen.append(residual.cpu())
    model.admit("x")
    model.step([StepEntry("x", ids, [0])])
    model.decoder.after_entry = None
    assert len(seen) == len(want) == len(config["layers"])
    for layer, (got, expected) in enumerate(zip(seen, want)):
        close(got, expected, 3e-5, f"after layer {layer}")


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("name", sorted(ALL))
def test_whole_prompts_token_by_token_and_portions(tmp_path, name, dtype):
    """A prompt whole; the same token by token from its first token (150 single steps: long decoding, windows that pass over
    decoded tokens, the first tokens of a sequence); in portions of changing size down to two tokens; and most of it whole
    with the rest decoded."""
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
    if dtype == "float32":      # 32-bit results do not depend on the cut at all
        assert np.array_equal(whole, single) and np.array_equal(whole, portions) and np.array_equal(whole, late)
    for group in model.cache_stats()["groups"]:
        assert group["free"] == group["pages"]


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("name", ["A", "C", "D"])
def test_batches_of_unequal_requests_with_pages_and_slots_that_change_hands(tmp_path, name, dtype):
    """Up to three live requests of unequal lengths, portions of some beside single tokens of others, requests that sit a
    step out, in a pool so small that pages and state slots are used again; every request against itself alone (the plain
    implementation)."""
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
    assert stats["free_slots"] == 3
    for group in stats["groups"]:
        assert group["free"] == group["pages"] and group["reused"] > 0


FAR_LAYERS = {
    # steep scores and a temperature that lifts late queries; the flat slopes of many heads reach far back
    "parallel": [{"type": "parallel", "mlp": None, "mixer": {
        "left_scale": 1.0, "right_scale": 0.3,
        "left": {"heads": 8, "kv_heads": 2, "dim": 64, "vdim": 32, "scale": 0.13, "q_temp": {"coef": 0.35, "every": 100}},
        "right": {"heads": 2, "dim": 16, "vdim": 24, "decay": [0.9995, 0.998]}}}],
    # heads of 128 channels: many key tiles of the tcgen05 kernels, from the query backwards
    "wide": [{"type": "parallel", "mlp": None, "mixer": {
        "left_scale": 1.0, "right_scale": 0.2,
        "left": {"heads": 8, "kv_heads": 2, "dim": 128, "vdim": 64, "scale": 0.05, "q_temp": {"coef": 0.3, "every": 90}},
        "right": {"heads": 1, "dim": 16, "vdim": 24, "decay": [0.99]}}}],
    "attention": [{"type": "attention", "mlp": None, "mixer": {
        "heads": 4, "kv_heads": 2, "dim": 64, "vdim": 64, "scale": 0.13, "rot": {"dims": 16, "base": 10000.0}}}],
    "kept": [{"type": "attention", "mlp": None, "mixer": {
        "heads": 2, "kv_heads": 1, "dim": 64, "vdim": 64, "scale": 0.13, "mask": {"size": 90, "keep_first": 70}}}],
    "wkv": [{"type": "wkv", "mlp": None, "mixer": {"heads": 2, "dim": 16, "decay_rank": 4}}],
}


@pytest.mark.parametrize("kind", sorted(FAR_LAYERS))
def test_far_tokens_decide_the_logits_in_prompt_and_in_decoding(tmp_path, kind):
    """One mixer whose memory reaches far: attention with a linear bias beside lightning attention with decays near one,
    attention without a window over many pages, kept first tokens far outside the window, and wkv with slow decays: the
    last positions depend on tokens hundreds of tokens back; whole, with the last tokens decoded, and in portions."""
    config = {"architecture": "Biravik", "vocab": 90, "width": 64, "norm": {"eps": 1e-5}, "postln_alpha": 0.5,
              "layers": FAR_LAYERS[kind]}
    ids = random_ids(np.random.default_rng(4), 90, 700)
    for dtype in ("float32", "bfloat16"):
        folder = make_folder(tmp_path / dtype, config, seed=6, dtype=dtype, sharpen=3.0)
        plain_config, weights = plain.read_model(folder)
        if kind == "wkv":                                        # decays of a few thousandths a token
            from libmir_b200.weights import load_tensor, read_catalog, write_file
            tensors = {name: load_tensor(entry) for name, entry in read_catalog(folder).items()}
            tensors["l0.mix.w0"] = tensors["l0.mix.w0"] - 6.0
            write_file(folder / "model.safetensors", tensors)
            plain_config, weights = plain.read_model(folder)
        want = plain.forward(plain_config, weights, ids).numpy()
        early = 250 if kind == "wide" else 60                    # (a bias takes weight off what lies far back)
        changed = [(t + 1) % 90 for t in ids[:early]] + ids[early:]
        moved = relative_error(plain.forward(plain_config, weights, changed).numpy()[-20:], want[-20:])
        assert np.median(moved) > 5e-3, f"{kind}: the first tokens hardly matter ({np.median(moved):.1e})"
        model = load(folder, dtype, 16, 50)
        for label, cuts in (("whole", [700]), ("late", [650, 1]), ("cut", [15, 17, 300, 2, 31])):
            got = feed(model, label, ids, cuts)
            close_logits(got, want, dtype, f"{kind}, {label}, {dtype}")
            if dtype == "float32":
                assert relative_error(got, want).max() < 0.05 * np.median(moved)


@pytest.mark.parametrize("dim,page,keep", [(24, 8, 5), (64, 4, 0), (64, 16, 3), (128, 16, 17)])
def test_the_windows_edges_show_in_the_logits(tmp_path, dim, page, keep):
    """Two attention layers with windows, sharp scores: the plain implementation with a window one token wider or narrower,
    or with one kept token more or less, gives other logits, and the engine gives the configured ones', in a prompt and in
    decoding (heads of 24 channels run the reference kernel, of 64 and 128 the tensor-core kernels in bfloat16)."""
    def model_config(size, kept):
        mixer = {"heads": 2, "kv_heads": 1, "dim": dim, "vdim": dim, "scale": 0.5 / math.sqrt(dim),
                 "mask": {"size": size, "keep_first": kept}, "rot": {"dims": 8, "base": 100.0}}
        return {"architecture": "Biravik", "vocab": 80, "width": 64, "norm": {"eps": 1e-5}, "postln_alpha": 0.4,
                "layers": [{"type": "attention", "mlp": None, "mixer": mixer}] * 2}
    config = model_config(29, keep)
    ids = random_ids(np.random.default_rng(dim), 80, 120)
    others = [model_config(30, keep), model_config(28, keep), model_config(29, keep + 1)]
    if keep:
        others.append(model_config(29, keep - 1))
    for dtype in ("float32", "bfloat16"):
        folder = make_folder(tmp_path / dtype, config, seed=8, dtype=dtype, sharpen=1.0)
        _, weights = plain.read_model(folder)
        want = plain.forward(config, weights, ids).numpy()
        seen = []
        for other in others:
            moved = relative_error(plain.forward(other, weights, ids).numpy(), want)
            seen.append(np.median(moved[60:]))
            assert seen[-1] > 0.01                               # a window or a kept token off by one is seen
        model = load(folder, dtype, page, 80)
        for label, cuts in (("whole", [120]), ("decoded", [30, 1]), ("portions", [28, 2, 19, 2, 1, 22])):
            relative = relative_error(feed(model, label, ids, cuts), want)
            if dtype == "float32":
                assert relative.max() <= 2e-4, f"{label}: {relative.max():.3e} at position {int(relative.argmax())}"
            else:
                assert np.median(relative[60:]) <= 0.5 * min(seen) and relative.max() <= 1.5 * TOL[dtype], \
                    f"{label}/{dtype}: median {np.median(relative[60:]):.3e} of {min(seen):.3e}, max {relative.max():.3e}"


@pytest.mark.parametrize("graphs", [False, True])
@pytest.mark.parametrize("name", ["A", "B"])
def test_greedy_generation_through_the_scheduler(tmp_path, name, graphs):
    """Model.generate_batch (scheduler, sampler, decode steps as captured graphs or not) against the plain implementation
    choosing greedily; float32, so that equal choices are expected wherever the best two logits are not closer than the
    tolerance."""
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


@pytest.mark.parametrize("name", ["A", "C", "D"])
def test_decode_steps_replayed_from_captured_graphs_in_bfloat16(tmp_path, name):
    """Two requests decoded together through captured graphs in bfloat16: the teacher-forced logits of every step against
    the plain implementation."""
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


def test_the_tensor_core_kernels_run_where_the_sizes_fit(tmp_path):
    """A step function that fell back to the reference attention kernel would still be right: count the launches."""
    from libmir_b200 import StepEntry, kernels
    folder = make_folder(tmp_path, ALL["D"], seed=3, dtype="bfloat16")
    model = load(folder, "bfloat16", 16, 40)
    ids = random_ids(np.random.default_rng(3), 97, 90)
    kernels.launch_counts(reset=True)
    model.admit("x")
    model.step([StepEntry("x", ids[:80], [0])])
    for token in ids[80:]:
        model.step([StepEntry("x", [token], [0])])
    counts = kernels.launch_counts()
    assert counts.get("paged_attention_generic", 0) == 0
    assert counts.get("prefill_attention_tc", 0) == 3 and counts.get("prefill_attention", 0) == 1     # (values of 32)
    assert counts.get("decode_attention_tc", 0) == 20 and counts.get("decode_attention", 0) == 20     # (and kept tokens)
    assert counts.get("norm_scaled_sum", 0) == 11 * 7


def test_trace_runner_picks_the_design_by_its_configuration(tmp_path):
    """bin/trace_run as a user runs it: the model class comes from config.json; prompts in portions, decoded tokens, a pool
    that holds less than all requests together."""
    config = ALL["A"]
    folder = make_folder(tmp_path / "model", config, seed=4, dtype="bfloat16")
    (folder / "config.json").write_text(json.dumps(dict(config, vocab_size=config["vocab"])))   # (helpers read this key)
    rng = np.random.default_rng(3)
    requests = {f"q{i}": random_ids(rng, config["vocab"], n) for i, n in enumerate((100, 64, 37))}
    want = {name: reference(folder, ids) for name, ids in requests.items()}
    # (the third run replays every single-token step from a captured graph, as generation does)
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
    """bin/generate on a model folder of the design: two prompts as one batch, greedy, against the plain implementation."""
    import subprocess
    import sys
    from helpers import ROOT
    folder = make_folder(tmp_path / "model", ALL["D"], seed=12, dtype="float32")
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


@pytest.mark.parametrize("seed", range(10))
def test_configurations_drawn_at_random(tmp_path, seed):
    """Sizes nobody chose: a prompt whole, token by token, in portions and as a prompt followed by decoding, in both dtypes,
    against the plain implementation (32-bit: the same bits under every cut; bfloat16: nine positions in ten within the
    tolerance, or within four times what rounding the sublayers' inputs alone does to the 64-bit implementation where a
    model drawn at random magnifies that)."""
    rng = np.random.default_rng(900 + seed)
    config = random_config(rng)
    page = int(rng.choice([4, 8, 16]))
    ids = random_ids(rng, config["vocab"], 100)
    for dtype in ("float32", "bfloat16"):
        folder = make_folder(tmp_path / dtype, config, seed=seed, dtype=dtype)
        want = reference(folder, ids)
        bound = TOL["bfloat16"]
        if dtype == "bfloat16":
            rounded = plain.forward(*plain.read_model(folder), ids, read=lambda h: h.to(BF16).double()).numpy()
            bound = max(bound, 4.0 * np.quantile(relative_error(rounded, want), 0.9))
        model = load(folder, dtype, page, 80)
        outputs = [feed(model, "whole", ids, [len(ids)]), feed(model, "single", ids, [1]),
                   feed(model, "portions", ids, [2, 5, 1, 33, 3, 16, 2, 7]), feed(model, "late", ids, [80, 1])]
        for got in outputs:
            relative = relative_error(got, want)
            assert np.isfinite(relative).all(), json.dumps(config)
            if dtype == "float32":
                assert relative.max() <= 2e-4, f"{relative.max():.3e} at {int(relative.argmax())}: {json.dumps(config)}"
            else:
                assert np.quantile(relative, 0.9) <= bound, f"{bound:.3e} < {np.quantile(relative, 0.9):.3e}: {json.dumps(config)}"
        if dtype == "float32":
            assert all(np.array_equal(outputs[0], other) for other in outputs[1:]), json.dumps(config)
        model.unload()
