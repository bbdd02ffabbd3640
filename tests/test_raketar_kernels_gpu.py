"""The kernels of the Raketar parts alone, each against the stand-in of the same name
(``fake_kernels``: float64, rounded once), at sizes other than any model's and in both types: the
softmax maps on every route of the masked attention kernels with shared value heads and float output,
the difference behind them, and both in one launch (prompt portions in tensor memory, single tokens by
TMA) with planted keys at tile, page and window edges; the matrix memory's gates, its walked and
its chunked recurrence with carried states and long portions, its output, its step of single rows in
one launch against the calls it replaces; weights on the experts' inputs; the side input's gate; rows
added to the stream; the normed output."""

import math

import pytest
import torch

import fake_kernels as fake
from test_kernels_gpu import close, make_step, ops, rnd

pytestmark = pytest.mark.gpu
DTYPES = [torch.float32, torch.bfloat16]


# --------------------------------------------------------------------------- differential attention


def attention_step(q_lens, starts, page, all_decode, seed):
    pages = sum(-(-(s + n) // page) for s, n in zip(starts, q_lens)) + 3
    cpu, gpu, table = make_step(q_lens, starts, page, pages, seed)
    gpu.h_q_start = cpu.q_start.tolist()
    cpu.all_decode = gpu.all_decode = all_decode
    cpu.max_q_len = gpu.max_q_len = max(q_lens)
    return cpu, gpu, table, pages


SHARED = [  # pairs, groups, map size, value size, page: tiles or TMA sizes, odd sizes, wide heads
    (4, 2, 64, 128, 16), (6, 1, 32, 64, 8), (3, 3, 16, 48, 16), (2, 1, 20, 12, 4), (2, 2, 7, 5, 4), (2, 1, 128, 200, 16)]


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("all_decode", [False, True])
@pytest.mark.parametrize("case", SHARED)
def test_maps_over_shared_values_and_their_difference(dtype, all_decode, case):
    pairs, groups, dim, vdim, page = case
    t = ops()
    q_lens, starts = ([1] * 5, [0, 3, 63, 200, 129]) if all_decode else ([90, 1, 33, 2], [0, 40, 129, 70])
    cpu, gpu, table, pages = attention_step(q_lens, starts, page, all_decode, 51)
    tokens, scale = sum(q_lens), 1.0 / math.sqrt(dim)
    k, v = rnd((pages, page, 2 * groups, dim), dtype, 52), rnd((pages, page, groups, vdim), dtype, 53)
    rows = rnd((tokens, 2 * pairs * dim + pairs * vdim + 8), dtype, 54)
    q, gate = rows[:, : 2 * pairs * dim], rows[:, 2 * pairs * dim : 2 * pairs * dim + pairs * vdim]
    want = fake.masked_attention(q, 2 * pairs, k, v, table, page, scale, "window", 1 << 30, 0, cpu, out_dtype=torch.float32)
    outs = torch.zeros(tokens, pairs * vdim + 8, dtype=dtype)
    want_d = fake.map_difference(want, pairs, groups, 0.45, 0.7, 1e-6, gate, outs.clone()[:, : pairs * vdim])
    dev = rows.cuda()
    q_dev, gate_dev = dev[:, : 2 * pairs * dim], dev[:, 2 * pairs * dim : 2 * pairs * dim + pairs * vdim]
    for general in (True, False):
        got = t.masked_attention(q_dev, 2 * pairs, k.cuda(), v.cuda(), table.cuda(), page, scale, "window", 1 << 30, 0, gpu, general=general,
                                 out_dtype=torch.float32)
        assert got.dtype == torch.float32
        close(got, want, dtype if not general else torch.float32, f"maps {case} general {general}", rel32=1e-5)
        plain = t.masked_attention(q_dev, 2 * pairs, k.cuda(), v.cuda(), table.cuda(), page, scale, "window", 1 << 30, 0, gpu, general=general)
        close(plain, want, dtype, f"maps in the row type {case}", rel32=1e-5)
    got = outs.cuda()
    t.map_difference(want.cuda(), pairs, groups, 0.45, 0.7, 1e-6, gate_dev, got[:, : pairs * vdim])
    close(got[:, : pairs * vdim], want_d, dtype, f"difference {case}", rel32=1e-5)
    assert not got[:, pairs * vdim :].any()


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("case", [(8, 4, 2, 64, 128, 64), (4, 4, 1, 48, 80, 32), (6, 2, 1, 20, 7, 6), (4, 4, 2, 16, 24, 0)])
def test_keys_and_fewer_value_heads_are_stored(dtype, case):
    heads, kv_heads, v_heads, dim, vdim, rot = case
    page = 16
    cpu, gpu, table, pages = attention_step([130, 3, 1], [0, 37, 1000], page, False, 61)
    proj = rnd((134, (heads + kv_heads) * dim + v_heads * vdim + 8), dtype, 62)
    inv_freq = 10000.0 ** (-torch.arange(max(rot // 2, 1), dtype=torch.float32) * 2 / max(rot, 1))
    k, v = torch.zeros(pages, page, kv_heads, dim, dtype=dtype), torch.zeros(pages, page, v_heads, vdim, dtype=dtype)
    want, want_k, want_v = proj.clone(), k.clone(), v.clone()
    fake.head_prepare_store(want, heads, kv_heads, dim, vdim, None, None, 0.0, None, inv_freq, rot, 1.0, cpu, want_k, want_v, table, page)
    got, got_k, got_v = proj.cuda(), k.cuda(), v.cuda()
    ops().head_prepare_store(got, heads, kv_heads, dim, vdim, None, None, 0.0, None, inv_freq.cuda(), rot, 1.0, gpu, got_k, got_v, table.cuda(), page)
    close(got, want, dtype, f"queries {case}", slack=2e-4)
    close(got_k, want_k, dtype, f"keys {case}", slack=2e-4)
    assert torch.equal(got_v.cpu(), want_v)


IN_ONE = [(4, 2, 64, 128, 16), (5, 1, 32, 64, 8), (8, 1, 64, 64, 64), (2, 2, 32, 128, 32)]


@pytest.mark.parametrize("all_decode", [False, True])
@pytest.mark.parametrize("case", IN_ONE)
@pytest.mark.parametrize("window", [1 << 30, 1, 64, 100])
def test_differential_attention_in_one_launch(all_decode, case, window):
    """Against the maps and their difference apart; with a key made to stand out - for one map of one head -
    at the sequence's first positions, at tile and page edges, just inside and just outside the window."""
    pairs, groups, dim, vdim, page = case
    t = ops()
    q_lens, starts = ([1] * 7, [0, 3, 63, 64, 700, 1500, 129]) if all_decode else ([300, 1, 33, 260], [0, 40, 129, 500])
    cpu, gpu, table, pages = attention_step(q_lens, starts, page, all_decode, 71)
    tokens, scale = sum(q_lens), 1.0 / math.sqrt(dim)
    k, v = rnd((pages, page, 2 * groups, dim), torch.bfloat16, 72), rnd((pages, page, groups, vdim), torch.bfloat16, 73)
    rows = rnd((tokens, 2 * pairs * dim + pairs * vdim), torch.bfloat16, 74)
    per = pairs // groups
    for s, (n, start) in enumerate(zip(q_lens, starts)):
        last, row = start + n - 1, int(cpu.q_start[s + 1]) - 1
        spots = {0, 1, 62, 63, 64, last // 2, last - window, last - window + 1, last - 1}
        for i, p in enumerate(sorted(x for x in spots if 0 <= x < last)):
            m, group = i % 2, i % groups
            sub = ((2 * group + m) * per) * dim
            k[int(table[s, p // page]), p % page, 2 * group + m] = rows[row, sub : sub + dim] * (1.0 + 0.5 * (i % 3))
    dev, kd, vd, td = rows.cuda(), k.cuda(), v.cuda(), table.cuda()
    q, gate = dev[:, : 2 * pairs * dim], dev[:, 2 * pairs * dim :]
    want = torch.empty(tokens, pairs * vdim, dtype=torch.bfloat16, device="cuda")
    maps = t.masked_attention(q, 2 * pairs, kd, vd, td, page, scale, "window", window, 0, gpu, general=True, out_dtype=torch.float32)
    t.map_difference(maps, pairs, groups, 0.3, 0.6, 1e-6, gate, want)
    out = torch.zeros_like(want)
    got = t.differential_attention(q, pairs, groups, kd, vd, td, page, scale, window, 0, gpu, 0.3, 0.6, 1e-6, gate, out)
    assert got is out
    t.check_kernel_status()
    # (P is rounded to bfloat16 ahead of the second product, and the difference is brought to unit size behind it)
    ratio = (out.double() - want.double()).view(tokens, pairs, vdim).pow(2).mean(-1).sqrt() / want.double().view(tokens, pairs, vdim).pow(2).mean(-1).sqrt().clamp_min(1e-9)
    assert ratio.median().item() <= 5e-3 and (ratio > 3e-2).double().mean().item() <= 0.01 and ratio.max().item() <= 0.3, (ratio.median(), ratio.max())


def test_what_the_one_launch_refuses():
    t = ops()
    cpu, gpu, table, pages = attention_step([300], [0], 16, False, 81)
    for dtype, dim, vdim, keep, scale in ((torch.float32, 64, 128, 0, 0.1), (torch.bfloat16, 48, 128, 0, 0.1), (torch.bfloat16, 64, 96, 0, 0.1),
                                          (torch.bfloat16, 64, 128, 3, 0.1), (torch.bfloat16, 64, 128, 0, -0.1)):
        k, v = torch.zeros(pages, 16, 4, dim, dtype=dtype, device="cuda"), torch.zeros(pages, 16, 2, vdim, dtype=dtype, device="cuda")
        rows = torch.zeros(300, 4 * dim + 2 * vdim, dtype=dtype, device="cuda")
        out = torch.zeros(300, 2 * vdim, dtype=dtype, device="cuda")
        assert t.differential_attention(rows[:, : 4 * dim], 2, 2, k, v, table.cuda(), 16, scale, 1 << 30, keep, gpu, 0.3, 0.6, 1e-6, rows[:, 4 * dim :], out) is None


# --------------------------------------------------------------------------- matrix memory


def memory_inputs(tokens, heads, dim, vdim, dtype, seed, pad, forget=3.0):
    rows = rnd((tokens, 2 * heads * (dim + vdim) + pad), dtype, seed)
    logits = rnd((tokens, 2 * heads), torch.float32, seed + 1, 2.0)
    logits[:, heads:] += forget
    return rows, logits, 1.0 + 0.2 * rnd((heads * vdim,), torch.float32, seed + 2)


def memory_state(slots, heads, dim, vdim, seed, zero=False):
    f = 0.0 if zero else 1.0
    return (rnd((slots, heads, dim, vdim), torch.float32, seed, 0.3 * f), rnd((slots, heads, dim), torch.float32, seed + 1, 0.3 * f),
            rnd((slots, heads), torch.float32, seed + 2).abs() * f)


def run_memory(table, rows, logits, weight, state, step, heads, dim, vdim, dtype, dev, logs=None, cap=15.0):
    qk, v = heads * dim, heads * vdim
    S, n, top = state
    more = {"logs": True} if logs else {}
    keep, add, floor = table.memory_gates(logits.to(dev), cap, top, step, **more)
    raw, read = table.memory_recurrence(rows[:, :qk], rows[:, qk : 2 * qk], rows[:, 2 * qk : 2 * qk + v], keep, add, S, n, step, heads, dim, vdim, **more)
    out = torch.zeros(rows.shape[0], v, dtype=dtype, device=dev)
    table.memory_output(raw, read, floor, rows[:, 2 * qk + v : 2 * (qk + v)], weight.to(dev), heads, vdim, dim**-0.5, 1e-6, 1e-5, out)
    return raw, read, floor, out


def wide_views(state, pad):
    """Device views into wider slots, as the cache manager hands out."""
    views = []
    for s in state:
        flat = torch.zeros(s.shape[0], s[0].numel() + pad, device="cuda")
        view = flat[:, : s[0].numel()].unflatten(1, s.shape[1:])
        view.copy_(s)
        views.append(view)
    return tuple(views)


MEMORY = [(4, 128, 128, 0), (3, 48, 40, 8), (2, 16, 8, 8), (1, 112, 136, 0), (2, 7, 5, 1), (3, 200, 12, 4), (2, 256, 66, 2), (5, 32, 1, 3)]


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("shape", MEMORY)
@pytest.mark.parametrize("pad", [4, 3])
def test_matrix_memory(dtype, shape, pad):
    heads, dim, vdim, cols = shape
    t = ops()
    q_lens, starts = [9, 1, 64, 130, 63, 2], [0, 5, 3, 0, 17, 8]
    cpu, gpu, _ = make_step(q_lens, starts, 16, 60, 3, num_slots=9)
    rows, logits, weight = memory_inputs(sum(q_lens), heads, dim, vdim, dtype, 5, cols)
    ref = memory_state(9, heads, dim, vdim, 9)
    got_state = wide_views(ref, pad)
    dev = rows.cuda()
    want = run_memory(fake, rows, logits, weight, ref, cpu, heads, dim, vdim, dtype, "cpu")
    routes = [False] + ([True] if t.memory_chunks_supported(dev, dim, vdim) else [])
    if dtype == torch.bfloat16 and dim % 16 == 0 and dim <= 128 and vdim % 8 == 0 and cols % 8 == 0:
        assert routes == [False, True]
    for logs in routes:
        state = tuple(v.clone(memory_format=torch.preserve_format) for v in got_state)
        got = run_memory(t, dev, logits, weight, state, gpu, heads, dim, vdim, dtype, "cuda", logs)
        # (float inside whatever the input type; in chunks, products of split floats keep about 2^-17)
        bound = 3e-5 if logs else 1e-5
        for name, a, b in zip(("numerators", "n . q", "floor"), got, want):
            close(a, b, torch.float32, f"{name} {shape} {dtype} chunks {logs}", rel32=bound)
        for name, a, b in zip(("states", "normalisers", "maxima"), state, ref):
            close(a, b, torch.float32, f"{name} {shape} {dtype} chunks {logs}", rel32=bound)
        rms = (got[3].double().cpu() - want[3].double()).pow(2).mean().sqrt() / want[3].double().pow(2).mean().sqrt()
        assert rms.item() <= (1e-4 if dtype == torch.float32 else 5e-3), (shape, logs, rms)


@pytest.mark.parametrize("forget", [6.0, 0.0, -8.0])
@pytest.mark.parametrize("logs", [False, True])
def test_matrix_memory_over_a_long_portion_and_over_cuts_of_it(logs, forget):
    """1,000 rows whole against the stand-in and against the same rows in portions; memories from a
    few rows to the whole sequence."""
    heads, dim, vdim = 3, 64, 32
    t = ops()
    rows, logits, weight = memory_inputs(1000, heads, dim, vdim, torch.bfloat16, 15, 0, forget)
    cpu, gpu, _ = make_step([1000], [0], 16, 80, 3)
    ref = memory_state(1, heads, dim, vdim, 19, zero=True)
    want = run_memory(fake, rows, logits, weight, ref, cpu, heads, dim, vdim, torch.bfloat16, "cpu")
    for sizes in ([1000], [64, 1, 63, 128, 200], [100]):
        state = tuple(s.cuda() for s in memory_state(1, heads, dim, vdim, 19, zero=True))
        raws, reads, at, i = [], [], 0, 0
        while at < 1000:
            n = min(sizes[i % len(sizes)], 1000 - at)
            _, step, _ = make_step([n], [at], 16, 80, 3)
            raw, read, _, _ = run_memory(t, rows[at : at + n].cuda(), logits[at : at + n].contiguous(), weight, state, step, heads, dim, vdim, torch.bfloat16, "cuda", logs)
            raws.append(raw), reads.append(read)
            at, i = at + n, i + 1
        close(torch.cat(raws), want[0], torch.float32, f"numerators in {sizes}", rel32=5e-5)
        close(torch.cat(reads), want[1], torch.float32, f"n . q in {sizes}", rel32=5e-5)
        for name, a, b in zip(("states", "normalisers", "maxima"), state, ref):
            close(a, b, torch.float32, f"{name} in {sizes}", rel32=5e-5)


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("shape", MEMORY + [(2, 64, 1100, 0)])
def test_the_step_of_single_rows(dtype, shape):
    """One launch against product, gates, recurrence and output; slots in any order, wide and odd strides."""
    heads, dim, vdim, cols = shape
    t, hidden, tokens = ops(), 72, 7
    cpu, gpu, _ = make_step([1] * tokens, [0, 3, 9, 100, 1, 2, 7], 16, 40, 23, num_slots=11)
    rows, _, weight = memory_inputs(tokens, heads, dim, vdim, dtype, 25, cols)
    x, gate_w, gate_b = rnd((tokens, hidden), dtype, 26), rnd((2 * heads, hidden), dtype, 27, 0.2), rnd((2 * heads,), torch.float32, 28)
    logits = fake.linear(x, gate_w, torch.float32, gate_b)
    for pad in (4, 1):
        ref = memory_state(11, heads, dim, vdim, 29)
        state = wide_views(ref, pad)
        want = run_memory(fake, rows, logits, weight, ref, cpu, heads, dim, vdim, dtype, "cpu")[3]
        out = torch.zeros(tokens, heads * vdim, dtype=dtype, device="cuda")
        args = (x.cuda(), gate_w.cuda(), gate_b.cuda(), rows.cuda()[:, : 2 * heads * (dim + vdim)], weight.cuda(), *state, gpu, heads, dim, vdim, 15.0, dim**-0.5, 1e-6, 1e-5, out)
        gpu.all_decode = False
        assert t.memory_step(*args) is None and not out.any()
        gpu.all_decode = True
        assert t.memory_step(*args) is out
        for name, a, b in zip(("states", "normalisers", "maxima"), state, ref):
            close(a, b, torch.float32, f"{name} {shape}", rel32=1e-5)
        rms = (out.double().cpu() - want.double()).pow(2).mean().sqrt() / want.double().pow(2).mean().sqrt()
        assert rms.item() <= (1e-4 if dtype == torch.float32 else 5e-3), (shape, rms)


# --------------------------------------------------------------------------- experts, side input, the stream


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("case", [(130, 16, 4, 64, 96), (5, 3, 2, 40, 56), (33, 9, 1, 33, 50), (1, 2, 2, 128, 256)])
def test_weights_on_the_experts_inputs(dtype, case):
    tokens, experts, top, ff, hidden = case
    x = rnd((tokens, hidden), dtype, 71)
    gate_up, down = rnd((experts, 2 * ff, hidden), dtype, 72, 0.1), rnd((experts, hidden, ff), dtype, 73, 0.1)
    ids, weights = fake.moe_route(rnd((tokens, experts), torch.float32, 74, 2.0), top, 1, 1, 1.0, sigmoid=True)
    extra = rnd((tokens, hidden), dtype, 75)
    for e in (None, extra):
        want = fake.routed_experts(x, ids, weights, gate_up, down, e, weigh_input=True)
        got = ops().routed_experts(x.cuda(), ids.cuda(), weights.cuda(), gate_up.cuda(), down.cuda(), e.cuda() if e is not None else None, weigh_input=True)
        close(got, want, dtype, f"experts {case}")


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("case", [(7, 24, 96, 24), (1, 5, 17, 3), (300, 128, 256, 128)])
def test_side_gate(dtype, case):
    tokens, dim, columns, first = case
    z, table = rnd((tokens, dim), torch.float32, 81, 2.0), rnd((40, columns), dtype, 82)
    ids = torch.arange(tokens, dtype=torch.int32) * 7 % 40
    feed = torch.where(torch.arange(tokens) % 3 == 0, torch.arange(tokens) % 4, torch.full((tokens,), -1)).to(torch.int32)
    fed = torch.tensor([39, 0, 5, 11], dtype=torch.int32)
    for f in ((None, None), (feed, fed)):
        want = fake.side_gate(z, table, first, ids, *f, dtype)
        got = ops().side_gate(z.cuda(), table.cuda(), first, ids.cuda(), *(x.cuda() if x is not None else None for x in f), dtype)
        close(got, want, dtype, f"side gate {case}")


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("width", [50, 64, 2048, 7])
def test_rows_added_to_the_stream_and_the_normed_output(dtype, width):
    x, a, b, w, w2 = (rnd((9, width), torch.float32, 91, 3.0), rnd((9, width), dtype, 92), rnd((9, width), dtype, 93),
                      1.0 + 0.2 * rnd((width,), torch.float32, 94), 1.0 + 0.2 * rnd((width,), torch.float32, 95))
    t = ops()
    for deltas in ((a,), (a, b)):
        for out_dtype in (None, dtype):
            ref, got = x.clone(), x.clone().cuda()
            want = fake.stream_add_rows(ref, deltas, 0.3, out_dtype)
            rows = t.stream_add_rows(got, [d.cuda() for d in deltas], 0.3, out_dtype)
            close(got, ref, torch.float32, f"stream {width}")
            assert (rows is None) == (want is None)
            if rows is not None:
                close(rows, want, dtype, f"rows {width}")
    ref, got = x.clone(), x.clone().cuda()
    want = fake.add_normed_pair_rmsnorm(ref, a, None, w, None, 0.4, 1e-5, w2, 1e-6)
    y = t.add_normed_pair_rmsnorm(got, a.cuda(), None, w.cuda(), None, 0.4, 1e-5, w2.cuda(), 1e-6)
    close(y, want, dtype, f"normed output {width}")
    close(got, ref, torch.float32, f"its stream {width}")
