"""The kernels of the Nodepel parts alone, each against the stand-in of the same name
(``fake_kernels``: float64, rounded once), at sizes other than any model's and in both types: the
delta rule at every register layout, with portions on either side of its blocks of eight rows, states
carried over and q and k shared by several heads; its step of single rows in one launch against the
three separate calls; the output norm with its gate; the 16-byte convolution; sinks on every route of the softmax
attention; the joined head norm with a rotation; the pair of normed branches; ungated experts."""

import math

import pytest
import torch

import fake_kernels as fake
from test_kernels_gpu import close, make_step, ops, rnd

pytestmark = pytest.mark.gpu
DTYPES = [torch.float32, torch.bfloat16]


def delta_inputs(tokens, heads, groups, dim, vdim, dtype, seed, pad):
    """Columns [q | k | v | gate | b | a] of rows that are `pad` wider, and the per-head constants."""
    c, v = 2 * groups * dim + heads * vdim, heads * vdim
    rows = rnd((tokens, c + v + 2 * heads + pad), dtype, seed)
    return rows, c, v, rnd((heads,), torch.float32, seed + 1), rnd((heads,), torch.float32, seed + 2) - 1.0


SHAPES = [(4, 4, 128, 128, 0), (6, 3, 64, 40, 8), (3, 1, 32, 64, 8), (2, 2, 200, 24, 4), (5, 5, 130, 16, 6), (4, 2, 256, 32, 0), (3, 3, 7, 5, 1),
          (18, 1, 16, 12, 2), (2, 1, 96, 200, 0)]


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("shape", SHAPES)
def test_delta_rule(dtype, shape):
    heads, groups, dim, vdim, pad = shape
    t = ops()
    q_lens, starts = [9, 1, 40, 8, 7, 16, 2], [0, 5, 3, 0, 17, 8, 1]
    cpu, gpu, _ = make_step(q_lens, starts, 16, 40, 3, num_slots=9)
    rows, c, v, dt_bias, a_log = delta_inputs(sum(q_lens), heads, groups, dim, vdim, dtype, 5, pad)
    gd = groups * dim
    state = rnd((9, heads, dim, vdim), torch.float32, 9, 0.3)
    for untouched in (False, True):  # a view into wider slots, as the cache manager hands out
        wide = torch.zeros(9, heads * dim * vdim + (4 if not untouched else 3))
        wide[:, : heads * dim * vdim] = state.reshape(9, -1)
        views = []
        for device in ("cpu", "cuda"):
            buf = wide.clone().to(device)
            views.append((buf, buf[:, : heads * dim * vdim].view(9, heads, dim, vdim) if device == "cpu" else
                          buf.as_strided((9, heads, dim, vdim), (wide.shape[1], dim * vdim, vdim, 1))))

        def run(table, x, s, step, dev):
            b, a = x[:, c + v : c + v + heads], x[:, c + v + heads : c + v + 2 * heads]
            return table.delta_rule(x[:, :gd], x[:, gd : 2 * gd], x[:, 2 * gd : c], b, a, dt_bias.to(dev), a_log.to(dev), s, step, heads, groups,
                                    dim, vdim, dim**-0.5, 1e-6)

        want = run(fake, rows, views[0][1], cpu, "cpu")
        got = run(t, rows.cuda(), views[1][1], gpu, "cuda")
        # (float inside whatever the input type: both types are held to float's bound; 40 rows of a recurrence)
        close(got, want, torch.float32, f"delta rule {shape} {dtype}", rel32=2e-5)
        close(views[1][0], views[0][0], torch.float32, f"its states {shape} {dtype}", rel32=2e-5)


@pytest.mark.parametrize("dtype", DTYPES)
def test_delta_rule_over_a_long_portion_and_over_cuts_of_it(dtype):
    """1,000 rows whole against the stand-in and against the same rows in portions."""
    heads, groups, dim, vdim = 3, 3, 64, 32
    t = ops()
    rows, c, v, dt_bias, a_log = delta_inputs(1000, heads, groups, dim, vdim, dtype, 15, 0)
    a_log = a_log - 3.0  # long memories
    gd = groups * dim

    def run(table, x, s, step, dev):
        b, a = x[:, c + v : c + v + heads], x[:, c + v + heads :]
        return table.delta_rule(x[:, :gd], x[:, gd : 2 * gd], x[:, 2 * gd : c], b, a, dt_bias.to(dev), a_log.to(dev), s, step, heads, groups, dim, vdim, dim**-0.5, 1e-6)

    cpu, gpu, _ = make_step([1000], [0], 16, 80, 3)
    s_cpu, s_gpu, s_cut = torch.zeros(1, heads, dim, vdim), torch.zeros(1, heads, dim, vdim).cuda(), torch.zeros(1, heads, dim, vdim).cuda()
    want = run(fake, rows, s_cpu, cpu, "cpu")
    got = run(t, rows.cuda(), s_gpu, gpu, "cuda")
    close(got, want, torch.float32, "1,000 rows", rel32=2e-5)
    close(s_gpu, s_cpu, torch.float32, "their state", rel32=2e-5)
    at, parts = 0, []
    for n in (1, 2, 3, 250, 8, 7, 129, 600):
        _, step, _ = make_step([n], [at], 16, 80, 3)
        parts.append(run(t, rows[at : at + n].cuda(), s_cut, step, "cuda"))
        at += n
    close(torch.cat(parts), got, torch.float32, "in portions", rel32=1e-5)


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("taps", [2, 4, 8])
@pytest.mark.parametrize("shape", SHAPES)
def test_delta_step_is_the_three_calls_in_one(dtype, taps, shape):
    heads, groups, dim, vdim, pad = shape
    t = ops()
    S = 5
    cpu, gpu, _ = make_step([1] * S, [0, 3, 63, 64, 700], 16, 120, 3, num_slots=8)
    rows, c, v, dt_bias, a_log = delta_inputs(S, heads, groups, dim, vdim, dtype, 25, pad)
    gd = groups * dim
    conv = rnd((c, taps), torch.float32, 26, 0.5)
    norm = 1.0 + 0.2 * rnd((vdim,), torch.float32, 27)
    window, state = rnd((8, taps - 1, c), torch.float32, 28), rnd((8, heads, dim, vdim), torch.float32, 29, 0.3)
    w_cpu, s_cpu, w_gpu, s_gpu = window.clone(), state.clone(), window.clone().cuda(), state.clone().cuda()
    qkv = fake.causal_conv(rows[:, :c], conv, None, w_cpu, cpu)
    raw = fake.delta_rule(qkv[:, :gd], qkv[:, gd : 2 * gd], qkv[:, 2 * gd :], rows[:, c + v : c + v + heads], rows[:, c + v + heads : c + v + 2 * heads],
                          dt_bias, a_log, s_cpu, cpu, heads, groups, dim, vdim, dim**-0.5, 1e-6)
    want = fake.delta_output(raw, rows[:, c : c + v], norm, heads, 1e-5, torch.zeros(S, v, dtype=dtype))
    gpu.all_decode = True
    out = torch.zeros(S, v, dtype=dtype, device="cuda")
    x = rows.cuda()
    got = t.delta_step(x[:, : c + v + 2 * heads], c, conv.cuda(), dt_bias.cuda(), a_log.cuda(), norm.cuda(), w_gpu, s_gpu, gpu, heads, groups, dim, vdim,
                       dim**-0.5, 1e-6, 1e-5, out)
    assert got is out
    assert torch.equal(w_gpu.cpu(), w_cpu), "the windows moved on"
    # (bfloat16: a convolution's output on a rounding border may fall to either side, one part in 256 of one input)
    loose = dtype == torch.bfloat16
    close(s_gpu, s_cpu, torch.float32, f"states {shape}", rel32=4e-3 if loose else 5e-6)
    rms = (got.double().cpu() - want.double()).pow(2).mean().sqrt().item() / want.double().pow(2).mean().sqrt().item()
    assert rms <= (1e-2 if loose else 1e-5), f"outputs {shape}: {rms:.2e}"
    gpu.all_decode = False
    assert t.delta_step(x[:, : c + v + 2 * heads], c, conv.cuda(), dt_bias.cuda(), a_log.cuda(), norm.cuda(), w_gpu, s_gpu, gpu, heads, groups, dim, vdim,
                        dim**-0.5, 1e-6, 1e-5, out) is None


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("case", [(7, 4, 128, 0), (33, 3, 40, 5), (2, 5, 7, 1), (9, 2, 300, 4)])
def test_delta_output(dtype, case):
    tokens, heads, vdim, pad = case
    width = heads * vdim
    x = rnd((tokens, width), torch.float32, 31) * torch.logspace(-3, 2, tokens)[:, None]
    gates = rnd((tokens, width + 2 * pad), dtype, 32, 2.0)
    w = 1.0 + 0.2 * rnd((vdim,), torch.float32, 33)
    outs = torch.zeros(tokens, width + pad, dtype=dtype)
    want = fake.delta_output(x, gates[:, pad : pad + width], w, heads, 1e-5, outs.clone()[:, :width])
    got = outs.cuda()
    ops().delta_output(x.cuda(), gates.cuda()[:, pad : pad + width], w.cuda(), heads, 1e-5, got[:, :width])
    close(got[:, :width], want, dtype, f"delta output {case}")
    assert not got[:, width:].any()


@pytest.mark.parametrize("taps", [2, 3, 4, 5])
@pytest.mark.parametrize("channels,pad", [(64, 8), (136, 0), (50, 3), (1032, 16)])
def test_convolution_of_rows_that_allow_wide_accesses(taps, channels, pad):
    """Runs of eight rows inside a sequence, across several, behind a portion's start; wide and narrow kernels."""
    q_lens, starts = [21, 1, 2, 8, 40, 3, 1], [0, 9, 1, 2, 100, 0, 30]
    cpu, gpu, _ = make_step(q_lens, starts, 16, 40, 41, num_slots=9)
    x = rnd((sum(q_lens), channels + pad), torch.bfloat16, 42)
    w, bias = rnd((channels, taps), torch.float32, 43), rnd((channels,), torch.float32, 44)
    for b, silu in ((None, True), (bias, False)):
        s_cpu = rnd((9, taps - 1, channels), torch.float32, 45)
        s_gpu = s_cpu.clone().cuda()
        want = fake.causal_conv(x[:, :channels], w, b, s_cpu, cpu, silu)
        got = ops().causal_conv(x.cuda()[:, :channels], w.cuda(), b.cuda() if b is not None else None, s_gpu, gpu, silu)
        close(got, want, torch.bfloat16, f"convolution {channels} x {taps}")
        assert torch.equal(s_gpu.cpu(), s_cpu)


ATTENTION = [  # heads, kv heads, key size, value size, page: tensor memory / TMA; tiles; general
    (8, 2, 64, 64, 16), (4, 1, 96, 96, 16), (3, 3, 128, 48, 8), (5, 1, 20, 12, 4), (2, 2, 256, 256, 16)]


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("all_decode", [False, True])
@pytest.mark.parametrize("case", ATTENTION)
def test_sinks_on_every_route(dtype, all_decode, case):
    """Sinks far below, among and far above the scores, one per head; windows whose edge a planted key
    stands on: inside it takes nearly everything (but for the sink's share), outside it is not felt."""
    heads, kv_heads, dim, vdim, page = case
    t = ops()
    q_lens, starts = ([1] * 6, [0, 3, 63, 200, 700, 129]) if all_decode else ([150, 1, 33, 260], [0, 40, 129, 500])
    pages = sum(-(-(s + n) // page) for s, n in zip(starts, q_lens)) + 3
    cpu, gpu, table = make_step(q_lens, starts, page, pages, 51)
    gpu.h_q_start = cpu.q_start.tolist()
    cpu.all_decode = gpu.all_decode = all_decode
    cpu.max_q_len = gpu.max_q_len = max(q_lens)
    tokens = sum(q_lens)
    k, v = rnd((pages, page, kv_heads, dim), dtype, 52), rnd((pages, page, kv_heads, vdim), dtype, 53)
    rows = rnd((tokens, heads * dim + 16), dtype, 54)
    scale = 1.0 / math.sqrt(dim)
    for size in (1, 40, 64, 100, 1000):
        # each sequence's last row asks for the key just inside its window, and would weigh the one just outside more
        for s, (n, start) in enumerate(zip(q_lens, starts)):
            last, row = start + n - 1, int(cpu.q_start[s + 1]) - 1
            for back, much in ((size - 1, 2.0), (size, 4.0)):
                if back <= last and back > 0:
                    p = last - back
                    k[int(table[s, p // page]), p % page] = rows[row, :dim] * much
        sinks = torch.tensor([-50.0, 0.5, 3.0, 40.0, 2.0, -3.0, 1.0, 12.0])[:heads]
        q = rows[:, : heads * dim]
        want = fake.masked_attention(q, heads, k, v, table, page, scale, "window", size, 0, cpu, sink=sinks)
        given = torch.zeros(tokens, heads * vdim, dtype=dtype, device="cuda")
        for more in ({}, {"general": True}, {"out": given}):
            got = t.masked_attention(rows.cuda()[:, : heads * dim], heads, k.cuda(), v.cuda(), table.cuda(), page, scale, "window", size, 0, gpu,
                                     sink=sinks.cuda(), **more)
            close(got, want, dtype, f"sinks {case} window {size} decode {all_decode} {list(more)}", rel32=1e-5)
        assert got is given
    t.check_kernel_status()


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("case", [(8, 2, 64, 64, 64), (4, 4, 48, 80, 32), (6, 1, 96, 96, 96), (3, 1, 20, 7, 6), (2, 2, 16, 8, 2), (2, 1, 256, 64, 256)])
def test_joined_norm_with_a_rotation(dtype, case):
    heads, kv_heads, dim, vdim, rot = case
    page = 16
    for q_lens, starts in (([1, 1, 1], [5, 700, 64]), ([130, 3, 70], [0, 37, 1000])):
        pages = sum(-(-(s + n) // page) for s, n in zip(starts, q_lens)) + 2
        cpu, gpu, table = make_step(q_lens, starts, page, pages, 61)
        tokens = sum(q_lens)
        proj = rnd((tokens, (heads + kv_heads) * dim + kv_heads * vdim + 8), dtype, 62)
        q_w, k_w = (1.0 + 0.2 * rnd((n * dim,), torch.float32, 63) for n in (heads, kv_heads))
        inv_freq = 10000.0 ** (-torch.arange(rot // 2, dtype=torch.float32) * 2 / rot)
        k, v = torch.zeros(pages, page, kv_heads, dim, dtype=dtype), torch.zeros(pages, page, kv_heads, vdim, dtype=dtype)
        want, want_k, want_v = proj.clone(), k.clone(), v.clone()
        fake.joined_norm_store(want, heads, kv_heads, dim, vdim, q_w, k_w, 1e-5, None, False, cpu, want_k, want_v, table, page, inv_freq, rot)
        got, got_k, got_v = proj.cuda(), k.cuda(), v.cuda()
        ops().joined_norm_store(got, heads, kv_heads, dim, vdim, q_w.cuda(), k_w.cuda(), 1e-5, None, False, gpu, got_k, got_v, table.cuda(), page,
                                inv_freq.cuda(), rot)
        close(got, want, dtype, f"queries {case}", slack=2e-4)
        close(got_k, want_k, dtype, f"keys {case}", slack=2e-4)
        assert torch.equal(got_v.cpu(), want_v) and torch.equal(got[:, heads * dim :].cpu(), proj[:, heads * dim :])


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("case", [(130, 16, 4, 64, 96), (5, 3, 2, 40, 56), (33, 9, 1, 33, 50), (1, 2, 2, 128, 256)])
def test_ungated_experts(dtype, case):
    tokens, experts, top, ff, hidden = case
    x = rnd((tokens, hidden), dtype, 71)
    up, down = rnd((experts, ff, hidden), dtype, 72, 0.1), rnd((experts, hidden, ff), dtype, 73, 0.1)
    logits = rnd((tokens, experts), torch.float32, 74, 2.0)
    ids, weights = fake.moe_route(logits, top, 1, 1, 1.0, scores="chosen_softmax")
    got_ids, got_weights = ops().moe_route(logits.cuda(), top, 1, 1, 1.0, scores="chosen_softmax")
    assert torch.equal(got_ids.cpu(), ids)
    close(got_weights, weights, torch.float32, "weights")
    extra, gate = rnd((tokens, hidden), dtype, 75), rnd((tokens, 1), torch.float32, 76)
    want = fake.routed_experts(x, ids, weights, up, down, extra, act="relu2", extra_gate=gate)
    got = ops().routed_experts(x.cuda(), ids.cuda(), weights.cuda(), up.cuda(), down.cuda(), extra.cuda(), act="relu2", extra_gate=gate.cuda())
    close(got, want, dtype, f"ungated experts {case}")
