"""The Raketar design in the engine, on the CPU with the plain stand-in kernels and on the GPU
with the CUDA kernels (``-m gpu``): same bodies.

Everything is compared with ``plain_raketar`` (float64, whole sequences, one function per
mechanism).  The configurations are made here; they differ from each other in every size and in
which options they have: a looped stretch behind the first layer, from the first layer on, over the
last one, or none; a rotation over the whole map, part of it, or none, its ladder stretched or not;
values narrower and wider than the maps; one key/value head or as many as query heads; one expert,
every expert chosen, a shared expert or none; layers without feed-forward; a side
input or none; a residual factor of 1 or another; sizes that no vector width divides.
"""

import copy

import pytest
import torch

import fake_kernels
import helpers
import plain_raketar as plain
import replay
from shiso_llm_b200 import LLM, SamplingParams
from shiso_llm_b200.config import ConfigMissing, InvalidValue, RaketarConfig, plan_from_document
from shiso_llm_b200.parts import (
    BLOCKS, FEED_FORWARDS, MIXERS, NORMS, SIDES, BuildEnv, FixedState, Model, NormedOutput, PagedKV, PartSpec, Stream,
)
from shiso_llm_b200.weights import write_model_folder
from test_zetavik import BACKENDS, Feeder, Reference, backend_args, bind, build_env, close, dtypes, in_steps_and_batches, mixer_dtypes


def attention(heads, kv_heads, dim, vdim, scale, diff, dims, base=100.0, factor=None):
    doc = {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "scale": scale, "diff": diff, "rot": {"dims": dims, "base": base}}
    if factor is not None:
        doc["rot"]["scaling"] = {"factor": factor}
    return doc


def memory(heads, dim, vdim, cap):
    return {"heads": heads, "dim": dim, "vdim": vdim, "gate_cap": cap}


def dense(ff):
    return {"kind": "dense", "ff": ff}


def moe(experts, top, ff, shared=None):
    doc = {"kind": "moe", "expert": {"ff": ff}, "router": {"experts": experts, "top": top}}
    if shared is not None:
        doc["shared"] = {"ff": shared}
    return doc


def layer(mixer, mlp):
    return {"type": "mlstm" if "gate_cap" in mixer else "attention", "mixer": mixer, "mlp": mlp}


# a stretch of two layers behind the first, three passes; a layer without feed-forward inside it
DOC_A = {
    "architecture": "Raketar", "vocab": 300, "width": 48, "norm": {"eps": 1e-5}, "residual_mult": 0.7, "token_side": {"dim": 10},
    "loop": {"start": 1, "stop": 3, "times": 3},
    "layers": [
        layer(memory(4, 12, 8, 5.0), moe(6, 2, 16, 24)),
        layer(attention(4, 2, 12, 8, 0.3, 0.2, 8, 100.0, 2.0), dense(64)),
        layer(memory(2, 8, 16, 10.0), None),
        layer(attention(6, 1, 16, 20, 0.25, 0.6, 16), moe(5, 3, 10)),
    ],
}

# no stretch, a factor of 1, no rotation; heads of one; one expert
DOC_B = {
    "architecture": "Raketar", "vocab": 211, "width": 64, "norm": {"eps": 1e-6}, "residual_mult": 1.0, "token_side": {"dim": 30},
    "layers": [
        layer(attention(1, 1, 20, 24, 0.2, 0.0, 20, 10000.0, 8.0), moe(1, 1, 24, 16)),
        layer(memory(1, 20, 36, 2.0), dense(96)),
        layer(attention(5, 5, 16, 8, 0.3, 0.8, 0), None),
        layer(memory(3, 40, 16, 15.0), moe(8, 1, 40, 32)),
    ],
}

# every layer inside the stretch, from the first on; sizes that no vector width divides
DOC_C = {
    "architecture": "Raketar", "vocab": 333, "width": 50, "norm": {"eps": 1e-5}, "residual_mult": 0.33, "token_side": {"dim": 7},
    "loop": {"start": 0, "stop": 2, "times": 2},
    "layers": [
        layer(attention(3, 1, 6, 5, 0.5, 0.35, 2, 7.0, 1.5), moe(7, 2, 6, 14)),
        layer(memory(3, 7, 5, 6.0), moe(3, 3, 9)),
    ],
}

# a stretch that runs once, over the last layer; no side input; a factor on the residual all the same
DOC_D = {
    "architecture": "Raketar", "vocab": 128, "width": 32, "norm": {"eps": 1e-6}, "residual_mult": 0.5,
    "loop": {"start": 1, "stop": 2, "times": 1},
    "layers": [
        layer(memory(2, 8, 8, 4.0), dense(40)),
        layer(attention(2, 2, 8, 12, 0.3, 0.5, 6), None),
    ],
}

DOCS = {"A": (DOC_A, 3), "B": (DOC_B, 4), "C": (DOC_C, 5), "D": (DOC_D, 6)}


def make_folder(path, doc, seed, std=0.15):
    """Random weights, with router rows that are longer: the choice of experts then differs from token
    to token but seldom hangs on what bfloat16 rounds away."""
    tensors = helpers.make_tensors(doc, seed, std=std)
    for name in tensors:
        if name.endswith(".router"):
            tensors[name] = (tensors[name].float() * 4.0).to(torch.bfloat16)
    write_model_folder(str(path), doc, tensors)
    return tensors


CLOSE_CALL = 0.1  # of a logit of the router


def check_rows(got, ref, dtype, what):
    """Per-row error against the plain logits, relative to their spread.  float32: below 1e-4 in every
    row.  bfloat16: matrices, activations and the cache rounded to 8 bits of mantissa; the median over the
    rows stays below 0.05.  Of the rows without a router's close call in them or before them at most one in
    twenty (or one) is off by more than 0.1 (where a head's or a side input's row is tiny before it is
    brought to unit size, in the stand-in kernels too) and none by half the spread; behind a close call
    none by more than twice the spread."""
    margin = getattr(ref, "margin", None)
    got, ref = got.double(), torch.Tensor(ref).double()
    assert got.shape == ref.shape, (what, got.shape, ref.shape)
    assert torch.isfinite(got).all(), f"{what}: non-finite logits"
    rms = (got - ref).pow(2).mean(-1).sqrt() / ref.std().item()
    if dtype == "float32":
        worst = int(rms.argmax())
        assert rms.max().item() <= 1e-4, f"{what}: row {worst} differs by {rms.max().item():.3e} of the spread"
        return
    touched = torch.cumsum((margin < CLOSE_CALL).long(), 0) > 0 if margin is not None else torch.zeros(len(rms), dtype=torch.bool)
    assert rms.max().item() <= 2.0, f"{what}: a row is off by twice the spread"
    assert len(rms) < 5 or rms.median().item() <= 0.05, f"{what}: half the rows are off by {rms.median().item():.3e} of the spread"
    clean = rms[~touched]
    if clean.numel():
        assert clean.max().item() <= 0.5, f"{what}: a row without a close call differs by {clean.max().item():.3e} of the spread"
        assert int((clean > 0.1).sum()) <= max(1, len(clean) // 20), f"{what}: {int((clean > 0.1).sum())} of {len(clean)} rows differ by more than 0.1 of the spread"


def reference_logits(doc, tensors, tokens):
    margins = []
    logits = plain.plain_logits(doc, dict(tensors), tokens, margins=margins)
    out = logits.as_subclass(Reference)
    out.margin = torch.stack(margins).min(0).values if margins else None
    return out


# --------------------------------------------------------------------------- configuration


def test_configuration_is_read_from_its_own_keys():
    arch, config, plan = plan_from_document(DOC_A)
    assert arch.name == "Raketar" and isinstance(config, RaketarConfig)
    assert (config.vocab, config.width, config.eps, config.residual_mult, config.side_dim, config.loop) == (300, 48, 1e-5, 0.7, 10, (1, 3, 3))
    assert config.to_dict() == DOC_A and RaketarConfig.from_dict(config.to_dict()) == config
    assert all(l.block.kind == "parallel_pre_norm" and l.block.params["scale"] == 0.7 and l.side.kind == "token_side" for l in plan.layers)
    assert [l.mixer.kind for l in plan.layers] == ["matrix_memory", "differential_attention", "matrix_memory", "differential_attention"]
    assert [l.side.params["first_column"] for l in plan.layers] == [0, 10, 20, 30] and plan.layers[2].feed_forward is None
    assert [(e.layer, e.add_first, e.add_vector) for e in plan.order] == [
        (0, False, None), (1, False, ("loop.step", 0)), (2, False, None), (1, True, ("loop.step", 1)), (2, False, None),
        (1, True, ("loop.step", 2)), (2, False, None), (3, False, None)]
    a, f = plan.layers[1].mixer.params, plan.layers[0].feed_forward.params
    assert a["position"].params == {"theta": 100.0, "rotary_dim": 8, "interleaved": True, "factor": 2.0} and a["mask"] == {"kind": "causal"}
    assert (f["experts"], f["top"], f["scores"], f["weigh"]) == (6, 2, "sigmoid", "input") and plan.layers[3].feed_forward.params["shared"] is None
    shapes = {s.name: s.shape for s in helpers.tensor_specs_of(DOC_A)}
    assert shapes["loop.step"] == (3, 48) and shapes["side.embed"] == (300, 40) and shapes["head"] == (300, 48)
    assert shapes["l1.mix.q"] == (96, 48) and shapes["l1.mix.k"] == (48, 48) and shapes["l1.mix.v"] == (16, 48) and shapes["l1.mix.o"] == (48, 32)
    assert shapes["l1.mix.g"] == (32, 48) and shapes["l1.mix.lk2"] == (12,) and shapes["l0.mix.norm"] == (32,) and shapes["l0.mix.f.b"] == (4,)
    assert shapes["l0.side.gate"] == (10, 48) and shapes["l0.side.proj"] == (48, 10) and shapes["l0.mlp.e5.gate"] == (16, 48)
    assert not any(n.startswith(("l2.mlp", "l0.norm2")) for n in shapes)
    names_d = {s.name for s in helpers.tensor_specs_of(DOC_D)}
    assert not any("side" in n for n in names_d) and "loop.step" in names_d
    assert "loop.step" not in {s.name for s in helpers.tensor_specs_of(DOC_B)} and "loop.step" in plan_from_document(DOC_B)[2].unused_tensors
    empty = copy.deepcopy(DOC_D)
    empty["loop"] = {"start": 1, "stop": 1, "times": 3}
    assert [(e.layer, e.add_vector) for e in plan_from_document(empty)[2].order] == [(0, None), (1, None)]


def test_configuration_refusals():
    def changed(path, value):
        doc = copy.deepcopy(DOC_A)
        at = doc
        for key in path[:-1]:
            at = at[key]
        if value is None:
            del at[path[-1]]
        else:
            at[path[-1]] = value
        return doc

    m0, m1 = ("layers", 0, "mixer"), ("layers", 1, "mixer")
    for path in [("norm",), (*m1, "kv_heads"), (*m1, "diff"), (*m1, "rot", "base"), (*m1, "rot", "scaling", "factor"), (*m0, "gate_cap"),
                 ("layers", 0, "mlp", "expert", "ff"), ("layers", 0, "mlp", "shared", "ff"), ("loop", "times"), ("token_side", "dim")]:
        with pytest.raises(ConfigMissing):
            RaketarConfig.from_dict(changed(path, None))
    for path, value in [
        (("layers", 0, "type"), "serial"), ((*m1, "kv_heads"), 3), ((*m1, "rot", "dims"), 3), ((*m1, "rot", "dims"), 14),
        ((*m1, "rot", "scaling", "factor"), 0.0), ((*m0, "gate_cap"), 0.0), (("layers", 0, "mlp", "router", "top"), 7),
        (("layers", 1, "mlp", "kind"), "glu"), (("loop", "stop"), 5), (("loop", "start"), 4), (("vocab",), 0), (("layers",), []),
        (("token_side", "dim"), 0),
    ]:
        with pytest.raises(InvalidValue):
            RaketarConfig.from_dict(changed(path, value))


def test_cache_needs():
    _, _, plan = plan_from_document(DOC_A)
    needs = Model(plan, BuildEnv(dtype=torch.float32, device=torch.device("cpu"), ops=fake_kernels)).cache_needs()
    assert len(needs) == 8  # a cache of its own for every pass of a repeated layer
    assert needs[0] == (FixedState((4, 12, 8)), FixedState((4, 12)), FixedState((4,)))
    assert needs[1] == needs[3] == needs[5] == PagedKV(4, 12, None, 8, num_v_heads=2) and needs[1].value_heads == 2
    assert needs[7] == PagedKV(2, 16, None, 20, num_v_heads=1)
    from shiso_llm_b200.cache import CacheManager
    cache = CacheManager([needs[1]], 4, 6, 2, torch.float32, "cpu")
    assert cache.view(0).k.shape == (6, 4, 4, 12) and cache.view(0).v.shape == (6, 4, 2, 8)
    assert CacheManager.costs([needs[1]], 4, torch.float32)[0] == 4 * (4 * 12 + 2 * 8) * 4


# --------------------------------------------------------------------------- the whole model, every cut


@pytest.mark.parametrize("backend", BACKENDS)
@pytest.mark.parametrize("name", ["A", "B", "C", "D"])
def test_every_cut_matches_the_plain_implementation(tmp_path, backend, name):
    doc, seed = DOCS[name]
    tensors = make_folder(tmp_path, doc, seed)
    lengths = [70, 40, 7, 33, 1]
    requests = {f"r{i}": helpers.random_prompt(n, doc["vocab"], 20 + i) for i, n in enumerate(lengths)}
    reference = {rid: reference_logits(doc, tensors, toks) for rid, toks in requests.items()}
    for dtype in dtypes(backend):
        engine = helpers.make_engine(tmp_path, dtype, page_size=4, kv_cache_tokens=192, ctx=128,
                                     max_num_batched_tokens=128, **backend_args(backend))
        free = list(engine.cache.free_pages())
        steps, expect = [], []
        for rid, toks in requests.items():
            steps += helpers.whole(f"w-{rid}", toks)
            expect.append((f"w-{rid}", rid))
        steps += helpers.tail_one_by_one("t-r0", requests["r0"], 40)
        steps += helpers.portions("p-r0", requests["r0"], [13, 2, 7, 1, 3])
        steps += helpers.portions("p-r1", requests["r1"], [5, 4, 1])
        steps += helpers.portions("p-r3", requests["r3"], [2])
        expect += [("t-r0", "r0"), ("p-r0", "r0"), ("p-r1", "r1"), ("p-r3", "r3")]
        steps += replay.mixed_trace({f"m-{k}": v for k, v in requests.items()}, 3, 192)
        expect += [(f"m-{rid}", rid) for rid in requests]
        steps += replay.mixed_trace({f"n-{k}": v for k, v in reversed(list(requests.items()))}, 8, 192, tail=3)
        expect += [(f"n-{rid}", rid) for rid in requests]
        rows = helpers.run_steps(engine, steps)  # (checks the cache's books after every step)
        for trace_id, rid in expect:
            got = replay.stack_rows(rows, trace_id, len(requests[rid]))
            check_rows(got, reference[rid], dtype, f"{name} {dtype} {trace_id}")
        assert sorted(engine.cache.free_pages()) == sorted(free) and engine.cache.slots.free_slots == 4


@pytest.mark.parametrize("backend", BACKENDS)
@pytest.mark.parametrize("name", ["A", "B", "C", "D"])
def test_the_residual_stream_after_every_layer_run(tmp_path, backend, name):
    """The stream after every run of a layer (a repeated layer counts each time), side input included and
    before what the next pass adds: an addition at the wrong place, or twice, shows here."""
    doc, seed = DOCS[name]
    tensors = make_folder(tmp_path, doc, seed)
    toks = helpers.random_prompt(19, doc["vocab"], 9)
    want = []
    plain.plain_logits(doc, dict(tensors), toks, hook=lambda run, x: want.append(x.clone()))
    from shiso_llm_b200.engine import StepEntry
    from shiso_llm_b200.parts.model import stream_value
    engine = helpers.make_engine(tmp_path, "float32", page_size=4, kv_cache_tokens=64, ctx=64, max_num_batched_tokens=64, **backend_args(backend))
    got = {}
    engine.layer_hook = lambda pos, stream: got.__setitem__(pos, stream_value(stream).double().cpu())
    engine.step([StepEntry("a", toks, [len(toks) - 1])])
    assert sorted(got) == list(range(-1, len(want)))
    for run, x in enumerate(want):
        err = (got[run] - x).abs().max().item()
        assert err <= 2e-5 * x.abs().max().item(), f"after layer run {run}: {err:.3e}"


@pytest.mark.parametrize("backend", BACKENDS)
def test_cuts_agree_with_each_other_far_more_closely(tmp_path, backend):
    doc, seed = DOCS["C"]
    make_folder(tmp_path, doc, seed)
    toks = helpers.random_prompt(90, doc["vocab"], 77)
    for dtype in dtypes(backend):
        engine = helpers.make_engine(tmp_path, dtype, page_size=16, kv_cache_tokens=256, ctx=256, max_num_batched_tokens=256,
                                     **backend_args(backend))
        whole = replay.stack_rows(helpers.run_steps(engine, helpers.whole("a", toks)), "a", len(toks))
        single = replay.stack_rows(helpers.run_steps(engine, helpers.portions("b", toks, [1])), "b", len(toks))
        cut = replay.stack_rows(helpers.run_steps(engine, helpers.portions("c", toks, [5, 2, 31, 3])), "c", len(toks))
        for other in (single, cut):
            if dtype == "float32":
                assert (whole - other).pow(2).mean(-1).sqrt().max().item() <= 2e-5 * whole.std().item()
            else:  # (a router's close call may fall otherwise in another cut)
                assert (whole - other).abs().median().item() <= 0.1 * whole.std().item()


@pytest.mark.parametrize("backend", BACKENDS)
def test_long_decoding_with_a_request_that_joins(tmp_path, backend):
    """300 tokens one by one after a short prompt, with a second request joining half-way; the trace
    runs twice in one engine, so every page and slot is used again."""
    doc, seed = DOCS["A"]
    tensors = make_folder(tmp_path, doc, seed)
    a = helpers.random_prompt(330, doc["vocab"], 5)
    b = helpers.random_prompt(110, doc["vocab"], 6)
    reference = {"a": reference_logits(doc, tensors, a), "b": reference_logits(doc, tensors, b)}
    steps = [([("a", a[:30], list(range(30)))], [])]
    for i in range(30, 330):
        entries = [("a", [a[i]], [0])]
        j = i - 130  # b: a prompt of 20 at a's position 130, then one token a step
        if j == 0:
            entries.insert(0, ("b", b[:20], list(range(20))))
        elif 0 < j <= 90:
            entries.append(("b", [b[19 + j]], [0]))
        steps.append((entries, [r for r, n in (("a", 329), ("b", 220)) if i == n]))
    for dtype in dtypes(backend):
        engine = helpers.make_engine(tmp_path, dtype, page_size=8, kv_cache_tokens=456, ctx=336, max_num_batched_tokens=64,
                                     **backend_args(backend))
        free = list(engine.cache.free_pages())
        if backend != "cpu":
            helpers.run_steps(engine, steps[:150])
            engine.finish("a"), engine.finish("b")
        rows = helpers.run_steps(engine, steps)
        check_rows(replay.stack_rows(rows, "a", 330), reference["a"], dtype, f"long decoding {dtype}")
        check_rows(replay.stack_rows(rows, "b", 110), reference["b"], dtype, f"the request that joined {dtype}")
        assert sorted(engine.cache.free_pages()) == sorted(free) and engine.cache.slots.free_slots == 4


# heads of real widths: both tensor-memory and TMA kernels (maps of 64 and 32, values of 128 and 64), the tiled one
# (48, 96), states in chunks on the tensor cores (64 x 48, 128 x 128) and walked (72 x 20)
DOC_WIDE = {
    "architecture": "Raketar", "vocab": 400, "width": 128, "norm": {"eps": 1e-6}, "residual_mult": 0.6, "token_side": {"dim": 16},
    "loop": {"start": 1, "stop": 3, "times": 2},
    "layers": [
        layer(attention(4, 2, 64, 128, 0.11, 0.4, 64, 10000.0, 4.0), moe(6, 2, 64, 80)),
        layer(memory(2, 64, 48, 12.0), dense(160)),
        layer(attention(8, 2, 32, 64, 0.16, 0.3, 16), None),
        layer(memory(1, 128, 128, 15.0), moe(4, 1, 32)),
        layer(attention(2, 1, 48, 96, 0.14, 0.7, 48), dense(96)),
        layer(memory(2, 72, 20, 8.0), None),
    ],
}


@pytest.mark.gpu
def test_long_portions_and_wide_heads(tmp_path):
    """A 700-token request: whole, in long and short portions, with a second request in the batch, and
    the last tokens decoded alone and beside others."""
    tensors = make_folder(tmp_path, DOC_WIDE, 9, std=0.08)
    a = helpers.random_prompt(700, DOC_WIDE["vocab"], 1)
    b = helpers.random_prompt(150, DOC_WIDE["vocab"], 2)
    reference = {"a": reference_logits(DOC_WIDE, tensors, a), "b": reference_logits(DOC_WIDE, tensors, b)}
    for dtype in ("bfloat16", "float32"):
        engine = helpers.make_engine(tmp_path, dtype, page_size=16, kv_cache_tokens=4096, ctx=2048, max_num_batched_tokens=1024)
        rows = helpers.run_steps(engine, helpers.whole("w", a))
        check_rows(replay.stack_rows(rows, "w", 700), reference["a"], dtype, f"one long portion {dtype}")
        rows = helpers.run_steps(engine, helpers.portions("p", a, [300, 100, 260, 1, 39]))
        check_rows(replay.stack_rows(rows, "p", 700), reference["a"], dtype, f"long and short portions {dtype}")
        rows = helpers.run_steps(engine, helpers.tail_one_by_one("t", a, 24))
        check_rows(replay.stack_rows(rows, "t", 700), reference["a"], dtype, f"decoded at a long context {dtype}")
        steps = [([("a", a[:400], list(range(400))), ("b", b[:5], list(range(5)))], []),
                 ([("b", b[5:6], [0]), ("a", a[400:650], list(range(250)))], []),
                 ([("b", b[6:140], list(range(134)))], [])]
        steps += [([("a", [a[650 + i]], [0]), ("b", [b[140 + i]], [0])], []) for i in range(10)]
        steps.append(([("a", a[660:], list(range(40)))], ["a", "b"]))
        rows = helpers.run_steps(engine, steps)
        check_rows(replay.stack_rows(rows, "a", 700), reference["a"], dtype, f"a long portion in a batch {dtype}")
        check_rows(replay.stack_rows(rows, "b", 150), reference["b"], dtype, f"its neighbour {dtype}")


@pytest.mark.gpu
@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_replay_through_the_trace_runner(tmp_path, dtype):
    """``bin/trace_run`` in a process of its own over a pool that holds barely the live requests:
    whole, last tokens one by one, changing portions and a mixed trace, against the plain logits."""
    doc, seed = DOCS["C"]
    model_dir = tmp_path / "model"
    tensors = make_folder(model_dir, doc, seed)
    lengths = [70, 100, 40, 7, 33, 1]
    requests = {f"r{i}": helpers.random_prompt(n, doc["vocab"], 60 + i) for i, n in enumerate(lengths)}
    steps, expect = [], []
    for rid, toks in requests.items():
        steps += helpers.whole(f"w-{rid}", toks)
        expect.append((f"w-{rid}", rid))
    steps += helpers.tail_one_by_one("t-r1", requests["r1"], 32)
    steps += helpers.portions("p-r1", requests["r1"], [13, 2, 7, 64, 3])
    steps += helpers.portions("p-r0", requests["r0"], [2, 3, 1, 2, 5, 1, 1, 17])
    expect += [("t-r1", "r1"), ("p-r1", "r1"), ("p-r0", "r0")]
    steps += replay.mixed_trace({f"m-{k}": v for k, v in requests.items()}, 5, 320)
    expect += [(f"m-{rid}", rid) for rid in requests]
    rows = replay.run_trace_run(model_dir, dtype, steps, 320, tmp_path / "out", doc["vocab"])
    for trace_id, rid in expect:
        got = replay.stack_rows(rows, trace_id, len(requests[rid]))
        check_rows(got, reference_logits(doc, tensors, requests[rid]), dtype, f"{dtype} {trace_id}")


@pytest.mark.parametrize("backend", BACKENDS)
def test_greedy_generation_through_the_scheduler(tmp_path, backend):
    """Tokens picked on the device are fed on without the host seeing them: the side input has to follow."""
    doc, seed = DOCS["A"]
    tensors = make_folder(tmp_path, doc, seed)
    prompts = [helpers.random_prompt(n, doc["vocab"], 40 + n) for n in (19, 3, 30)]
    new = 12

    def plain_greedy(prompt):
        seq = list(prompt)
        for _ in range(new):
            seq.append(int(plain.plain_logits(doc, dict(tensors), seq)[-1].argmax()))
        return seq[len(prompt):]

    want = [plain_greedy(p) for p in prompts]
    args = backend_args(backend)
    llm = LLM(str(tmp_path), dtype="float32", ctx=64, page_size=4, max_num_seqs=2, max_num_batched_tokens=16, prefill_chunk=7,
              ops=args["ops"], device=args["device"])
    outs = llm.generate(prompts, SamplingParams(temperature=0.0, max_new_tokens=new, ignore_eos=True))
    assert [o.token_ids for o in outs] == want
    llm.engine.cache.check()
    assert llm.engine.cache.slots.free_slots == 2


# --------------------------------------------------------------------------- mechanisms alone


def plan_layer(mixer_doc, width, mlp=None, eps=1e-5, mult=1.0, side=None, vocab=8):
    """The layer's specs as the plan builder makes them, with tensors named ``l0.*``."""
    doc = {"architecture": "Raketar", "vocab": vocab, "width": width, "norm": {"eps": eps}, "residual_mult": mult, "layers": [layer(mixer_doc, mlp)]}
    if side is not None:
        doc["token_side"] = {"dim": side}
    return plan_from_document(doc)[2].layers[0]


MIXER_DOCS = {
    "attention": attention(6, 3, 10, 7, 0.4, 0.3, 6, 50.0, 3.0), "attention-one-head": attention(1, 1, 8, 16, 0.5, 0.0, 8),
    "attention-no-rotation": attention(4, 1, 5, 5, 0.5, 0.9, 0), "memory": memory(3, 9, 5, 6.0), "memory-wide": memory(2, 40, 70, 1.5),
    "memory-one": memory(1, 1, 1, 20.0),
}


@pytest.mark.parametrize("backend", BACKENDS)
@pytest.mark.parametrize("name", list(MIXER_DOCS))
def test_each_mixer_alone_in_steps_and_batches(backend, name):
    doc = MIXER_DOCS[name]
    fn = plain.mlstm if "gate_cap" in doc else plain.differential_attention
    for dtype in mixer_dtypes(backend):
        if dtype == torch.bfloat16 and name in ("memory-one", "attention-one-head"):
            continue  # (a head's output may be small before its norm: bfloat16 is compared kernel by kernel)
        env = build_env(backend, dtype)
        mixer = MIXERS.build(plan_layer(doc, 40).mixer, env)
        w = bind(mixer, env, 11)
        g = torch.Generator().manual_seed(1)
        a, b = torch.randn(37, 40, generator=g).to(dtype), torch.randn(9, 40, generator=g).to(dtype)
        want_a, want_b = (fn(w, "l0.mix", doc, x.double(), 1e-5) for x in (a, b))
        in_steps_and_batches(mixer, env, dtype, a, b, want_a, want_b, name, 10.0 if dtype == torch.bfloat16 else 4.0)


@pytest.mark.parametrize("backend", BACKENDS)
@pytest.mark.parametrize("planted_map", [0, 1])
def test_a_planted_key_decides_its_map(backend, planted_map):
    """One key is made to stand out for one map only (that map's key rows are its query rows, the other's
    are zero): first positions, far back, on either side of page borders, right before the asking row,
    which ends a portion or is decoded.  A map that reads the other's queries or keys, a wrong value
    head, or a key that is not seen differs."""
    env = build_env(backend, torch.float32)
    doc = attention(4, 2, 8, 12, 1.5, 0.4, 4, 5000.0, 2.0)
    mixer = MIXERS.build(plan_layer(doc, 32).mixer, env)
    from shiso_llm_b200.weights import random_tensors
    from shiso_llm_b200.weights.loader import target_dtype
    specs = {s.name: s for s in mixer.tensor_specs()}
    stored = random_tensors(list(specs.values()), 31, 0.3, "bfloat16", 0.1)
    q = stored["l0.mix.q"].view(2, 2, 2, 8, 32)  # key head, query head of the group, map
    q[:, :, 1 - planted_map] = 0.0
    stored["l0.mix.k"] = q[:, 0].reshape(32, 32).contiguous()
    mixer.bind({k: v.to(env.device, target_dtype(specs[k], v.dtype, env.dtype)) for k, v in stored.items()})
    w = {k: v.double() for k, v in stored.items()}
    T = 150
    g = torch.Generator().manual_seed(3)
    base, probe = torch.randn(T, 32, generator=g) * 0.1, torch.randn(32, generator=g)
    quiet = base.clone()
    quiet[T - 1] = probe * 3.0
    without = plain.differential_attention(w, "l0.mix", doc, quiet.double(), 1e-5)[T - 1]
    for place in (0, 1, 3, 4, 31, 32, 70, 127, 128, 147, 148):
        h = quiet.clone()
        h[place] = probe * 30.0
        want = plain.differential_attention(w, "l0.mix", doc, h.double(), 1e-5)
        assert (want[T - 1] - without).abs().max().item() > 0.02 * without.abs().max().item()
        for tail in (0, 9):
            feeder = Feeder(mixer, env, pages=64)
            got = [feeder.step([("a", h[: T - tail - 7])])["a"], feeder.step([("a", h[T - tail - 7 : T - tail])])["a"]]
            for t in range(T - tail, T):
                got.append(feeder.step([("a", h[t : t + 1])])["a"])
            close(torch.cat(got), want, torch.float32, f"map {planted_map}: planted at {place}, {tail} decoded", 8.0)


@pytest.mark.parametrize("backend", BACKENDS)
def test_the_second_maps_weight(backend):
    """Vectors so large that the two exponentials matter: the weight is their difference plus the constant,
    and the factor behind the norm is one minus the constant."""
    env = build_env(backend, torch.float32)
    for diff, scales in ((0.7, (3.0, 3.0)), (0.0, (8.0, 0.0)), (0.25, (0.0, 6.0))):
        doc = attention(2, 1, 9, 6, 0.5, diff, 4)
        mixer = MIXERS.build(plan_layer(doc, 24).mixer, env)
        w = bind(mixer, env, 5, 0.3, {f"l0.mix.l{x}{i}": (lambda t, s=scales[i - 1]: t * s) for x in "qk" for i in (1, 2)})
        assert abs(mixer.second - float(plain.map_weight(w, "l0.mix", diff))) < 1e-12
        h = torch.randn(21, 24, generator=torch.Generator().manual_seed(2))
        close(Feeder(mixer, env).step([("a", h)])["a"], plain.differential_attention(w, "l0.mix", doc, h.double(), 1e-5), torch.float32, f"weight {diff}", 4.0)


@pytest.mark.parametrize("backend", BACKENDS)
def test_a_lost_state_or_running_maximum_shows(backend):
    """Forget gates of nearly one and a first token whose write is huge: what it wrote, and the maximum it
    set, are felt for the whole sequence, so a state, a normaliser or a maximum dropped (or taken
    twice) at a portion's start changes every row behind it; portions on either side of 64 rows."""
    env = build_env(backend, torch.float32)
    doc = memory(3, 12, 10, 9.0)
    mixer = MIXERS.build(plan_layer(doc, 24).mixer, env)
    w = bind(mixer, env, 3, 0.4, {"l0.mix.f.b": lambda t: t * 0.0 + 8.0, "l0.mix.i": lambda t: t * 0.2, "l0.mix.f": lambda t: t * 0.1})
    g = torch.Generator().manual_seed(4)
    h = torch.randn(150, 24, generator=g) * 0.2
    h[0] *= 40.0
    want = plain.mlstm(w, "l0.mix", doc, h.double(), 1e-5)
    lost = plain.mlstm(w, "l0.mix", doc, h[1:].double(), 1e-5)
    assert (want[100] - lost[99]).abs().max().item() > 0.05 * want[100].abs().max().item()
    for sizes in ([150], [1], [2], [1, 2, 3], [63, 64, 65, 1], [16, 1, 15, 17], [3, 128]):
        feeder, got, at, i = Feeder(mixer, env), [], 0, 0
        while at < 150:
            n = min(sizes[i % len(sizes)], 150 - at)
            got.append(feeder.step([("a", h[at : at + n])])["a"])
            at, i = at + n, i + 1
        close(torch.cat(got), want, torch.float32, f"portions of {sizes}", 20.0)


@pytest.mark.parametrize("backend", BACKENDS)
@pytest.mark.parametrize("case", ["small-input-gates", "large-input-gates", "sudden"])
def test_the_running_maximum_and_the_denominators_floor(backend, case):
    """Input gates far below zero: the maximum is held up by its start at zero and the denominator by its
    floor ``exp(-m)`` (started at minus infinity, or without the floor, outputs blow up before the norm and
    eps is not felt).  Far above: exponentials would overflow without the maximum.  A sudden large gate
    takes the old state's share to zero in one step.  Compared before the head's norm, which would hide a scale."""
    env = build_env(backend, torch.float32)
    ops, T, H, D, V = env.ops, 70, 2, 8, 6
    from types import SimpleNamespace
    g = torch.Generator().manual_seed(7)
    z = torch.randn(T, 2 * H, generator=g)
    z[:, :H] += {"small-input-gates": -40.0, "large-input-gates": 90.0, "sudden": -3.0}[case]
    if case == "sudden":
        z[33, :H] = 60.0
    q, k = (torch.randn(T, H * D, generator=g) for _ in range(2))
    v, gate = torch.randn(T, H * V, generator=g), torch.randn(T, H * V, generator=g)
    cap = 50.0
    i, f = plain.capped(z[:, :H].double(), cap), plain.log_sigmoid(plain.capped(z[:, H:].double(), cap))
    want = torch.stack([plain.memory(q.view(T, H, D)[:, a].double() * D**-0.5, k.view(T, H, D)[:, a].double(), v.view(T, H, V)[:, a].double(), i[:, a], f[:, a])
                        for a in range(H)], dim=1)
    step = SimpleNamespace(num_seqs=1, q_start=torch.tensor([0, T], dtype=torch.int32, device=env.device),
                           state_slots=torch.zeros(1, dtype=torch.int32, device=env.device))
    top, state, n = (torch.zeros(1, *s, device=env.device) for s in ((H,), (H, D, V), (H, D)))
    keep, add, floor = ops.memory_gates(z.to(env.device), cap, top, step)
    raw, read = ops.memory_recurrence(*(x.to(env.device) for x in (q, k, v)), keep, add, state, n, step, H, D, V)
    r = raw.double().cpu().view(T, H, V) * D**-0.5
    o = r / (torch.maximum((read.double().cpu() * D**-0.5).abs(), floor.double().cpu()) + plain.DENOMINATOR_EPS)[..., None]
    scale = want.abs().amax((1, 2), keepdim=True)  # (a quotient whose n . q is nearly zero keeps fewer digits)
    assert ((o - want).abs() <= 1e-3 * scale + 1e-30).all() and ((o - want).abs() / scale).median() <= 1e-5, ((o - want).abs() / scale).max()
    out = torch.empty(T, H * V, device=env.device)
    ops.memory_output(raw, read, floor, gate.to(env.device), torch.ones(H * V, device=env.device), H, V, D**-0.5, plain.DENOMINATOR_EPS, 1e-5, out)
    close(out.double().cpu(), (plain.unit_rms(want, 1e-5).reshape(T, -1) * torch.sigmoid(gate.double())), torch.float32, case, 10.0)


def test_a_gates_cap_matters_in_the_oracle():
    """The cap squeezes both log gates: doubling it changes outputs, so a reader that ignored it would show."""
    g = torch.Generator().manual_seed(1)
    from shiso_llm_b200.weights import random_tensors
    env = BuildEnv(dtype=torch.float32, device=torch.device("cpu"), ops=fake_kernels)
    mixer = MIXERS.build(plan_layer(memory(2, 6, 5, 2.0), 24).mixer, env)
    w = {k: v.double() for k, v in random_tensors(mixer.tensor_specs(), 3, 0.5, "bfloat16", 0.1).items()}
    h = torch.randn(20, 24, generator=g).double()
    a, b = (plain.mlstm(w, "l0.mix", memory(2, 6, 5, cap), h, 1e-5) for cap in (2.0, 4.0))
    assert (a - b).abs().max().item() > 0.02 * a.abs().max().item()


MLPS = {"shared": moe(7, 3, 14, 20), "plain": moe(7, 2, 9), "all-chosen": moe(4, 4, 8, 8), "one": moe(1, 1, 12, 6), "first-only": moe(9, 1, 5), "dense": dense(22)}


@pytest.mark.parametrize("backend", BACKENDS)
@pytest.mark.parametrize("name", list(MLPS))
def test_feed_forwards_alone(backend, name):
    mlp = MLPS[name]
    for dtype in mixer_dtypes(backend):
        env = build_env(backend, dtype)
        part = FEED_FORWARDS.build(plan_layer(memory(1, 4, 4, 1.0), 36, mlp).feed_forward, env)
        w = bind(part, env, 17, 0.3, {"l0.mlp.router": lambda t: t * 3.0} if mlp["kind"] == "moe" else None)
        g = torch.Generator().manual_seed(2)
        for rows in (1, 5, 70):
            h = (torch.randn(rows, 36, generator=g) * 1.5).to(dtype)
            margins = []
            want = plain.feed_forward(w, "l0.mlp", mlp, h.double(), margins)
            y = part.forward(h.to(env.device), None)
            y = (y.materialize() if hasattr(y, "materialize") else y).double().cpu()
            sure = torch.ones(rows, dtype=torch.bool) if dtype == torch.float32 or not margins else margins[0] > CLOSE_CALL
            assert torch.isfinite(y).all()
            if sure.any():
                close(y[sure], want[sure], dtype, f"{name} feed-forward, {rows} rows {dtype}", 4.0)


@pytest.mark.parametrize("backend", BACKENDS)
def test_the_weight_goes_into_the_expert(backend):
    """Weights far from one: behind the activation they would scale the output, in front of it they pass a
    silu and a product of two; the two differ by far more than rounding.  Identity experts are linear."""
    env = build_env(backend, torch.float32)
    g = torch.Generator().manual_seed(3)
    x = torch.randn(5, 16, generator=g)
    gate_up, down = torch.randn(3, 24, 16, generator=g) * 0.3, torch.randn(3, 16, 12, generator=g) * 0.3
    ids = torch.tensor([[0, 1], [2, 0], [1, 2], [3, 0], [0, 3]], dtype=torch.int32)
    weights = torch.rand(5, 2, generator=g) * 0.5 + 0.05
    want = torch.zeros(5, 16, dtype=torch.float64)
    for t in range(5):
        for j in range(2):
            e, into = int(ids[t, j]), weights[t, j].double() * x[t].double()
            if e < 3:
                a, b = (gate_up[e].double() @ into).split(12)
                into = down[e].double() @ (plain.silu(a) * b)
            want[t] += into
    args = [v.to(env.device) for v in (x, ids, weights, gate_up, down)]
    got = env.ops.routed_experts(*args, identity=1, weigh_input=True)
    close(got.double().cpu(), want, torch.float32, "weights on the input", 2.0)
    other = env.ops.routed_experts(*args, identity=1)
    assert (other.double().cpu() - want).abs().max().item() > 0.05 * want.abs().max().item()


@pytest.mark.parametrize("backend", BACKENDS)
def test_the_token_side_input(backend):
    """The layer's own slice of the table, rows picked by token id - or, where the host has not seen the
    token, by what a sampler left on the device - under the norms that take it and on its own."""
    from types import SimpleNamespace
    for dtype in mixer_dtypes(backend):
        env = build_env(backend, dtype)
        # (a single column's row is the normed projection times a sign: bfloat16 may turn it)
        for dim, i in ((6, 0), (6, 1), (6, 2)) + (((1, 1),) if dtype == torch.float32 else ()):
            doc = {"architecture": "Raketar", "vocab": 31, "width": 40, "norm": {"eps": 1e-5}, "residual_mult": 0.3, "token_side": {"dim": dim},
                   "layers": [layer(memory(1, 4, 4, 1.0), None)] * 3}
            part = SIDES.build(plan_from_document(doc)[2].layers[i].side, env)
            w = bind(part, env, 5 + i, 0.3)
            assert part.table.shape == (31, 3 * dim)
            g = torch.Generator().manual_seed(i)
            x = torch.randn(7, 40, generator=g).to(env.device, dtype)
            tokens = [3, 30, 0, 7, 7, 12, 1]
            step = SimpleNamespace(token_ids=torch.tensor([3, 30, 0, 9, 7, 9, 1], dtype=torch.int32, device=env.device),
                                   feed_index=torch.tensor([-1, -1, -1, 2, -1, 0, -1], dtype=torch.int32, device=env.device),
                                   fed_tokens=torch.tensor([12, 5, 7], dtype=torch.int32, device=env.device))
            waiting = part.forward(x, step, 0.3)
            assert isinstance(waiting, NormedOutput)
            want = 0.3 * plain.token_side(w, i, dim, tokens, x.double().cpu(), 1e-5)
            close(waiting.materialize().double().cpu(), want, dtype, f"side input of layer {i} {dtype}", 4.0)


@pytest.mark.parametrize("backend", BACKENDS)
def test_the_normed_output_under_every_reader(backend):
    """Added to the stream under the next norm, with a row list (before the head), on its own, and under a
    norm that knows no such outputs; residual sums in float32."""
    for dtype in mixer_dtypes(backend):
        env = build_env(backend, dtype)
        for width in (50, 64, 2056):
            norm = NORMS.build(PartSpec("rmsnorm", {"tensor": "n", "size": width, "eps": 1e-5}), env)
            other = NORMS.build(PartSpec("layernorm", {"tensor": "n", "size": width, "eps": 1e-5}), env)
            w, w_other = bind(norm, env, 3), bind(other, env, 3)
            g = torch.Generator().manual_seed(6)
            x = (torch.randn(9, width, generator=g) * 3).to(env.device)
            y = (torch.randn(9, width, generator=g) * 7.0).to(env.device, dtype)
            yw = 1.0 + 0.3 * torch.randn(width, generator=g).to(env.device)
            out = NormedOutput(env.ops, y, yw, 0.4, 1e-5)
            c = [t.double().cpu() for t in (x, y, yw)]
            delta = 0.4 * plain.unit_rms(c[1], 1e-5) * c[2]
            close(out.materialize().double().cpu(), delta, torch.float32, f"normed output {width}", 2.0)
            want = plain.rms_norm(c[0] + delta, w, "n", 1e-5)
            stream = Stream(x.clone())
            stream.add(out)
            close(stream.normed(norm).double().cpu(), want, dtype, f"under a norm {width}", 2.0)
            assert (stream.residual.double().cpu() - c[0] - delta).abs().max().item() <= 1e-5 and stream.pending is None
            residual = x.clone()
            rows = torch.tensor([7, 2], dtype=torch.int32, device=env.device)
            close(norm.add_apply(residual, out, rows).double().cpu(), want[[7, 2]], dtype, "rows", 2.0)
            assert torch.equal(residual, x)
            stream = Stream(x.clone())
            stream.add(out)
            z = c[0] + delta
            z = (z - z.mean(-1, keepdim=True)) / torch.sqrt(z.var(-1, unbiased=False, keepdim=True) + 1e-5) * w_other["n"]
            close(stream.normed(other).double().cpu(), z, dtype, "under a layer norm", 2.0)


@pytest.mark.parametrize("backend", BACKENDS)
def test_outputs_added_at_once(backend):
    """``residual += scale * sum`` in float32, and the new rows in the compute type where they are wanted."""
    for dtype in mixer_dtypes(backend):
        env = build_env(backend, dtype)
        g = torch.Generator().manual_seed(8)
        for tokens, width in ((5, 50), (1, 64), (33, 132), (3, 7)):
            x = torch.randn(tokens, width, generator=g).to(env.device)
            ds = [torch.randn(tokens, width, generator=g).to(env.device, dtype) for _ in range(2)]
            for n in (1, 2):
                for wanted in (True, False):
                    stream = Stream(x.clone())
                    rows = stream.add_now(ds[:n], 0.7, env, wanted)
                    want = x.double().cpu() + 0.7 * sum(d.double().cpu() for d in ds[:n])
                    close(stream.residual.double().cpu(), want, torch.float32, f"{n} outputs")
                    assert (rows is not None) == wanted
                    if wanted:
                        assert rows.dtype == dtype
                        close(rows.double().cpu(), want, dtype, "rows")


@pytest.mark.parametrize("backend", BACKENDS)
@pytest.mark.parametrize("mult,side", [(1.0, None), (0.25, None), (1.0, 5), (-0.5, 3)])
def test_the_parallel_block(backend, mult, side):
    """One norm read by both sublayers, the factor on each sum, the side input behind them reading the stream
    itself - with and without each of them."""
    from types import SimpleNamespace
    env = build_env(backend, torch.float32)
    mix, mlp = memory(2, 6, 5, 3.0), moe(4, 2, 7, 9)
    spec = plan_layer(mix, 24, mlp, mult=mult, side=side, vocab=19)
    block = BLOCKS.build(spec.block, env, spec)
    w = bind(block, env, 13, 0.3)
    tokens = [4, 18, 0, 4, 9]
    x = torch.randn(5, 24, generator=torch.Generator().manual_seed(1))
    step = SimpleNamespace(num_seqs=1, num_tokens=5, q_start=torch.tensor([0, 5], dtype=torch.int32, device=env.device), all_decode=False,
                           state_slots=torch.zeros(1, dtype=torch.int32, device=env.device),
                           token_ids=torch.tensor(tokens, dtype=torch.int32, device=env.device))
    cache = tuple(SimpleNamespace(state=torch.zeros(1, *need.shape, device=env.device)) for need in block.mixer_part().cache_spec())
    stream = Stream(x.to(env.device).clone())
    block.forward(stream, step, cache)
    from shiso_llm_b200.parts.model import stream_value
    x64 = x.double()
    h = plain.rms_norm(x64, w, "l0.norm1", 1e-5)
    want = x64 + mult * (plain.mlstm(w, "l0.mix", mix, h, 1e-5) + plain.mixture(w, "l0.mlp", mlp, h))
    if side is not None:
        want = want + mult * plain.token_side(w, 0, side, tokens, want, 1e-5)
    close(stream_value(stream).double().cpu(), want, torch.float32, f"block {mult} {side}", 4.0)
