"""The Nodepel design in the engine, on the CPU with the plain stand-in kernels and on the GPU
with the CUDA kernels (``-m gpu``): same bodies.

Everything is compared with ``plain_nodepel`` (float64, whole sequences, one function per
mechanism).  The configurations are made here; they differ from each other in every size and in
which options they have: a looped stretch that starts at the first layer, behind it, covers every
layer, runs once, or is absent; windows of 1, narrower and wider than a page; a rotation over the
whole head, part of it, or none; values of another width than the keys; one key/value head or as
many as query heads, on either side; convolutions of one tap and more; every expert chosen, one
expert, a shared expert or none; layers without feed-forward; sizes that no vector width divides.
"""

import copy

import pytest
import torch

import fake_kernels
import helpers
import plain_nodepel as plain
import replay
from shiso_llm_b200 import LLM, SamplingParams
from shiso_llm_b200.config import ConfigMissing, InvalidValue, NodepelConfig, plan_from_document
from shiso_llm_b200.parts import FEED_FORWARDS, MIXERS, NORMS, BuildEnv, FixedState, Model, NormedPair, PagedKV, PartSpec, Stream
from shiso_llm_b200.weights import write_model_folder
from test_zetavik import BACKENDS, Feeder, Reference, backend_args, bind, build_env, close, dtypes, in_steps_and_batches, mixer_dtypes


def left(heads, kv_heads, dim, vdim, scale, size, dims, base=100.0):
    return {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "scale": scale, "mask": {"size": size},
            "rot": {"dims": dims, "base": base}}


def right(heads, kv_heads, dim, vdim, conv):
    return {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "conv": conv}


def moe(experts, top, ff, shared=None):
    doc = {"kind": "moe", "expert": {"ff": ff}, "router": {"experts": experts, "top": top}}
    if shared is not None:
        doc["shared"] = {"ff": shared}
    return doc


def layer(left_doc, right_doc, mlp):
    return {"type": "parallel", "mixer": {"left": left_doc, "right": right_doc}, "mlp": mlp}


# a stretch of two layers behind the first, three passes; a layer without feed-forward, a window of one position
DOC_A = {
    "architecture": "Nodepel", "vocab": 300, "width": 48, "norm": {"eps": 1e-5}, "embedding": {"scale": 2.0},
    "loop": {"start": 1, "stop": 3, "times": 3},
    "layers": [
        layer(left(4, 2, 12, 8, 0.3, 11, 12), right(4, 2, 12, 10, 3), moe(6, 2, 16, 24)),
        layer(left(2, 2, 8, 16, 0.5, 1, 4), right(2, 1, 8, 16, 4), moe(5, 3, 10)),
        layer(left(6, 1, 16, 16, 0.25, 30, 16), right(3, 3, 16, 8, 2), None),
        layer(left(3, 3, 10, 6, 0.4, 5, 0), right(6, 2, 6, 4, 1), moe(4, 4, 12, 8)),
    ],
}

# no stretch, no embedding scale; heads of one; one expert
DOC_B = {
    "architecture": "Nodepel", "vocab": 211, "width": 64, "norm": {"eps": 1e-6},
    "layers": [
        layer(left(1, 1, 20, 24, 0.2, 64, 20, 10000.0), right(1, 1, 20, 36, 4), moe(1, 1, 24, 16)),
        layer(left(5, 5, 16, 8, 0.3, 200, 8), right(4, 4, 40, 16, 2), None),
        layer(left(4, 1, 32, 32, 0.2, 17, 32), right(8, 4, 16, 8, 5), moe(8, 1, 40, 32)),
    ],
}

# every layer inside the stretch, from the first on; sizes that no vector width divides
DOC_C = {
    "architecture": "Nodepel", "vocab": 333, "width": 50, "norm": {"eps": 1e-5}, "embedding": {"scale": 0.5},
    "loop": {"start": 0, "stop": 2, "times": 2},
    "layers": [
        layer(left(3, 1, 6, 5, 0.5, 13, 2, 7.0), right(3, 1, 7, 5, 3), moe(7, 2, 6, 14)),
        layer(left(6, 3, 10, 7, 0.35, 32, 10), right(5, 5, 33, 3, 8), moe(3, 2, 9)),
    ],
}

# a stretch that runs once, over the last layer, which has no feed-forward (the final norm closes the mixer)
DOC_D = {
    "architecture": "Nodepel", "vocab": 128, "width": 32, "norm": {"eps": 1e-6}, "embedding": {"scale": 3.5},
    "loop": {"start": 1, "stop": 2, "times": 1},
    "layers": [
        layer(left(2, 1, 8, 8, 0.3, 9, 8), right(2, 2, 8, 8, 4), moe(4, 2, 16, 8)),
        layer(left(2, 1, 8, 8, 0.3, 40, 6), right(4, 1, 4, 12, 2), None),
    ],
}

DOCS = {"A": (DOC_A, 3), "B": (DOC_B, 4), "C": (DOC_C, 5), "D": (DOC_D, 6)}


def make_folder(path, doc, seed, std=0.15):
    """Random weights, with router biases that are far apart: the choice of experts then differs from
    token to token but seldom hangs on what bfloat16 rounds away."""
    tensors = helpers.make_tensors(doc, seed, std=std)
    for name in tensors:
        if name.endswith(".router.b"):
            tensors[name] = (tensors[name].float() * 60.0).to(torch.bfloat16)
    write_model_folder(str(path), doc, tensors)
    return tensors


CLOSE_CALL = 0.05  # of a logit of the router


def check_rows(got, ref, dtype, what):
    """Per-row error against the plain logits, relative to their spread.  float32: below 1e-4 in every
    row.  bfloat16: the plain implementation with its activations rounded where the engine rounds them
    is off by up to 0.1 in a row of these small models, where a branch's output is small before its norm
    (a first token whose key and query are nearly orthogonal), and by more behind a router's close
    call; so no row without one may be off by a quarter, at most one in twenty (or one) by more
    than 0.1, and a row with a close call in it or before it by more than twice the spread.  (A wrong
    key, state, page or expert that only bfloat16 kernels could have is looked for kernel by kernel.)"""
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
    clean = rms[~touched]
    if clean.numel():
        assert clean.max().item() <= 0.25, f"{what}: a row without a close call differs by {clean.max().item():.3e} of the spread"
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
    assert arch.name == "Nodepel" and isinstance(config, NodepelConfig)
    assert (config.vocab, config.width, config.eps, config.embedding_scale, config.loop) == (300, 48, 1e-5, 2.0, (1, 3, 3))
    assert config.to_dict() == DOC_A and NodepelConfig.from_dict(config.to_dict()) == config
    assert all(l.block.kind == "pre_norm" and l.mixer.kind == "parallel_mixer" for l in plan.layers)
    assert all(l.mixer_norm.params["offset"] == 1.0 for l in plan.layers) and plan.final_norm.params["offset"] == 1.0
    # the run order: layer 0, then layers 1 and 2 three times, then layer 3; every pass begins with the matrix and its vector
    assert [(e.layer, e.mix_first, e.add_vector, e.add_first) for e in plan.order] == [
        (0, None, None, False), (1, "loop.in", ("loop.step", 0), False), (2, None, None, False),
        (1, "loop.in", ("loop.step", 1), False), (2, None, None, False),
        (1, "loop.in", ("loop.step", 2), False), (2, None, None, False), (3, None, None, False)]
    (l, share), (r, share2) = plan.layers[0].mixer.params["branches"]
    assert (l.kind, r.kind, share, share2) == ("masked_attention", "gated_delta", 0.5, 0.5)
    assert l.params["mask"] == {"kind": "window", "size": 11} and l.params["head_norm"] == "joined" and l.params["sink"] == "l0.mix.left.sink"
    assert plan.layers[3].mixer.params["branches"][0][0].params["position"].kind == "none"
    f = plan.layers[1].feed_forward.params
    assert (f["experts"], f["top"], f["scores"], f["activation"], f["shared"]) == (5, 3, "chosen_softmax", "relu2", None)
    shapes = {s.name: s.shape for s in helpers.tensor_specs_of(DOC_A)}
    assert shapes["loop.in"] == (48, 96) and shapes["loop.step"] == (3, 48) and shapes["head"] == (300, 48)
    assert shapes["l0.mix.left.q"] == (48, 48) and shapes["l0.mix.left.k"] == (24, 48) and shapes["l0.mix.left.v"] == (16, 48)
    assert shapes["l0.mix.left.q.norm"] == (48,) and shapes["l0.mix.left.sink"] == (4,) and shapes["l0.mix.left.o"] == (48, 32)
    assert shapes["l0.mix.right.q"] == (24, 48) and shapes["l0.mix.right.v.conv"] == (40, 3) and shapes["l0.mix.right.norm"] == (10,)
    assert shapes["l0.mix.right.A_log"] == (4,) and shapes["l0.mix.right.out"] == (48,) and shapes["l0.mlp.router.b"] == (6,)
    assert shapes["l0.mlp.shared.sg"] == (1, 48) and "l0.mlp.e5.up" in shapes and "l0.mlp.e6.up" not in shapes and "l0.mlp.e0.gate" not in shapes
    assert not any(n.startswith(("l2.mlp", "l2.norm2")) for n in shapes) and "l2.norm2" in plan.unused_tensors
    # no stretch: every layer once, no matrix, no vectors
    names_b = {s.name for s in helpers.tensor_specs_of(DOC_B)}
    assert plan_from_document(DOC_B)[1].embedding_scale == 1.0 and not names_b & {"loop.in", "loop.step"}
    empty = copy.deepcopy(DOC_D)
    empty["loop"] = {"start": 1, "stop": 1, "times": 3}
    plan_e = plan_from_document(empty)[2]
    assert [(e.layer, e.mix_first) for e in plan_e.order] == [(0, None), (1, None)] and {"loop.in", "loop.step"} <= set(plan_e.unused_tensors)


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

    l0 = ("layers", 0, "mixer")
    for path in [("norm",), (*l0, "left", "kv_heads"), (*l0, "left", "mask"), (*l0, "left", "rot", "base"), (*l0, "right", "conv"),
                 (*l0, "right"), ("layers", 0, "mlp", "expert", "ff"), ("layers", 0, "mlp", "shared", "ff"), ("loop", "times")]:
        with pytest.raises(ConfigMissing):
            NodepelConfig.from_dict(changed(path, None))
    for path, value in [
        (("layers", 0, "type"), "serial"), ((*l0, "left", "kv_heads"), 3), ((*l0, "right", "kv_heads"), 3), ((*l0, "left", "mask", "size"), 0),
        ((*l0, "left", "rot", "dims"), 3), ((*l0, "left", "rot", "dims"), 14), ((*l0, "right", "conv"), 0), (("layers", 0, "mlp", "router", "top"), 7),
        (("layers", 0, "mlp", "kind"), "dense"), (("loop", "stop"), 5), (("loop", "start"), 4), (("vocab",), 0), (("layers",), []),
    ]:
        with pytest.raises(InvalidValue):
            NodepelConfig.from_dict(changed(path, value))


def test_cache_needs():
    _, _, plan = plan_from_document(DOC_A)
    needs = Model(plan, BuildEnv(dtype=torch.float32, device=torch.device("cpu"), ops=fake_kernels)).cache_needs()
    assert len(needs) == 8  # a cache of its own for every pass of a repeated layer
    assert needs[0] == (PagedKV(2, 12, 11, 8), FixedState((2, 88)), FixedState((4, 12, 10)))
    assert needs[1] == needs[3] == needs[5] == (PagedKV(2, 8, 1, 16), FixedState((3, 48)), FixedState((2, 8, 16)))
    assert needs[7] == (PagedKV(3, 10, 5, 6), FixedState((1, 48)), FixedState((6, 6, 4)))  # one tap is kept as two


# --------------------------------------------------------------------------- the whole model, every cut


@pytest.mark.parametrize("backend", BACKENDS)
@pytest.mark.parametrize("name", ["A", "B", "C", "D"])
def test_every_cut_matches_the_plain_implementation(tmp_path, backend, name):
    doc, seed = DOCS[name]
    tensors = make_folder(tmp_path, doc, seed, std=0.15)
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
@pytest.mark.parametrize("name", ["A", "C", "D"])
def test_the_residual_stream_after_every_layer_run(tmp_path, backend, name):
    """The stream after every run of a layer (a repeated layer counts each time), before the next
    pass's matrix: an embedding that is mixed in at the wrong place, or twice, shows here."""
    doc, seed = DOCS[name]
    tensors = make_folder(tmp_path, doc, seed, std=0.15)
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
    make_folder(tmp_path, doc, seed, std=0.15)
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
    """300 tokens one by one after a short prompt - the windows move over decoded tokens and their
    pages go back - with a second request joining half-way; the trace runs twice in one engine,
    so every page and slot is used again."""
    doc, seed = DOCS["A"]
    tensors = make_folder(tmp_path, doc, seed, std=0.15)
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
        helpers.run_steps(engine, steps[:150])
        engine.finish("a"), engine.finish("b")
        rows = helpers.run_steps(engine, steps)
        check_rows(replay.stack_rows(rows, "a", 330), reference["a"], dtype, f"long decoding {dtype}")
        check_rows(replay.stack_rows(rows, "b", 110), reference["b"], dtype, f"the request that joined {dtype}")
        assert sorted(engine.cache.free_pages()) == sorted(free) and engine.cache.slots.free_slots == 4


# heads of real widths: the tensor-memory and TMA attention kernels (64), the tiled kernel (96, 128), states of 64 x 128 and 128 x 32
DOC_WIDE = {
    "architecture": "Nodepel", "vocab": 400, "width": 128, "norm": {"eps": 1e-6}, "embedding": {"scale": 1.5},
    "loop": {"start": 1, "stop": 3, "times": 2},
    "layers": [
        layer(left(4, 2, 64, 64, 0.11, 200, 64, 10000.0), right(4, 2, 64, 128, 4), moe(6, 2, 64, 80)),
        layer(left(2, 1, 128, 96, 0.09, 70, 64), right(2, 2, 128, 32, 4), moe(4, 1, 32)),
        layer(left(8, 1, 64, 64, 0.1, 128, 32), right(3, 1, 256, 16, 2), None),
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
    tensors = make_folder(model_dir, doc, seed, std=0.15)
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
    doc, seed = DOCS["A"]
    tensors = make_folder(tmp_path, doc, seed, std=0.15)
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


def plan_layer(left_doc, right_doc, width, mlp=None, eps=1e-5):
    """The layer's specs as the plan builder makes them, with tensors named ``l0.*``."""
    doc = {"architecture": "Nodepel", "vocab": 8, "width": width, "norm": {"eps": eps}, "layers": [layer(left_doc, right_doc, mlp)]}
    return plan_from_document(doc)[2].layers[0]


LEFT = left(6, 3, 10, 7, 0.4, 9, 6, 50.0)
LEFT_ONE = left(5, 1, 8, 16, 0.5, 1, 8)
RIGHT = right(6, 3, 9, 5, 4)
RIGHT_ONE = right(2, 2, 16, 24, 1)
RIGHT_WIDE_CONV = right(4, 1, 70, 12, 8)


def side(which, left_doc, right_doc, width, eps=1e-5):
    return MIXERS.build, plan_layer(left_doc, right_doc, width, eps=eps).mixer.params["branches"][which][0]


@pytest.mark.parametrize("backend", BACKENDS)
@pytest.mark.parametrize("which,doc", [("left", LEFT), ("left", LEFT_ONE), ("right", RIGHT), ("right", RIGHT_ONE), ("right", RIGHT_WIDE_CONV)],
                         ids=["attention", "attention-window-of-one", "delta", "delta-one-tap", "delta-eight-taps"])
def test_each_branch_alone_in_steps_and_batches(backend, which, doc):
    for dtype in mixer_dtypes(backend):
        if which == "right" and dtype == torch.bfloat16:
            continue  # (a head's output may be small before its norm: bfloat16 is compared kernel by kernel)
        env = build_env(backend, dtype)
        build, spec = side(0 if which == "left" else 1, doc if which == "left" else LEFT, doc if which == "right" else RIGHT, 40)
        mixer = build(spec, env)
        w = bind(mixer, env, 11)
        g = torch.Generator().manual_seed(1)
        a, b = torch.randn(37, 40, generator=g).to(dtype), torch.randn(9, 40, generator=g).to(dtype)
        fn = plain.attention if which == "left" else plain.gated_delta
        want_a, want_b = (fn(w, f"l0.mix.{which}", doc, x.double(), 1e-5) for x in (a, b))
        in_steps_and_batches(mixer, env, dtype, a, b, want_a, want_b, which, 4.0)


@pytest.mark.parametrize("backend", BACKENDS)
@pytest.mark.parametrize("left_doc,right_doc", [(LEFT, RIGHT), (LEFT_ONE, RIGHT_ONE)], ids=["odd-columns", "even-columns"])
def test_both_branches_and_their_norms(backend, left_doc, right_doc):
    env = build_env(backend, torch.float32)
    mixer = MIXERS.build(plan_layer(left_doc, right_doc, 44).mixer, env)
    w = bind(mixer, env, 12)
    g = torch.Generator().manual_seed(2)
    a, b = torch.randn(37, 44, generator=g), torch.randn(9, 44, generator=g)
    m = {"left": left_doc, "right": right_doc}
    want_a, want_b = (plain.parallel_mixer(w, "l0.mix", m, x.double(), 1e-5) for x in (a, b))
    in_steps_and_batches(mixer, env, torch.float32, a, b, want_a, want_b, "both branches", 4.0)


@pytest.mark.parametrize("backend", BACKENDS)
@pytest.mark.parametrize("size", [5, 32, 70])
def test_a_planted_key_on_either_side_of_the_window_edge(backend, size):
    """One key is made to stand out (the key matrix is the query matrix and the asking row repeats its
    direction): right before the asking row, just inside and just outside the window, far outside, on
    either side of page borders; the asking row ends a portion or is decoded.  Inside it decides the
    output, outside it must not be felt at all."""
    env = build_env(backend, torch.float32)
    doc = left(2, 2, 16, 12, 2.0, size, 8, 5000.0)
    build, spec = side(0, doc, RIGHT, 32)
    mixer = build(spec, env)
    from shiso_llm_b200.weights import random_tensors
    from shiso_llm_b200.weights.loader import target_dtype
    specs = {s.name: s for s in mixer.tensor_specs()}
    stored = random_tensors(list(specs.values()), 31, 0.3, "bfloat16", 0.1)
    for k_name, q_name in {"l0.mix.left.k": "l0.mix.left.q", "l0.mix.left.k.norm": "l0.mix.left.q.norm"}.items():
        stored[k_name] = stored[q_name].clone()
    mixer.bind({k: v.to(env.device, target_dtype(specs[k], v.dtype, env.dtype)) for k, v in stored.items()})
    w = {k: v.double() for k, v in stored.items()}
    T = 150
    g = torch.Generator().manual_seed(3)
    base, probe = torch.randn(T, 32, generator=g) * 0.1, torch.randn(32, generator=g)
    quiet = base.clone()
    quiet[T - 1] = probe * 3.0
    without = plain.attention(w, "l0.mix.left", doc, quiet.double(), 1e-5)[T - 1]
    for back in sorted({1, size - 1, size, size + 1, 2 * size, 3, 4, 31, 32, 33, 120}):
        h = quiet.clone()
        h[T - 1 - back] = probe * 30.0
        want = plain.attention(w, "l0.mix.left", doc, h.double(), 1e-5)
        moved = (want[T - 1] - without).abs().max().item() / without.abs().max().item()
        assert (moved > 0.02) == (back < size) or back == 0, (back, moved)
        for tail in (0, 9):
            feeder = Feeder(mixer, env, pages=64)
            got = [feeder.step([("a", h[: T - tail - 7])])["a"], feeder.step([("a", h[T - tail - 7 : T - tail])])["a"]]
            for t in range(T - tail, T):
                got.append(feeder.step([("a", h[t : t + 1])])["a"])
            close(torch.cat(got), want, torch.float32, f"window of {size}: planted {back} back, {tail} decoded", 4.0)


@pytest.mark.parametrize("backend", BACKENDS)
def test_the_sink_takes_its_share(backend):
    """Sinks far above, near and far below the scores: a head whose sink dominates gives (nearly)
    nothing, one whose sink is far below is an ordinary softmax; a sink that is scaled with the scores,
    counted per key or left out differs."""
    env = build_env(backend, torch.float32)
    doc = left(4, 2, 12, 12, 0.3, 20, 12)
    build, spec = side(0, doc, RIGHT, 32)
    mixer = build(spec, env)
    sinks = torch.tensor([30.0, 1.5, -2.0, -200.0])
    w = bind(mixer, env, 7, 0.3, {"l0.mix.left.sink": lambda t: sinks})
    g = torch.Generator().manual_seed(5)
    h = torch.randn(50, 32, generator=g)
    want = plain.attention(w, "l0.mix.left", doc, h.double(), 1e-5)
    gone = plain.attention({**w, "l0.mix.left.sink": torch.full((4,), -1e9)}, "l0.mix.left", doc, h.double(), 1e-5)
    assert (want - gone).abs().max().item() > 0.1 * want.abs().max().item()
    feeder = Feeder(mixer, env)
    got = [feeder.step([("a", h[:1])])["a"], feeder.step([("a", h[1:40])])["a"]]
    got += [feeder.step([("a", h[t : t + 1])])["a"] for t in range(40, 50)]
    close(torch.cat(got), want, torch.float32, "sinks", 2.0)


@pytest.mark.parametrize("backend", BACKENDS)
def test_a_lost_state_or_convolution_window_shows(backend):
    """Decays of nearly one and a large first token: what it wrote is read for the whole sequence, so a
    state or a convolution window dropped (or taken twice) at a portion's start changes every row
    behind it; portions on either side of blocks of eight rows."""
    env = build_env(backend, torch.float32)
    doc = right(4, 2, 12, 10, 4)
    build, spec = side(1, LEFT, doc, 24)
    mixer = build(spec, env)
    w = bind(mixer, env, 3, 0.4, {"l0.mix.right.A_log": lambda t: t * 0.0 - 9.0})
    g = torch.Generator().manual_seed(4)
    h = torch.randn(75, 24, generator=g) * 0.2
    h[0] *= 40.0
    want = plain.gated_delta(w, "l0.mix.right", doc, h.double(), 1e-5)
    for sizes in ([75], [1], [2], [1, 2, 3], [7, 8, 9, 1], [16, 1, 15, 17], [3, 64]):
        feeder, got, at, i = Feeder(mixer, env), [], 0, 0
        while at < 75:
            n = min(sizes[i % len(sizes)], 75 - at)
            got.append(feeder.step([("a", h[at : at + n])])["a"])
            at, i = at + n, i + 1
        close(torch.cat(got), want, torch.float32, f"portions of {sizes}", 10.0)


@pytest.mark.parametrize("backend", BACKENDS)
def test_the_state_is_corrected_not_added_to(backend):
    """The same key again and again with a step of nearly one and no forgetting: a second write with
    the same value changes nothing, one with another value replaces it.  Plain linear attention would
    add them up; a correction taken before the decay, or a read-out before the write, differs."""
    env = build_env(backend, torch.float32)
    ops, T, D, V = env.ops, 21, 8, 4
    from types import SimpleNamespace
    step = SimpleNamespace(num_seqs=1, q_start=torch.tensor([0, T], dtype=torch.int32, device=env.device),
                           state_slots=torch.zeros(1, dtype=torch.int32, device=env.device))
    g = torch.Generator().manual_seed(1)
    key = torch.randn(1, D, generator=g).expand(T, D).contiguous()
    v = torch.randn(T, V, generator=g)
    v[5:13] = v[5]
    one = torch.full((T, 1), 40.0)  # beta = 1
    state = torch.zeros(1, 1, D, V, device=env.device)
    out = ops.delta_rule(*(x.to(env.device) for x in (key, key, v, one, -one)), torch.zeros(1, device=env.device), torch.zeros(1, device=env.device),
                         state, step, 1, 1, D, V, 1.0, 1e-12).double().cpu()
    assert (out - v.double()).abs().max().item() <= 1e-5 * v.abs().max().item()  # every read-out is the latest value
    # beta one half and a decay of one half each: u = (v - S k / 2) / 2 on the decayed state
    half = torch.zeros(T, 1)
    decay = torch.full((T, 1), 0.5)
    want = plain.delta_rule(plain.unit_vector(key.double()), plain.unit_vector(key.double()), v.double(), torch.full((T,), 0.5, dtype=torch.float64), decay[:, 0].double())
    state.zero_()
    out = ops.delta_rule(*(x.to(env.device) for x in (key, key, v, half, half)), torch.zeros(1, device=env.device), torch.zeros(1, device=env.device),
                         state, step, 1, 1, D, V, 1.0, 1e-6).double().cpu()
    close(out, want, torch.float32, "beta and decay of one half")  # softplus(0) = ln 2, exp(-ln 2) = 1/2


MLPS = {"shared": moe(7, 3, 14, 20), "plain": moe(7, 2, 9), "all-chosen": moe(4, 4, 8, 8), "one": moe(1, 1, 12, 6), "first-only": moe(9, 1, 5)}


@pytest.mark.parametrize("backend", BACKENDS)
@pytest.mark.parametrize("name", list(MLPS))
def test_feed_forwards_alone(backend, name):
    mlp = MLPS[name]
    for dtype in mixer_dtypes(backend):
        env = build_env(backend, dtype)
        part = FEED_FORWARDS.build(plan_layer(LEFT, RIGHT, 36, mlp).feed_forward, env)
        w = bind(part, env, 17, 0.3, {"l0.mlp.router.b": lambda t: t * 50.0})
        g = torch.Generator().manual_seed(2)
        for rows in (1, 5, 70):
            h = (torch.randn(rows, 36, generator=g) * 1.5).to(dtype)
            margins = []
            want = plain.mixture(w, "l0.mlp", mlp, h.double(), margins)
            y = part.forward(h.to(env.device), None)
            y = (y.materialize() if hasattr(y, "materialize") else y).double().cpu()
            sure = torch.ones(rows, dtype=torch.bool) if dtype == torch.float32 else margins[0] > CLOSE_CALL
            assert torch.isfinite(y).all()
            if sure.any():
                close(y[sure], want[sure], dtype, f"{name} feed-forward, {rows} rows {dtype}", 4.0)


@pytest.mark.parametrize("backend", BACKENDS)
def test_the_softmax_over_the_chosen_logits(backend):
    """Weights come from the chosen logits alone, whatever the others are, and logits so far apart that
    a softmax over all of them would round the second choice to zero still choose it; ties fall to the
    lower expert; logits may be a column range."""
    env = build_env(backend, torch.float32)
    logits = torch.tensor([[1.0, 3.0, 2.0, 2.5, -1.0], [0.5, 0.5, 0.5, 0.5, 0.5], [-300.0, 200.0, -150.0, -290.0, -400.0], [5.0, -5.0, 4.0, 4.5, 4.25]])
    wide = torch.cat([logits, torch.full((4, 3), 999.0)], dim=1).to(env.device)
    for z in (logits.to(env.device), wide[:, :5]):
        ids, weights = env.ops.moe_route(z, 2, 1, 1, 1.0, scores="chosen_softmax")
        assert ids.cpu().tolist() == [[1, 3], [0, 1], [1, 2], [0, 3]]
        want = torch.stack([plain.choose(row.double(), 2)[1] for row in logits])
        assert (weights.cpu().double() - want).abs().max().item() <= 1e-6
        ids, weights = env.ops.moe_route(z, 5, 1, 1, 1.0, scores="chosen_softmax")
        assert ids.cpu()[2].tolist() == [1, 2, 3, 0, 4] and abs(float(weights[0].sum()) - 1.0) < 1e-6


@pytest.mark.parametrize("backend", BACKENDS)
def test_the_pair_of_normed_branches(backend):
    """The pair added to the stream under the next norm, with a row list (before the head), on its own,
    and under a norm that knows no pairs; residual sums in float32."""
    for dtype in mixer_dtypes(backend):
        env = build_env(backend, dtype)
        for width in (50, 64, 2056):
            norm = NORMS.build(PartSpec("rmsnorm", {"tensor": "n", "size": width, "eps": 1e-5, "offset": 1.0}), env)
            other = NORMS.build(PartSpec("layernorm", {"tensor": "n", "size": width, "eps": 1e-5}), env)
            w = bind(norm, env, 3)
            w_other = bind(other, env, 3)
            g = torch.Generator().manual_seed(6)
            x = (torch.randn(9, width, generator=g) * 3).to(env.device)
            l, r = (torch.randn(9, width, generator=g).to(env.device, dtype) * s for s in (0.01, 7.0))
            lw, rw = (1.0 + 0.3 * torch.randn(width, generator=g).to(env.device) for _ in range(2))
            pair = NormedPair(env.ops, l, r, lw, rw, 0.5, 1e-5)
            c = [t.double().cpu() for t in (x, l, r, lw, rw)]
            delta = 0.5 * (plain.rms_norm(c[1], c[3], 1e-5) + plain.rms_norm(c[2], c[4], 1e-5))
            close(pair.materialize().double().cpu(), delta, torch.float32, f"pair {width}", 2.0)
            want = plain.centred_norm(c[0] + delta, w, "n", 1e-5)
            stream = Stream(x.clone())
            stream.add(pair)
            close(stream.normed(norm).double().cpu(), want, dtype, f"pair under a norm {width}", 2.0)
            assert (stream.residual.double().cpu() - c[0] - delta).abs().max().item() <= 1e-5 and stream.pending is None
            residual = x.clone()
            rows = torch.tensor([7, 2], dtype=torch.int32, device=env.device)
            close(norm.add_apply(residual, pair, rows).double().cpu(), want[[7, 2]], dtype, "rows", 2.0)
            assert torch.equal(residual, x)
            stream = Stream(x.clone())
            stream.add(pair)
            y = c[0] + delta
            y = (y - y.mean(-1, keepdim=True)) / torch.sqrt(y.var(-1, unbiased=False, keepdim=True) + 1e-5) * w_other["n"]
            close(stream.normed(other).double().cpu(), y, dtype, "under a layer norm", 2.0)


@pytest.mark.parametrize("backend", BACKENDS)
def test_the_stream_beside_the_first_rows(backend):
    for dtype in mixer_dtypes(backend):
        env = build_env(backend, dtype)
        g = torch.Generator().manual_seed(8)
        for tokens, width in ((5, 50), (1, 64), (33, 132)):
            x, first = (torch.randn(tokens, width, generator=g).to(env.device) for _ in range(2))
            d0 = torch.randn(tokens, width, generator=g).to(env.device, dtype)
            d1 = torch.randn(tokens, width, generator=g).to(env.device)
            kept = x.clone()
            for deltas in ((), (d0,), (d0, d1)):
                got = env.ops.stream_concat(x, deltas, first, dtype)
                total = sum((d.double() for d in deltas), x.double())
                assert got.dtype == dtype and torch.equal(x, kept)
                close(got.double().cpu(), torch.cat([total, first.double()], -1).cpu(), dtype, f"{tokens} x {width}, {len(deltas)} waiting")
