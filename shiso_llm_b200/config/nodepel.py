"""Nodepel: typed configuration and model plan.

A pre-norm decoder with RMS norms whose weights are stored around zero.  Every layer's mixer is
``parallel``: windowed softmax attention ("left": one RMS norm over all query heads together and one
over all key heads, half-split rotation, a sink per head) and the gated delta rule ("right") read the
same input, and the mixer's output is half the sum of their outputs' RMS norms.  Its feed-forward
is a mixture of ungated squared-relu experts (a biased router, the softmax taken over the chosen
logits only) beside a shared expert times a sigmoid per token, or absent.  A stretch of layers may run
several times with the same weights, each pass with caches of its own; every pass starts by
projecting the stream and the embedding's output, side by side, back to the width and adding a
vector of its own.  The embedding is scaled; the head has a matrix of its own.

config.json keys: ``architecture``, ``vocab``, ``width``, ``norm.eps``, ``embedding.scale``,
``loop.{start, stop, times}`` and ``layers``: a list of ``{"type", "mixer", "mlp"}`` with
``mixer.left.{heads, kv_heads, dim, vdim, scale, mask.size, rot.{dims, base}}``,
``mixer.right.{heads, kv_heads, dim, vdim, conv}`` and ``mlp.{kind, expert.ff, router.{experts, top},
shared.ff}`` or null.  Tensor names: ``embed``, ``head``, ``final.norm``, ``loop.in``, ``loop.step`` and, for
layer ``i``, ``l<i>.norm1/2``, ``l<i>.mix.left.{q, k, v, q.norm, k.norm, sink, o, out}``,
``l<i>.mix.right.{q, k, v, q.conv, k.conv, v.conv, g, b, a, A_log, dt_bias, norm, o, out}``,
``l<i>.mlp.{router, router.b, e<j>.{up, down}, shared.{up, down, sg}}``.
"""

from __future__ import annotations

import copy
from dataclasses import dataclass
from typing import Any, Mapping, Optional

from ..parts.plan import LayerSpec, ModelPlan, PartSpec, RunEntry
from .errors import ConfigMissing, InvalidValue
from .registry import register_architecture

ARCHITECTURE = "Nodepel"
PARALLEL = "parallel"
MOE = "moe"
UNIT_EPS = 1e-6  # inside the root that brings the delta rule's keys and queries to unit length
BRANCH_SHARE = 0.5  # of each branch's normed output
LOOP_VECTORS, LOOP_MATRIX = "loop.step", "loop.in"


def _get(document: Mapping[str, Any], path: str, at: str = ""):
    value = document
    for key in path.split("."):
        if not isinstance(value, Mapping) or key not in value or value[key] is None:
            raise ConfigMissing(at + path)
        value = value[key]
    return value


def _int(document, path: str, least: int = 1, at: str = "") -> int:
    value = _get(document, path, at)
    if isinstance(value, bool) or not isinstance(value, int) or value < least:
        raise InvalidValue(at + path, value, f"expected an integer of at least {least}")
    return value


def _num(document, path: str, at: str = "") -> float:
    value = _get(document, path, at)
    if isinstance(value, bool) or not isinstance(value, (int, float)):
        raise InvalidValue(at + path, value, "expected a number")
    return float(value)


@dataclass(frozen=True)
class NodepelConfig:
    vocab: int
    width: int
    eps: float
    layers: tuple  # the documents of the layers, checked
    embedding_scale: float = 1.0
    loop: Optional[tuple] = None  # (start, stop, times)

    @classmethod
    def from_dict(cls, document: Mapping[str, Any]) -> "NodepelConfig":
        if document.get("architecture") != ARCHITECTURE:
            raise InvalidValue("architecture", document.get("architecture"), f"expected {ARCHITECTURE!r}")
        vocab, width = _int(document, "vocab"), _int(document, "width")
        eps = _num(document, "norm.eps")
        if not 0.0 < eps < 1.0:
            raise InvalidValue("norm.eps", eps, "expected a small positive number")
        embedding = document.get("embedding") or {}
        scale = _num(document, "embedding.scale") if embedding.get("scale") is not None else 1.0
        layers = _get(document, "layers")
        if not isinstance(layers, list) or not layers:
            raise InvalidValue("layers", layers, "expected a non-empty list of layers")
        for i, layer in enumerate(layers):
            cls._check_layer(f"layers[{i}].", layer)
        loop = None
        if document.get("loop") is not None:
            loop = (_int(document, "loop.start", 0), _int(document, "loop.stop", 0), _int(document, "loop.times", 1))
            if not loop[0] <= loop[1] <= len(layers):
                raise InvalidValue("loop", document["loop"], f"start <= stop <= {len(layers)} layers is needed")
        return cls(vocab=vocab, width=width, eps=eps, layers=tuple(copy.deepcopy(layers)), embedding_scale=scale, loop=loop)

    @staticmethod
    def _check_layer(at: str, layer) -> None:
        if not isinstance(layer, Mapping):
            raise InvalidValue(at[:-1], layer, "expected an object")
        if layer.get("type") != PARALLEL:
            raise InvalidValue(f"{at}type", layer.get("type"), f"expected {PARALLEL!r}")
        for side in ("left", "right"):
            for key in ("heads", "kv_heads", "dim", "vdim"):
                _int(layer, f"mixer.{side}.{key}", at=at)
            m = layer["mixer"][side]
            if m["heads"] % m["kv_heads"]:
                raise InvalidValue(f"{at}mixer.{side}.kv_heads", m["kv_heads"], f"does not divide {m['heads']} heads")
        left = layer["mixer"]["left"]
        _num(layer, "mixer.left.scale", at=at), _int(layer, "mixer.left.mask.size", at=at)
        dims = _int(layer, "mixer.left.rot.dims", 0, at=at)
        if dims % 2 or dims > left["dim"]:
            raise InvalidValue(f"{at}mixer.left.rot.dims", dims, f"must be even and at most dim = {left['dim']}")
        if dims and _num(layer, "mixer.left.rot.base", at=at) <= 0:
            raise InvalidValue(f"{at}mixer.left.rot.base", left["rot"]["base"], "expected a positive base")
        _int(layer, "mixer.right.conv", at=at)
        mlp = layer.get("mlp")
        if mlp is None:
            return
        if mlp.get("kind") != MOE:
            raise InvalidValue(f"{at}mlp.kind", mlp.get("kind"), f"expected {MOE!r}")
        experts, top = _int(layer, "mlp.router.experts", at=at), _int(layer, "mlp.router.top", at=at)
        if top > experts:
            raise InvalidValue(f"{at}mlp.router.top", top, f"more than the {experts} experts")
        _int(layer, "mlp.expert.ff", at=at)
        if mlp.get("shared") is not None:
            _int(layer, "mlp.shared.ff", at=at)

    def to_dict(self) -> dict:
        document = {"architecture": ARCHITECTURE, "vocab": self.vocab, "width": self.width, "norm": {"eps": self.eps},
                    "embedding": {"scale": self.embedding_scale}, "layers": copy.deepcopy(list(self.layers))}
        if self.loop is not None:
            document["loop"] = dict(zip(("start", "stop", "times"), self.loop))
        return document

    def run_order(self) -> list:
        """``(layer, pass)`` in running order: ``pass`` is the number of the pass that begins with
        this run of the layer, or None."""
        n = len(self.layers)
        if self.loop is None or self.loop[0] == self.loop[1]:  # (a stretch without layers has no pass to begin)
            return [(i, None) for i in range(n)]
        start, stop, times = self.loop
        order = [(i, None) for i in range(start)]
        for t in range(times):
            order += [(i, t if i == start else None) for i in range(start, stop)]
        return order + [(i, None) for i in range(stop, n)]


def _left_spec(m: Mapping[str, Any], p: str, width: int, eps: float) -> PartSpec:
    rot = m["rot"]
    position = PartSpec("rope_half_split", {"theta": rot["base"], "rotary_dim": rot["dims"]}) if rot["dims"] else PartSpec("none")
    return PartSpec("masked_attention", {
        "hidden_size": width, "num_heads": m["heads"], "num_kv_heads": m["kv_heads"], "head_dim": m["dim"], "v_head_dim": m["vdim"],
        "scale": m["scale"], "mask": {"kind": "window", "size": m["mask"]["size"]}, "weights": "softmax", "sink": f"{p}.sink",
        "head_norm": "joined", "eps": eps, "position": position, "q_proj": f"{p}.q", "k_proj": f"{p}.k", "v_proj": f"{p}.v",
        "q_norm": f"{p}.q.norm", "k_norm": f"{p}.k.norm", "out_proj": f"{p}.o",
    })


def _right_spec(m: Mapping[str, Any], p: str, width: int, eps: float) -> PartSpec:
    return PartSpec("gated_delta", {
        "hidden_size": width, "num_heads": m["heads"], "num_kv_heads": m["kv_heads"], "head_dim": m["dim"], "v_head_dim": m["vdim"],
        "taps": m["conv"], "eps": eps, "unit_eps": UNIT_EPS,
        **{f"{x}_proj": f"{p}.{x}" for x in "qkvgba"}, **{f"{x}_conv": f"{p}.{x}.conv" for x in "qkv"},
        "a_log": f"{p}.A_log", "dt_bias": f"{p}.dt_bias", "out_norm": f"{p}.norm", "out_proj": f"{p}.o",
    })


def _ff_spec(mlp: Mapping[str, Any], p: str, width: int) -> PartSpec:
    shared = None
    if mlp.get("shared") is not None:
        shared = PartSpec("relu2_ff", {"hidden_size": width, "intermediate_size": mlp["shared"]["ff"],
                                       "up": f"{p}.shared.up", "down": f"{p}.shared.down"})
    return PartSpec("routed_experts", {
        "hidden_size": width, "intermediate_size": mlp["expert"]["ff"], "experts": mlp["router"]["experts"], "top": mlp["router"]["top"],
        "scores": "chosen_softmax", "router": f"{p}.router", "router_bias": f"{p}.router.b", "activation": "relu2",
        "expert_names": tuple({"up": f"{p}.e{e}.up", "down": f"{p}.e{e}.down"} for e in range(mlp["router"]["experts"])),
        "shared": shared, "shared_gate": f"{p}.shared.sg" if shared is not None else None,
    })


def build_plan(config: NodepelConfig) -> ModelPlan:
    width, eps = config.width, config.eps

    def norm(name: str) -> PartSpec:
        return PartSpec("rmsnorm", {"tensor": name, "size": width, "eps": eps, "offset": 1.0})

    layers = []
    for i, layer in enumerate(config.layers):
        prefix, mlp, m = f"l{i}", layer.get("mlp"), layer["mixer"]
        layers.append(LayerSpec(
            name=prefix,
            block=PartSpec("pre_norm"),
            mixer=PartSpec("parallel_mixer", {
                "branches": [(_left_spec(m["left"], f"{prefix}.mix.left", width, eps), BRANCH_SHARE),
                             (_right_spec(m["right"], f"{prefix}.mix.right", width, eps), BRANCH_SHARE)],
                "norms": (f"{prefix}.mix.left.out", f"{prefix}.mix.right.out"), "eps": eps, "hidden_size": width,
            }),
            mixer_norm=norm(f"{prefix}.norm1"),
            feed_forward=_ff_spec(mlp, f"{prefix}.mlp", width) if mlp is not None else None,
            feed_forward_norm=norm(f"{prefix}.norm2") if mlp is not None else None,
        ))
    order = tuple(
        RunEntry(layer=i, mix_first=LOOP_MATRIX if begins is not None else None,
                 add_vector=(LOOP_VECTORS, begins) if begins is not None else None)
        for i, begins in config.run_order()
    )
    unused = tuple(f"l{i}.norm2" for i, layer in enumerate(config.layers) if layer.get("mlp") is None)
    if not any(entry.mix_first is not None for entry in order):
        unused += (LOOP_VECTORS, LOOP_MATRIX)
    return ModelPlan(
        architecture=ARCHITECTURE,
        hidden_size=width,
        vocab_size=config.vocab,
        embedding=PartSpec("token_embedding", {"tensor": "embed", "vocab_size": config.vocab, "hidden_size": width,
                                               "scale": config.embedding_scale}),
        layers=tuple(layers),
        order=order,
        final_norm=norm("final.norm"),
        head=PartSpec("linear_head", {"vocab_size": config.vocab, "hidden_size": width, "tied_to": None, "tensor": "head"}),
        unused_tensors=unused,
    )


register_architecture(ARCHITECTURE, NodepelConfig, build_plan)
