"""Raketar: typed configuration and model plan.

A decoder of parallel layers: one RMS norm per layer, whose output both the mixer and the
feed-forward read; their sum joins the residual stream times a constant.  Behind that every layer
takes a second, narrow look at its token: a slice of a per-layer table, gated by the stream, projected
back to the width, normed and added times the same constant.  A layer's mixer is ``attention`` -
differential attention: two softmax maps per head over the same values, the second subtracted with a
learned weight, the difference normed per head and gated entry by entry; neighbouring rotation pairs
on a linearly scaled ladder - or ``mlstm`` - a matrix memory with an exponential input gate, a sigmoid
forget gate and a running maximum that keeps both in range.  Its feed-forward is ``dense`` (a silu
gated pair), ``moe`` (sigmoid scores that scale the chosen experts' inputs, beside a shared expert) or
absent.  A stretch of layers may run several times with the same weights, each pass with caches and
states of its own; every pass starts by adding a vector of its own to the stream and, from the second
on, the embedding's output.  The head has a matrix of its own.

config.json keys: ``architecture``, ``vocab``, ``width``, ``norm.eps``, ``residual_mult``,
``token_side.dim``, ``loop.{start, stop, times}`` and ``layers``: a list of ``{"type", "mixer", "mlp"}``
with, for ``attention``, ``mixer.{heads, kv_heads, dim, vdim, scale, diff, rot.{dims, base,
scaling.factor}}``; for ``mlstm``, ``mixer.{heads, dim, vdim, gate_cap}``; and ``mlp.{kind, ff}`` or
``mlp.{kind, expert.ff, router.{experts, top}, shared.ff}`` or null.
Tensor names: ``embed``, ``head``, ``final.norm``, ``side.embed``, ``loop.step`` and, for layer ``i``,
``l<i>.norm1``, ``l<i>.mix.*`` (``q, k, v, lq1, lk1, lq2, lk2, g, o`` / ``q, k, v, g, o, norm, i, i.b, f,
f.b``), ``l<i>.mlp.{gate, up, down}`` or ``l<i>.mlp.{router, e<j>.{gate, up, down}, shared.{gate, up,
down}}`` and ``l<i>.side.{gate, proj, norm}``.
"""

from __future__ import annotations

import copy
from dataclasses import dataclass
from typing import Any, Mapping, Optional

from ..parts.plan import LayerSpec, ModelPlan, PartSpec, RunEntry
from .errors import ConfigMissing, InvalidValue
from .registry import register_architecture

ARCHITECTURE = "Raketar"
ATTENTION = "attention"
MEMORY = "mlstm"
DENSE = "dense"
MOE = "moe"
MAPS = 2  # softmax maps per attention head
DENOMINATOR_EPS = 1e-6  # added to the matrix memory's denominator
LOOP_VECTORS = "loop.step"
SIDE_TABLE = "side.embed"


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


def _positive(document, path: str, at: str = "") -> float:
    value = _num(document, path, at)
    if value <= 0.0:
        raise InvalidValue(at + path, value, "expected a positive number")
    return value


@dataclass(frozen=True)
class RaketarConfig:
    vocab: int
    width: int
    eps: float
    layers: tuple  # the documents of the layers, checked
    residual_mult: float = 1.0
    side_dim: Optional[int] = None
    loop: Optional[tuple] = None  # (start, stop, times)

    @classmethod
    def from_dict(cls, document: Mapping[str, Any]) -> "RaketarConfig":
        if document.get("architecture") != ARCHITECTURE:
            raise InvalidValue("architecture", document.get("architecture"), f"expected {ARCHITECTURE!r}")
        vocab, width = _int(document, "vocab"), _int(document, "width")
        eps = _num(document, "norm.eps")
        if not 0.0 < eps < 1.0:
            raise InvalidValue("norm.eps", eps, "expected a small positive number")
        mult = _num(document, "residual_mult") if document.get("residual_mult") is not None else 1.0
        side = _int(document, "token_side.dim") if document.get("token_side") is not None else None
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
        return cls(vocab=vocab, width=width, eps=eps, layers=tuple(copy.deepcopy(layers)), residual_mult=mult, side_dim=side, loop=loop)

    @staticmethod
    def _check_layer(at: str, layer) -> None:
        if not isinstance(layer, Mapping):
            raise InvalidValue(at[:-1], layer, "expected an object")
        kind = layer.get("type")
        if kind == ATTENTION:
            for key in ("heads", "kv_heads", "dim", "vdim"):
                _int(layer, f"mixer.{key}", at=at)
            _num(layer, "mixer.scale", at=at), _num(layer, "mixer.diff", at=at)
            m = layer["mixer"]
            if m["heads"] % m["kv_heads"]:
                raise InvalidValue(f"{at}mixer.kv_heads", m["kv_heads"], f"does not divide {m['heads']} query heads")
            if m.get("rot") is not None:
                dims = _int(layer, "mixer.rot.dims", 0, at=at)
                if dims % 2 or dims > m["dim"]:
                    raise InvalidValue(f"{at}mixer.rot.dims", dims, f"must be even and at most dim = {m['dim']}")
                if dims:
                    _positive(layer, "mixer.rot.base", at=at)
                if m["rot"].get("scaling") is not None:
                    _positive(layer, "mixer.rot.scaling.factor", at=at)
        elif kind == MEMORY:
            for key in ("heads", "dim", "vdim"):
                _int(layer, f"mixer.{key}", at=at)
            _positive(layer, "mixer.gate_cap", at=at)
        else:
            raise InvalidValue(f"{at}type", kind, f"expected {ATTENTION!r} or {MEMORY!r}")
        mlp = layer.get("mlp")
        if mlp is None:
            return
        if mlp.get("kind") == DENSE:
            _int(layer, "mlp.ff", at=at)
        elif mlp.get("kind") == MOE:
            experts, top = _int(layer, "mlp.router.experts", at=at), _int(layer, "mlp.router.top", at=at)
            if top > experts:
                raise InvalidValue(f"{at}mlp.router.top", top, f"more than the {experts} experts")
            _int(layer, "mlp.expert.ff", at=at)
            if mlp.get("shared") is not None:
                _int(layer, "mlp.shared.ff", at=at)
        else:
            raise InvalidValue(f"{at}mlp.kind", mlp.get("kind"), f"expected {DENSE!r} or {MOE!r}")

    def to_dict(self) -> dict:
        document = {"architecture": ARCHITECTURE, "vocab": self.vocab, "width": self.width, "norm": {"eps": self.eps},
                    "residual_mult": self.residual_mult, "layers": copy.deepcopy(list(self.layers))}
        if self.side_dim is not None:
            document["token_side"] = {"dim": self.side_dim}
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


def _position_spec(rot: Optional[Mapping[str, Any]]) -> PartSpec:
    if rot is None or not rot["dims"]:
        return PartSpec("none")
    scaling = rot.get("scaling") or {"factor": 1.0}
    return PartSpec("rope_half_split", {"theta": rot["base"], "rotary_dim": rot["dims"], "interleaved": True, "factor": scaling["factor"]})


def _mixer_spec(kind: str, m: Mapping[str, Any], p: str, width: int, eps: float) -> PartSpec:
    if kind == ATTENTION:
        return PartSpec("differential_attention", {
            "hidden_size": width, "num_heads": m["heads"], "num_kv_heads": m["kv_heads"], "head_dim": m["dim"], "v_head_dim": m["vdim"],
            "maps": MAPS, "scale": m["scale"], "mask": {"kind": "causal"}, "diff": m["diff"], "eps": eps, "position": _position_spec(m.get("rot")),
            "q_proj": f"{p}.q", "k_proj": f"{p}.k", "v_proj": f"{p}.v", "gate": f"{p}.g", "out_proj": f"{p}.o",
            "weight_vectors": ((f"{p}.lq1", f"{p}.lk1"), (f"{p}.lq2", f"{p}.lk2")),
        })
    return PartSpec("matrix_memory", {
        "hidden_size": width, "num_heads": m["heads"], "head_dim": m["dim"], "v_head_dim": m["vdim"], "gate_cap": m["gate_cap"],
        "eps": eps, "denominator_eps": DENOMINATOR_EPS, **{f"{x}_proj": f"{p}.{x}" for x in "qkvgif"}, "i_bias": f"{p}.i.b",
        "f_bias": f"{p}.f.b", "out_norm": f"{p}.norm", "out_proj": f"{p}.o",
    })


def _pair_names(p: str) -> dict:
    return {"gate": f"{p}.gate", "up": f"{p}.up", "down": f"{p}.down"}


def _ff_spec(mlp: Mapping[str, Any], p: str, width: int) -> PartSpec:
    if mlp["kind"] == DENSE:
        return PartSpec("swiglu", {"hidden_size": width, "intermediate_size": mlp["ff"], **_pair_names(p)})
    shared = None
    if mlp.get("shared") is not None:
        shared = PartSpec("swiglu", {"hidden_size": width, "intermediate_size": mlp["shared"]["ff"], **_pair_names(f"{p}.shared")})
    return PartSpec("routed_experts", {
        "hidden_size": width, "intermediate_size": mlp["expert"]["ff"], "experts": mlp["router"]["experts"], "top": mlp["router"]["top"],
        "scores": "sigmoid", "weigh": "input", "router": f"{p}.router",
        "expert_names": tuple(_pair_names(f"{p}.e{e}") for e in range(mlp["router"]["experts"])), "shared": shared,
    })


def build_plan(config: RaketarConfig) -> ModelPlan:
    width, eps = config.width, config.eps

    def norm(name: str) -> PartSpec:
        return PartSpec("rmsnorm", {"tensor": name, "size": width, "eps": eps})

    layers = []
    for i, layer in enumerate(config.layers):
        prefix, mlp, side = f"l{i}", layer.get("mlp"), None
        if config.side_dim is not None:
            side = PartSpec("token_side", {
                "hidden_size": width, "vocab_size": config.vocab, "dim": config.side_dim, "columns": len(config.layers) * config.side_dim,
                "first_column": i * config.side_dim, "eps": eps, "table": SIDE_TABLE, "gate": f"{prefix}.side.gate",
                "proj": f"{prefix}.side.proj", "norm": f"{prefix}.side.norm",
            })
        layers.append(LayerSpec(
            name=prefix,
            block=PartSpec("parallel_pre_norm", {"scale": config.residual_mult}),
            mixer=_mixer_spec(layer["type"], layer["mixer"], f"{prefix}.mix", width, eps),
            mixer_norm=norm(f"{prefix}.norm1"),
            feed_forward=_ff_spec(mlp, f"{prefix}.mlp", width) if mlp is not None else None,
            side=side,
        ))
    order = tuple(
        RunEntry(layer=i, add_first=bool(begins), add_vector=(LOOP_VECTORS, begins) if begins is not None else None)
        for i, begins in config.run_order()
    )
    unused = () if any(entry.add_vector is not None for entry in order) else (LOOP_VECTORS,)
    return ModelPlan(
        architecture=ARCHITECTURE,
        hidden_size=width,
        vocab_size=config.vocab,
        embedding=PartSpec("token_embedding", {"tensor": "embed", "vocab_size": config.vocab, "hidden_size": width}),
        layers=tuple(layers),
        order=order,
        final_norm=norm("final.norm"),
        head=PartSpec("linear_head", {"vocab_size": config.vocab, "hidden_size": width, "tied_to": None, "tensor": "head"}),
        unused_tensors=unused,
    )


register_architecture(ARCHITECTURE, RaketarConfig, build_plan)
