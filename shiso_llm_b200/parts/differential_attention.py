"""Differential attention: two softmax maps per head over the same values, one subtracted from the other.

Every query head and every key head has ``maps`` parts of ``dim`` entries, laid out head by head; part
``i`` of a query head attends to part ``i`` of its key head, and all parts of a head read the head's
one value row.  With ``a_1`` and ``a_2`` the two maps' outputs, ``lambda = exp(sum(lq1 lk1)) -
exp(sum(lq2 lk2)) + diff`` (one number for the layer, formed when the weights are bound) and ``rms`` over a
head's ``vdim`` entries,

    o = (a_1 - lambda a_2) / rms(a_1 - lambda a_2) * (1 - diff) * sigmoid(W_g h),

entry by entry, and the joined heads are projected.

To the attention kernels the maps are heads: the mixer is ``masked_attention`` (masks, position
encodings, cache) over ``2 heads`` query and ``2 kv_heads`` key heads of which neighbours share a value
head.  A map's query heads of one key head have to be neighbours for that, so the rows of ``W_q`` are
put in the order (key head, map, query head of the group) when bound.  The maps' outputs stay float32
until the difference is taken, normed and gated by one row kernel - or, in bfloat16 at the sizes of
``ops.differential_attention``, all of it is one launch, for long prompt portions and for single tokens.
"""

from __future__ import annotations

import torch

from ..config.errors import UnsupportedShape
from ..weights.spec import NORMAL, VECTOR, TensorSpec
from .base import MIXERS, DeferredLinear
from .masked_attention import MaskedAttention
from .plan import PartSpec


@MIXERS.register("differential_attention")
class DifferentialAttention(MaskedAttention):
    """``params``: those of ``masked_attention`` that a softmax without head norms, biases and sinks takes
    (``num_heads`` and ``num_kv_heads`` count heads, not maps), ``maps`` (2), ``diff``, ``eps``, ``gate`` (a gate per
    entry) and ``weight_vectors``, two pairs of names of ``[dim]`` vectors."""

    def __init__(self, spec, env):
        p = dict(spec.params)
        self.maps = int(p.get("maps", 2))
        if self.maps != 2:
            raise UnsupportedShape("maps", self.maps, "one map is subtracted from the other: two are expected")
        self.pairs, self.groups = int(p["num_heads"]), int(p["num_kv_heads"])
        p.update(num_heads=self.pairs * self.maps, num_kv_heads=self.groups * self.maps, value_share=self.maps, gate_per="element")
        super().__init__(PartSpec(spec.kind, p), env)
        if self.head_norm is not None or self.weights != "softmax" or self.names["sink"] is not None or self.values != "projected":
            raise UnsupportedShape("differential attention", spec.kind, "plain softmax maps without head norms or sinks are expected")
        if self.names["gate"] is None:
            raise UnsupportedShape("gate", None, "the difference is gated entry by entry")
        self.diff = float(p["diff"])
        self.vectors = tuple(tuple(pair) for pair in p["weight_vectors"])
        self.second = None  # lambda

    @property
    def gate_cols(self):
        return self.pairs * self.vdim

    @property
    def out_width(self):
        return self.pairs * self.vdim

    def tensor_specs(self):
        return super().tensor_specs() + [TensorSpec(n, (self.dim,), VECTOR, NORMAL, init_std=0.1) for pair in self.vectors for n in pair]

    def _query_rows(self):
        # stored (head, map), wanted (key head, map, head of the group)
        rows = torch.arange(self.pairs * self.maps).view(self.groups, self.pairs // self.groups, self.maps)
        heads = rows.transpose(1, 2).reshape(-1)
        return (heads[:, None] * self.dim + torch.arange(self.dim)[None, :]).reshape(-1)

    def bind(self, tensors):
        tensors = dict(tensors)
        q = tensors[self.names["q_proj"]]
        tensors[self.names["q_proj"]] = q[self._query_rows().to(q.device)].contiguous()
        super().bind(tensors)
        first, second = (torch.exp((tensors[a].double() * tensors[b].double()).sum()) for a, b in self.vectors)
        self.second = float(first - second) + self.diff

    def mix(self, proj, step, cache, out, out_scale=1.0):
        """``proj[T, in_width]`` (rows may be strided) -> ``out[T, out_width]``."""
        if out_scale != 1.0:
            raise RuntimeError("this mixer's output has no scale")
        ops = self.env.ops
        gate = proj[:, self.q_cols + self.kv_cols :]
        q, table = self._prepare(proj, step, cache)
        in_one = getattr(ops, "differential_attention", None)
        if in_one is not None and self.mask == "window" and self.softcap is None and in_one(
            q, self.pairs, self.groups, cache.k, cache.v, table, cache.page_size, self.scale, self.size, self.keep_first, step, self.second,
            1.0 - self.diff, self.eps, gate, out,
        ) is not None:
            return  # both maps and their difference in one launch
        maps = ops.masked_attention(q, self.heads, cache.k, cache.v, table, cache.page_size, self.scale, self.mask, self.size,
                                    self.keep_first, step, softcap=self.softcap, out_dtype=torch.float32)
        ops.map_difference(maps, self.pairs, self.groups, self.second, 1.0 - self.diff, self.eps, gate, out)

    def forward(self, x, step, cache):
        ops = self.env.ops
        proj = ops.linear(x, self.in_matrix, self.env.dtype)
        out = torch.empty((proj.shape[0], self.out_width), dtype=self.env.dtype, device=proj.device)
        self.mix(proj, step, cache, out)
        return DeferredLinear(ops, out, self.out_matrix, self.env.dtype)
