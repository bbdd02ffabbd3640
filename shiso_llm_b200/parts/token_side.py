"""A layer's own look at its token, behind its sublayers.

``e`` is a slice of a second token table, ``table[token, first_column : first_column + dim]``, one slice
per layer; with the stream ``x`` as the sublayers left it,

    g = gelu_tanh(W_gate x) * e,        y = W_proj g,        x <- x + scale * norm(y) * w,

the norm an RMS norm over the model width.  The products run in the compute type, the gate's
activation and the table's entry in float32, and the last line waits on the stream (``NormedOutput``)
until the next norm adds it while it normalises.
"""

from __future__ import annotations

import torch

from ..config.errors import UnsupportedShape
from ..weights.spec import ONES, VECTOR, TensorSpec
from .base import SIDES, NormedOutput, SideInput


@SIDES.register("token_side")
class TokenSide(SideInput):
    """``params``: ``hidden_size``, ``vocab_size``, ``dim``, ``columns`` (of the whole table), ``first_column``,
    ``eps``, and names ``table``, ``gate``, ``proj``, ``norm``."""

    def __init__(self, spec, env):
        super().__init__(spec, env)
        p = spec.params
        self.hidden, self.vocab = int(p["hidden_size"]), int(p["vocab_size"])
        self.dim, self.columns, self.first = int(p["dim"]), int(p["columns"]), int(p["first_column"])
        self.eps = float(p["eps"])
        if not 0 <= self.first <= self.columns - self.dim:
            raise UnsupportedShape("side table", (self.first, self.dim, self.columns), "the layer's slice lies inside the table")
        self.names = {k: p[k] for k in ("table", "gate", "proj", "norm")}
        self.table = self.gate = self.proj = self.norm_weight = None

    def tensor_specs(self):
        n = self.names
        return [
            TensorSpec(n["table"], (self.vocab, self.columns), init_std=1.0, shared=True),
            TensorSpec(n["gate"], (self.dim, self.hidden)),
            TensorSpec(n["proj"], (self.hidden, self.dim)),
            TensorSpec(n["norm"], (self.hidden,), VECTOR, ONES),
        ]

    def bind(self, tensors):
        n = self.names
        self.table, self.gate, self.proj, self.norm_weight = (tensors[n[k]] for k in ("table", "gate", "proj", "norm"))

    def forward(self, rows, step, scale):
        ops, dtype = self.env.ops, self.env.dtype
        z = ops.linear(rows, self.gate, torch.float32)
        g = ops.side_gate(z, self.table, self.first, step.token_ids, getattr(step, "feed_index", None), getattr(step, "fed_tokens", None), dtype)
        return NormedOutput(ops, ops.linear(g, self.proj, dtype), self.norm_weight, scale, self.eps)
