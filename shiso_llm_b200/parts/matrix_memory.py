"""A matrix memory with exponential gating (the recurrence known as mLSTM).

``q = W_q h * dim^(-1/2)`` and ``k = W_k h`` in ``heads`` of ``dim``, ``v = W_v h`` in ``heads`` of ``vdim``.
Per head and token a log input gate ``i`` and a log forget gate ``f``,

    i = cap tanh((W_i h + b_i) / cap),        f = log sigmoid(cap tanh((W_f h + b_f) / cap)).

A running maximum ``m`` (zero at the start) keeps the exponentials in range:

    m' = max(f + m, i),    S <- e^(f + m - m') S + e^(i - m') k v^T,    n <- e^(f + m - m') n + e^(i - m') k,
    o  = S^T q / (max(|n . q|, e^(-m')) + denominator_eps).

Each head's ``o`` is divided by its root mean square; the joined heads are multiplied by a weight and
by ``sigmoid(W_g h)`` and projected.  Per request the mixer keeps ``S``, ``n`` and ``m`` of every head,
float32, zero for a new request.

q, k, v and the gate's logits are one product; the two log gates are another one, whose result stays
float32.  A step of single rows is one launch behind the first (``ops.memory_step``).  Otherwise one kernel
turns the gate logits into each row's two factors by a scan of the maximum, one walks or tiles each
sequence's rows with the state, the normaliser carried as one more value column that is always 1,
and one forms the quotient, the norm and the gate.
"""

from __future__ import annotations

import torch

from ..config.errors import UnsupportedShape
from ..weights.spec import NORMAL, ONES, VECTOR, TensorSpec
from .base import MIXERS, DeferredLinear, FixedState, Mixer
from .lightning import MAX_STATE_ROWS


@MIXERS.register("matrix_memory")
class MatrixMemory(Mixer):
    """``params``: ``hidden_size``, ``num_heads``, ``head_dim``, ``v_head_dim``, ``gate_cap``, ``eps``,
    ``denominator_eps``, and names ``q_proj``, ``k_proj``, ``v_proj``, ``g_proj``, ``i_proj``, ``f_proj``, ``i_bias``,
    ``f_bias``, ``out_norm``, ``out_proj``."""

    PROJECTIONS = ("q_proj", "k_proj", "v_proj", "g_proj")

    def __init__(self, spec, env):
        super().__init__(spec, env)
        p = spec.params
        self.hidden = int(p["hidden_size"])
        self.heads = int(p["num_heads"])
        self.dim = int(p["head_dim"])
        self.vdim = int(p["v_head_dim"])
        self.cap = float(p["gate_cap"])
        self.eps, self.denominator_eps = float(p["eps"]), float(p["denominator_eps"])
        if not 0 < self.dim <= MAX_STATE_ROWS or self.vdim < 1:
            raise UnsupportedShape("head sizes", (self.dim, self.vdim), f"the recurrence kernels take states of up to {MAX_STATE_ROWS} key rows")
        if self.cap <= 0.0:
            raise UnsupportedShape("gate_cap", self.cap, "a cap on the gates is positive")
        self.names = {k: p[k] for k in (*self.PROJECTIONS, "i_proj", "f_proj", "i_bias", "f_bias", "out_norm", "out_proj")}
        self.in_matrix = self.gate_matrix = self.gate_bias = self.out_matrix = self.norm_weight = None

    def tensor_specs(self):
        n, qk, v = self.names, self.heads * self.dim, self.heads * self.vdim
        return [
            *(TensorSpec(n[k], (rows, self.hidden)) for k, rows in zip(self.PROJECTIONS, (qk, qk, v, v))),
            TensorSpec(n["i_proj"], (self.heads, self.hidden)), TensorSpec(n["f_proj"], (self.heads, self.hidden)),
            TensorSpec(n["i_bias"], (self.heads,), VECTOR, NORMAL, init_std=0.5),
            TensorSpec(n["f_bias"], (self.heads,), VECTOR, NORMAL, init_mean=3.0, init_std=1.0),
            TensorSpec(n["out_norm"], (v,), VECTOR, ONES),
            TensorSpec(n["out_proj"], (self.hidden, v)),
        ]

    def bind(self, tensors):
        n = self.names

        def joined(keys):
            mats = [tensors[n[k]] for k in keys]
            if len({m.dtype for m in mats}) > 1:
                mats = [m.float() for m in mats]
            return torch.cat(mats, dim=0).contiguous()

        self.in_matrix, self.gate_matrix = joined(self.PROJECTIONS), joined(("i_proj", "f_proj"))
        self.gate_bias = torch.cat([tensors[n["i_bias"]].to(torch.float32), tensors[n["f_bias"]].to(torch.float32)]).contiguous()
        self.norm_weight, self.out_matrix = tensors[n["out_norm"]], tensors[n["out_proj"]]

    def cache_spec(self):
        return (FixedState((self.heads, self.dim, self.vdim)), FixedState((self.heads, self.dim)), FixedState((self.heads,)))

    def forward(self, x, step, cache):
        ops = self.env.ops
        state, normaliser, top = (c.state for c in cache)
        qk, v = self.heads * self.dim, self.heads * self.vdim
        proj = ops.linear(x, self.in_matrix, self.env.dtype)
        out = torch.empty((x.shape[0], v), dtype=self.env.dtype, device=x.device)
        sizes = (self.heads, self.dim, self.vdim)
        in_one = getattr(ops, "memory_step", None)
        if in_one is None or in_one(
            x, self.gate_matrix, self.gate_bias, proj, self.norm_weight, state, normaliser, top, step, *sizes, self.cap, self.dim**-0.5,
            self.denominator_eps, self.eps, out,
        ) is None:
            logits = ops.linear(x, self.gate_matrix, torch.float32, self.gate_bias)
            fits = getattr(ops, "memory_chunks_supported", None)
            chunks = {"logs": True} if fits is not None and fits(proj, self.dim, self.vdim) else {}
            keep, add, floor = ops.memory_gates(logits, self.cap, top, step, **chunks)
            raw, read = ops.memory_recurrence(
                proj[:, :qk], proj[:, qk : 2 * qk], proj[:, 2 * qk : 2 * qk + v], keep, add, state, normaliser, step, *sizes, **chunks)
            ops.memory_output(raw, read, floor, proj[:, 2 * qk + v :], self.norm_weight, self.heads, self.vdim, self.dim**-0.5,
                              self.denominator_eps, self.eps, out)
        return DeferredLinear(ops, out, self.out_matrix, self.env.dtype)
