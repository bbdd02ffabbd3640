"""The gated delta rule: a linear attention whose state is corrected towards each new value.

``q = W_q h`` and ``k = W_k h`` in ``kv_heads`` of ``dim``, ``v = W_v h`` in ``heads`` of ``vdim``; head ``a``
reads query/key head ``a // (heads / kv_heads)``.  Each of the three passes a causal convolution
per channel (``taps`` wide, the last tap on the current token, zeros before a sequence's start, no
bias) and ``silu``; q and k are then brought to unit length per head, ``x / sqrt(sum x^2 +
unit_eps)``, and q is multiplied by ``dim^(-1/2)``.  With ``beta = sigmoid(W_b h)`` and
``g = exp(-exp(A_log) softplus(W_a h + dt_bias))``, one number each per head and token, a state
``S[dim, vdim]`` per head that starts at zero is walked in the order

    S <- g S,    u = beta (v - S^T k),    S <- S + k u^T,    o = S^T q,

so the read-out sees the current token's write.  Each head's ``o`` is divided by its root mean
square, times a ``[vdim]`` weight shared by the heads, times ``silu(W_g h)``, and the joined heads are
projected.  Per request the mixer keeps the convolutions' last ``taps - 1`` inputs and every head's
state, both float32.

The six input projections are one product with columns ``[q | k | v | g | b | a]``, the three
convolutions one over neighbouring columns.  Decays, step sizes, unit lengths, the state, norm and
gate are float32 inside the kernels.  The mixer also serves as a branch of ``parallel_mixer``.
"""

from __future__ import annotations

import torch

from ..config.errors import UnsupportedShape
from ..weights.spec import NORMAL, ONES, VECTOR, TensorSpec
from .base import MIXERS, DeferredLinear, FixedState, Mixer, project
from .lightning import MAX_STATE_ROWS
from .short_conv import MAX_TAPS


@MIXERS.register("gated_delta")
class GatedDelta(Mixer):
    """``params``: ``hidden_size``, ``num_heads``, ``num_kv_heads``, ``head_dim``, ``v_head_dim``, ``taps``,
    ``eps``, ``unit_eps``, and names ``q_proj``, ``k_proj``, ``v_proj``, ``g_proj``, ``b_proj``, ``a_proj``,
    ``q_conv``, ``k_conv``, ``v_conv``, ``a_log``, ``dt_bias``, ``out_norm``, ``out_proj``."""

    takes_deferred_norm = True
    PROJECTIONS = ("q_proj", "k_proj", "v_proj", "g_proj", "b_proj", "a_proj")

    def __init__(self, spec, env):
        super().__init__(spec, env)
        p = spec.params
        self.hidden = int(p["hidden_size"])
        self.heads = int(p["num_heads"])
        self.kv_heads = int(p["num_kv_heads"])
        self.dim = int(p["head_dim"])
        self.vdim = int(p["v_head_dim"])
        self.taps = int(p["taps"])
        self.eps = float(p["eps"])
        self.unit_eps = float(p["unit_eps"])
        if self.heads % self.kv_heads:
            raise UnsupportedShape("num_kv_heads", self.kv_heads, f"does not divide {self.heads} heads")
        if not 1 <= self.taps <= MAX_TAPS:
            raise UnsupportedShape("conv taps", self.taps, f"the convolution kernels take up to {MAX_TAPS} taps")
        if not 0 < self.dim <= MAX_STATE_ROWS or self.vdim < 1:
            raise UnsupportedShape("head sizes", (self.dim, self.vdim), f"the recurrence kernel takes states of up to {MAX_STATE_ROWS} rows")
        self.names = {k: p[k] for k in (*self.PROJECTIONS, "q_conv", "k_conv", "v_conv", "a_log", "dt_bias", "out_norm", "out_proj")}
        self.in_matrix = self.out_matrix = self.conv = self.dt_bias = self.a_log = self.norm = None

    @property
    def qk_cols(self):
        return self.kv_heads * self.dim

    @property
    def v_cols(self):
        return self.heads * self.vdim

    @property
    def conv_cols(self):
        return 2 * self.qk_cols + self.v_cols

    @property
    def window(self):
        """Inputs of the convolution that are kept (a convolution of one tap runs as one of two whose first is zero)."""
        return max(self.taps, 2) - 1

    @property
    def in_width(self):
        return self.conv_cols + self.v_cols + 2 * self.heads

    @property
    def out_width(self):
        return self.v_cols

    def tensor_specs(self):
        n = self.names
        rows = (self.qk_cols, self.qk_cols, self.v_cols, self.v_cols, self.heads, self.heads)
        specs = [TensorSpec(n[k], (r, self.hidden)) for k, r in zip(self.PROJECTIONS, rows)]
        specs += [TensorSpec(n[k], (r, self.taps), VECTOR, NORMAL, alt_shapes=((r, 1, self.taps),), init_std=0.5)
                  for k, r in zip(("q_conv", "k_conv", "v_conv"), rows)]
        return specs + [
            TensorSpec(n["a_log"], (self.heads,), VECTOR, NORMAL, init_mean=-1.0, init_std=0.7),
            TensorSpec(n["dt_bias"], (self.heads,), VECTOR, NORMAL, init_mean=-1.0, init_std=0.5),
            TensorSpec(n["out_norm"], (self.vdim,), VECTOR, ONES),
            TensorSpec(n["out_proj"], (self.hidden, self.v_cols)),
        ]

    def bind(self, tensors):
        n = self.names
        mats = [tensors[n[k]] for k in self.PROJECTIONS]
        if len({m.dtype for m in mats}) > 1:
            mats = [m.float() for m in mats]
        self.in_matrix = torch.cat(mats, dim=0).contiguous()
        conv = torch.cat([tensors[n[k]].to(torch.float32).reshape(-1, self.taps) for k in ("q_conv", "k_conv", "v_conv")], dim=0)
        if self.taps == 1:
            conv = torch.cat([torch.zeros_like(conv), conv], dim=1)
        self.conv = conv.contiguous()
        self.dt_bias, self.a_log, self.norm = tensors[n["dt_bias"]], tensors[n["a_log"]], tensors[n["out_norm"]]
        self.out_matrix = tensors[n["out_proj"]]

    def cache_spec(self):
        return (FixedState((self.window, self.conv_cols)), FixedState((self.heads, self.dim, self.vdim)))

    def mix(self, proj, step, cache, out, out_scale=1.0):
        """``proj[T, in_width]`` (rows may be strided) -> ``out[T, out_width]``."""
        if out_scale != 1.0:
            raise RuntimeError("this mixer's output has no scale")
        ops = self.env.ops
        window, state = cache
        c, qk, v, h = self.conv_cols, self.qk_cols, self.v_cols, self.heads
        in_one = getattr(ops, "delta_step", None)
        if in_one is not None and in_one(
            proj, c, self.conv, self.dt_bias, self.a_log, self.norm, window.state, state.state, step, self.heads, self.kv_heads,
            self.dim, self.vdim, self.dim**-0.5, self.unit_eps, self.eps, out,
        ) is not None:
            return  # a step of single rows: everything in one launch
        gate, b, a = proj[:, c : c + v], proj[:, c + v : c + v + h], proj[:, c + v + h : c + v + 2 * h]
        qkv = ops.causal_conv(proj[:, :c], self.conv, None, window.state, step, silu=True)
        raw = ops.delta_rule(
            qkv[:, :qk], qkv[:, qk : 2 * qk], qkv[:, 2 * qk :], b, a, self.dt_bias, self.a_log, state.state, step,
            self.heads, self.kv_heads, self.dim, self.vdim, self.dim**-0.5, self.unit_eps,
        )
        ops.delta_output(raw, gate, self.norm, self.heads, self.eps, out)

    def forward(self, x, step, cache):
        ops = self.env.ops
        proj = project(ops, x, self.in_matrix, self.env.dtype)
        out = torch.empty((proj.shape[0], self.out_width), dtype=self.env.dtype, device=proj.device)
        self.mix(proj, step, cache, out)
        return DeferredLinear(ops, out, self.out_matrix, self.env.dtype)
