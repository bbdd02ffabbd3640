"""Several mixers side by side on the same input: ``sum_b scale_b * mixer_b(h)``, or, for two branches
with ``norms``, ``scale * (norm_1(mixer_1(h)) + norm_2(mixer_2(h)))``.

Every branch is a mixer that can work on columns: it has ``in_matrix`` (its input
projections joined, ``[in_width, hidden]``), ``mix(proj, step, cache, out, out_scale)`` and
``out_matrix`` (``[hidden, out_width]``).  The branches' input matrices are joined into ONE
product over ``h``, each branch reads its columns of the result and writes its columns of
one joint buffer - already multiplied by its scale, in float32 before rounding - and the
output projections, joined along their inputs, are ONE product that adds the branches up.
A branch's cache needs are the mixer's, in the branches' order.

With ``norms`` (one RMS norm over the model width per branch) the outputs cannot be added up by a
product: each branch writes rows of its own and has its own output product, and the norms, the
scaled sum, the residual sum and the norm of whatever reads the stream next are ONE kernel (a
``NormedPair`` that waits on the stream).  A branch's columns start on a multiple of eight (zero
rows between the joined matrices), so that kernels may read them 16 bytes at a time.
"""

from __future__ import annotations

import torch

from ..weights.spec import ONES, VECTOR, TensorSpec
from .base import MIXERS, DeferredLinear, Mixer, NormedPair, project

COLUMN_GRID = 8  # a branch's first column


@MIXERS.register("parallel_mixer")
class ParallelMixer(Mixer):
    """``params``: ``branches``, a list of ``(PartSpec, scale)``; optionally ``norms``, a tensor name per
    branch (two branches of one scale), with ``eps`` and ``hidden_size``."""

    takes_deferred_norm = True

    def __init__(self, spec, env):
        super().__init__(spec, env)
        self.branches = [MIXERS.build(part, env) for part, _ in spec.params["branches"]]
        self.scales = [float(scale) for _, scale in spec.params["branches"]]
        for branch in self.branches:
            if not all(hasattr(branch, a) for a in ("mix", "in_width", "out_width")):
                raise ValueError(f"{type(branch).__name__} cannot work on the columns of a joint product")
        self.norm_names = spec.params.get("norms")
        if self.norm_names is not None:
            if len(self.branches) != 2 or len(self.norm_names) != 2 or self.scales[0] != self.scales[1]:
                raise ValueError("normed branches come in pairs of one scale, with a norm each")
            self.eps, self.hidden = float(spec.params["eps"]), int(spec.params["hidden_size"])
        self.in_matrix = self.out_matrix = None
        self.out_matrices = self.norm_weights = ()
        # where each branch's views lie in the tuple this mixer is handed
        self._needs, self._cache_slices = [], []
        for branch in self.branches:
            need = branch.cache_spec()
            members = list(need) if isinstance(need, (tuple, list)) else ([] if need is None else [need])
            self._cache_slices.append((len(self._needs), len(members), isinstance(need, (tuple, list))))
            self._needs += members

    def sub_parts(self):
        return list(self.branches)

    def tensor_specs(self):
        specs = [spec for branch in self.branches for spec in branch.tensor_specs()]
        return specs + [TensorSpec(name, (self.hidden,), VECTOR, ONES) for name in self.norm_names or ()]

    @property
    def _columns(self):
        """Each branch's first column in the joint product."""
        first, at = [], 0
        for branch in self.branches:
            first.append(at)
            at += branch.in_width + (-branch.in_width % COLUMN_GRID if self.norm_names is not None else 0)
        return first

    def bind(self, tensors):
        for branch in self.branches:
            branch.bind(tensors)
        ins = [b.in_matrix for b in self.branches]
        outs = [b.out_matrix for b in self.branches]
        if len({m.dtype for m in ins + outs}) > 1:
            ins, outs = [m.float() for m in ins], [m.float() for m in outs]
        if self.norm_names is not None:
            ins = [torch.cat([m, m.new_zeros((-m.shape[0] % COLUMN_GRID, m.shape[1]))]) for m in ins]
            self.out_matrices = tuple(outs)
            self.norm_weights = tuple(tensors[name] for name in self.norm_names)
        else:
            self.out_matrix = torch.cat(outs, dim=1).contiguous()
        self.in_matrix = torch.cat(ins, dim=0).contiguous()
        for branch in self.branches:  # the joint matrices stand for them
            branch.in_matrix = branch.out_matrix = None

    def cache_spec(self):
        return tuple(self._needs)

    def forward(self, x, step, cache):
        ops = self.env.ops
        proj = project(ops, x, self.in_matrix, self.env.dtype)
        views = [tuple(cache[first : first + count]) if is_tuple else (cache[first] if count else None)
                 for first, count, is_tuple in self._cache_slices]
        if self.norm_names is not None:
            sides = []
            for branch, view, col_in, matrix in zip(self.branches, views, self._columns, self.out_matrices):
                out = torch.empty((proj.shape[0], branch.out_width), dtype=self.env.dtype, device=proj.device)
                branch.mix(proj[:, col_in : col_in + branch.in_width], step, view, out)
                sides.append(ops.linear(out, matrix, self.env.dtype))
            return NormedPair(ops, *sides, *self.norm_weights, self.scales[0], self.eps)
        out = torch.empty((proj.shape[0], self.out_matrix.shape[1]), dtype=self.env.dtype, device=proj.device)
        col_out = 0
        for branch, scale, view, col_in in zip(self.branches, self.scales, views, self._columns):
            branch.mix(proj[:, col_in : col_in + branch.in_width], step, view, out[:, col_out : col_out + branch.out_width], scale)
            col_out += branch.out_width
        return DeferredLinear(ops, out, self.out_matrix, self.env.dtype)
