"""The model: parts assembled from a plan, run in the plan's order.

Nothing here names an architecture.  ``Model`` builds one block per layer of the
plan, collects the tensors they ask for, binds them after loading, reports the cache
need of every run entry, and runs a step: embedding, the run order, and the final
norm + head for the rows whose logits are wanted.
"""

from __future__ import annotations

from typing import Optional

import torch

from ..weights.spec import NORMAL, VECTOR, TensorSpec
from .base import BLOCKS, EMBEDDINGS, HEADS, NORMS, BuildEnv, Stream
from .plan import ModelPlan


def stream_value(stream: Stream) -> torch.Tensor:
    """The residual stream as float32 rows, with the block output that is still waiting to be
    added, without touching the stream: a product that has not run is run on the side."""
    lanes = stream.lane_values()
    if lanes is not None:
        return lanes.sum(0)
    x = stream.residual
    waiting = stream.pending
    if waiting is None:
        return x.clone()
    total = x.clone()
    for part in waiting if isinstance(waiting, tuple) else (waiting,):
        if hasattr(part, "materialize"):
            part = part.materialize()
        total += part.to(x.dtype)
    return total


def residual_stats(label: str, x: torch.Tensor) -> str:
    """One line about a block of float32 rows: element count, root mean square and largest
    magnitude of the finite values, zeros, non-finite values and the first four values - the
    line of the reference's layer dump (crates/shiso-engine/src/trace.rs:49-138)."""
    flat = x.detach().to(torch.float64).flatten().cpu()
    finite = torch.isfinite(flat)
    good = flat[finite]
    rms = float(good.pow(2).mean().sqrt()) if good.numel() else 0.0
    absmax = float(good.abs().max()) if good.numel() else 0.0
    first = [float(v) for v in flat[:4]]
    return (f"{label}: n={flat.numel()} rms={rms:.6e} absmax={absmax:.6e} zeros={int((good == 0).sum())} "
            f"non_finite={int((~finite).sum())} first={first}")


class Model:
    def __init__(self, plan: ModelPlan, env: BuildEnv):
        self.plan = plan
        self.env = env
        self.embedding = EMBEDDINGS.build(plan.embedding, env)
        self.blocks = [BLOCKS.build(layer.block, env, layer) for layer in plan.layers]
        self.final_norm = NORMS.build(plan.final_norm, env)
        self.head = HEADS.build(plan.head, env)
        # tensors whose rows run entries add to the stream: name -> rows, and, once bound, the tensor
        self.entry_vectors = {}
        for entry in plan.order:
            if entry.add_vector is not None:
                name, row = entry.add_vector
                self.entry_vectors[name] = max(self.entry_vectors.get(name, 0), int(row) + 1)
        self.vectors = {}
        # matrices that take the stream and the embedding's output side by side back to the width
        self.entry_mixes = tuple(dict.fromkeys(entry.mix_first for entry in plan.order if entry.mix_first is not None))
        self.mixes = {}
        self.keeps_first = any(entry.add_first or entry.mix_first is not None for entry in plan.order)
        self.bound = False

    # ------------------------------------------------------------------ weights

    def parts(self):
        return [self.embedding, *self.blocks, self.final_norm, self.head]

    def tensor_specs(self) -> list[TensorSpec]:
        specs, shared = [], {}
        for part in self.parts():
            for spec in part.tensor_specs():
                if shared.get(spec.name) == spec and spec.shared:
                    continue  # a table that several parts read
                shared[spec.name] = spec
                specs.append(spec)
        for name, rows in self.entry_vectors.items():
            specs.append(TensorSpec(name, (rows, self.plan.hidden_size), VECTOR, NORMAL))
        for name in self.entry_mixes:
            specs.append(TensorSpec(name, (self.plan.hidden_size, 2 * self.plan.hidden_size)))
        return specs

    def bind(self, tensors: dict[str, torch.Tensor]) -> None:
        for part in self.parts():
            part.bind(tensors)
        self.vectors = {name: tensors[name] for name in self.entry_vectors}
        self.mixes = {name: tensors[name] for name in self.entry_mixes}
        self.bound = True

    @property
    def graph_safe(self) -> bool:
        def walk(part):
            yield part
            for sub in part.sub_parts():
                yield from walk(sub)

        return all(p.graph_safe for top in self.parts() for p in walk(top))

    # ------------------------------------------------------------------ cache needs

    def cache_needs(self) -> list:
        """Per run entry: the cache its mixer needs (one need, a tuple of needs, or None - also
        for a borrowing entry); behind the run entries, the embedding's need if it has one."""
        needs = []
        for entry in self.plan.order:
            if entry.cache_of is not None:
                needs.append(None)
            else:
                needs.append(self.blocks[entry.layer].mixer_part().cache_spec())
        if self.embedding.cache_spec() is not None:
            needs.append(self.embedding.cache_spec())
        return needs

    # ------------------------------------------------------------------ additions between entries

    def _add_to_stream(self, stream: Stream, entry, first):
        """What ``entry`` does to the stream before its layer: ``mix_first``'s product over the stream and the
        embedding's rows side by side (the block output that was waiting is added on the way in), and / or additions: the block output that was waiting, the
        embedding's rows (``first``) and a row of a tensor, in one kernel.  Returns the embedding's
        rows, which the first call keeps apart (it then writes the sums to rows of their own)."""
        ops = self.env.ops
        if stream.lanes is not None or stream.lane_update is not None:
            raise RuntimeError("rows are added between entries of a model with one residual stream")
        vector = None
        if entry.add_vector is not None:
            name, row = entry.add_vector
            vector = self.vectors[name][row]
        waiting = stream.take_pending()
        deltas = list(waiting) if isinstance(waiting, tuple) else ([waiting] if waiting is not None else [])
        if entry.mix_first is not None:
            if first is None:  # the stream is the embedding's output itself, and is not written again
                first = stream.residual
            side_by_side = ops.stream_concat(stream.residual, tuple(deltas), first, self.env.dtype)
            # (a vector of the entry rides as the product's bias)
            stream.residual = ops.linear(side_by_side, self.mixes[entry.mix_first], torch.float32, None if entry.add_first else vector)
            stream.current = None
            if entry.add_first:
                ops.stream_add(stream.residual, (first,), vector)
            return first
        if entry.add_first:
            if first is None:
                raise RuntimeError("the first run entry cannot add the embedding's rows to themselves")
            deltas.append(first)
        keep = self.keeps_first and first is None
        if keep:
            first = stream.residual
        stream.residual = ops.stream_add(stream.residual, tuple(deltas), vector, in_place=not keep)
        stream.current = None
        return first

    # ------------------------------------------------------------------ one step

    def forward(self, step, cache, layer_hook=None, add_hook=None) -> Optional[torch.Tensor]:
        """Runs the rows of ``step`` through every run entry; returns float32 logits
        ``[len(step.want_rows), vocab]`` or None when no row is wanted.

        ``layer_hook(position, stream)`` is called after the embedding (position -1) and after
        every run entry; ``stream_value(stream)`` gives the residual rows at that point.
        ``add_hook(stream)`` is called whenever a part leaves its output on the stream (after the
        mixer and after the feed-forward of a block).  Both are diagnostics: they synchronise,
        so a step with a hook is never captured."""
        if not self.bound:
            raise RuntimeError("the model has no weights yet: load or bind them first")
        if self.embedding.cache_spec() is not None:
            stream = Stream(self.embedding.forward(step, cache.view(len(self.plan.order))), add_hook)
        else:
            stream = Stream(self.embedding.forward(step), add_hook)
        if layer_hook is not None:
            layer_hook(-1, stream)
        first = None
        for pos, entry in enumerate(self.plan.order):
            if entry.add_first or entry.add_vector is not None or entry.mix_first is not None:
                first = self._add_to_stream(stream, entry, first)
            elif self.keeps_first and first is None and pos == 0:
                first = stream.residual.clone()  # the first block adds to the residual in place
            if entry.cache_of is None:
                view = cache.view(pos)
            else:
                view = cache.view(entry.cache_of, owner=False)
            self.blocks[entry.layer].forward(stream, step, view)
            if layer_hook is not None:
                layer_hook(pos, stream)
        if step.num_wanted == 0:
            return None
        stream.merge_lanes(self.env.ops)
        if getattr(step, "wants_every_row", False):
            # every row in order (a decode step): the norm that closes the last block is the final norm
            # (handed over unevaluated to a head that says it takes that: its product may apply the row scale itself)
            return self.head.forward(stream.normed(self.final_norm, deferred=getattr(self.head, "takes_deferred_norm", False)))
        rows = step.want_rows
        delta = stream.take_pending(self.final_norm)
        if delta is not None:
            normed = self.final_norm.add_apply(stream.residual, delta, rows)
        else:
            normed = self.final_norm.apply(self.env.ops.gather_rows(stream.residual, rows))
        return self.head.forward(normed)
