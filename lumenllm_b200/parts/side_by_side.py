"""Several mixers side by side ("side_by_side"): all read the same normed rows, and the layer's
update is the weighted sum of theirs, sum_i scale_i * mixer_i(y).

Parameters: `parts`, a list of {"mixer": PartSpec, "scale": number}. Each child is a mixer part like
any other, with tensors under its own prefix. At most one child may keep a key/value cache: the
layer's run has one cache entry, and the child that declared the need is the one that finds it in the
EntryView. Children that keep a per-sequence state find it there too; where several do, the run's state
row is their states one behind the other (float32, each from a multiple of four numbers on) and each is
handed a view of its own. The children's updates are
not added up here: they go on as the groups of a ScaledUpdate, each with its factor, for the next
norm to add while it reads the stream. A child's entry may name an `out_norm` = {"tensor": name, "eps":
number, "size": width}: its update is then RMS-normed over the stream's width before it is added, and the
groups go on as a ShapedUpdate.

Where every child says `projects_input` (its first step is a product of the rows with matrices of
its own) the children are built with `external_projection`, their matrices are stacked row-wise,
and ONE product serves them all; a child is handed the product and the column where its own
columns begin. A child whose kernels read from column 0 (`needs_first_columns`) comes first in the
stack; two such children are not fused.
"""
from __future__ import annotations

import math

import torch

from ..config.spec import PartSpec
from .base import build_part, need, part_class, part_tensors, register_part
from .linear import Linear
from .norm import ScaledUpdate, ShapedUpdate


class _ChildView:
    """An EntryView whose mixer state is a child's piece of the run's state row."""

    def __init__(self, entry, offset, shape):
        self._entry, self._offset, self._shape = entry, offset, shape

    def __getattr__(self, name):
        return getattr(self._entry, name)

    def state(self, name="mixer"):
        if name != "mixer":
            return self._entry.state(name)
        return self._entry.state()[:, self._offset:self._offset + math.prod(self._shape)].unflatten(1, self._shape)


@register_part("mixer", "side_by_side")
class SideBySide:
    @classmethod
    def tensors(cls, spec):
        t = {}
        for child in need(spec.params, "parts", "side_by_side"):
            t.update(part_tensors("mixer", child["mixer"]))
            if child.get("out_norm"):
                t[child["out_norm"]["tensor"]] = ((int(child["out_norm"]["size"]),), "norm")
        return t

    def __init__(self, spec, weights, runtime):
        children = need(spec.params, "parts", "side_by_side")
        if not children:
            raise ValueError("side_by_side: at least one mixer")
        kinds = [part_class("mixer", c["mixer"].kind) for c in children]
        fused = (len(children) > 1 and all(getattr(k, "projects_input", False) for k in kinds)
                 and sum(bool(getattr(k, "needs_first_columns", False)) for k in kinds) <= 1)
        specs = [c["mixer"] if not fused else PartSpec(c["mixer"].kind, dict(c["mixer"].params, external_projection=True),
                                                        c["mixer"].prefix) for c in children]
        self.mixers = [build_part("mixer", sp, weights, runtime) for sp in specs]
        self.scales = [float(c.get("scale", 1.0)) for c in children]
        self.proj, self.col0 = None, [0] * len(children)
        if fused:
            order = sorted(range(len(children)), key=lambda i: not getattr(kinds[i], "needs_first_columns", False))
            mats, at = [], 0
            for i in order:
                self.col0[i] = at
                mats += self.mixers[i].input_mats
                at += sum(m.shape[0] for m in self.mixers[i].input_mats)
                self.mixers[i].input_mats = True        # the stack holds them now
            self.proj = Linear.stacked(mats, runtime)
        if sum(m.cache_need() is not None for m in self.mixers) > 1:
            raise ValueError("side_by_side: at most one of the mixers may keep a key/value cache")
        norms = [c.get("out_norm") for c in children]
        self.out_norms = [None if n is None else (weights[n["tensor"]].to(device=runtime.device, dtype=torch.float32).contiguous(),
                                                  float(n["eps"])) for n in norms]
        # several children with states: where each one's begins in the run's state row
        states = [m.state_shape() for m in self.mixers]
        self.state_at, self.state_size = [None] * len(states), 0
        if sum(s is not None for s in states) > 1:
            for i, s in enumerate(states):
                if s is not None:
                    if s[1] != torch.float32:
                        raise ValueError("side_by_side: states that share a row are float32")
                    self.state_at[i] = (self.state_size, tuple(s[0]))
                    self.state_size += (math.prod(s[0]) + 3) // 4 * 4

    @property
    def graph_safe(self):
        return all(getattr(m, "graph_safe", False) for m in self.mixers)

    def cache_need(self):
        return next((n for n in (m.cache_need() for m in self.mixers) if n is not None), None)

    def state_shape(self):
        if self.state_size:
            return ((self.state_size,), torch.float32)
        return next((s for s in (m.state_shape() for m in self.mixers) if s is not None), None)

    def forward(self, y, ctx, entry):
        views = [entry if at is None else _ChildView(entry, *at) for at in self.state_at]
        if self.proj is None:
            updates = [m.forward(y, ctx, v) for m, v in zip(self.mixers, views)]
        else:
            u = self.proj(y, split_ok=True)        # the children's columns side by side, possibly partial sums
            updates = [m.forward(y, ctx, v, projected=u, col0=c) for m, v, c in zip(self.mixers, views, self.col0)]
        if any(n is not None for n in self.out_norms):
            return ShapedUpdate([(d, s, None) + (n or (None, 0.0)) for d, s, n in zip(updates, self.scales, self.out_norms)])
        return ScaledUpdate(list(zip(updates, self.scales)))
