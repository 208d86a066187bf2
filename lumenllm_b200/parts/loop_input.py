"""What happens to the stream where a pass of a loop over layers begins ("loop_input"):
x <- [x ; x0] Win^T + step[t], x0 the embedding's output and t the number of the pass, step a learned
vector a pass. Tensors: `tensor` [D, 2 D] (x's columns first) and `step_tensor` [times, D].

x as it is (with whatever update is still pending added) and x0 lie side by side in one buffer in the run's
type; x0's half is written once a step. The product's float32 partial sums go on as a ShapedUpdate whose
`base` is the pass's step vector, so that the next layer's norm makes the new stream while it reads them.
"""
from __future__ import annotations

import torch

from ..ops import kernels as K
from .base import need, register_part
from .linear import Linear
from .norm import ShapedUpdate


@register_part("stream", "loop_input")
class LoopInput:
    """Parameters: hidden_size, times, tensor, step_tensor."""

    @classmethod
    def tensors(cls, spec):
        p = spec.params
        D, times = int(need(p, "hidden_size", "loop_input")), int(need(p, "times", "loop_input"))
        return {need(p, "tensor", "loop_input"): ((D, 2 * D), "matrix"),
                need(p, "step_tensor", "loop_input"): ((times, D), "matrix")}

    def __init__(self, spec, weights, runtime):
        p = spec.params
        self.runtime = runtime
        self.D = int(p["hidden_size"])
        self.proj = Linear(weights[p["tensor"]], runtime)
        self.step = weights[p["step_tensor"]].to(device=runtime.device, dtype=torch.float32).contiguous()
        # a pass's vector on a boundary of 16 bytes whatever the width
        self.steps = [row.clone() for row in self.step]

    def start(self, h, ctx):
        both = torch.empty((h.shape[0], 2 * self.D), dtype=self.runtime.dtype, device=h.device)
        K.add_shaped_rmsnorm(h, [], None, 0.0, None, write_h=False, cast_to=both[:, self.D:])
        ctx.extras.setdefault("per_step", {})[id(self)] = both

    def forward(self, h, pending, ctx, index):
        both = ctx.extras["per_step"][id(self)]
        base = pending.base if isinstance(pending, ShapedUpdate) else None
        groups = pending.groups if isinstance(pending, ShapedUpdate) else ShapedUpdate.groups_of(pending)
        K.add_shaped_rmsnorm(h, groups, None, 0.0, None, write_h=False, base=base, cast_to=both[:, :self.D])
        u = self.proj(both, split_ok=True)
        return h, ShapedUpdate([(u, 1.0, None, None, 0.0)], base=self.steps[index])
