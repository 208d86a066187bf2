"""A recurrent block with a real-gated linear recurrent unit ("real_gated_lru"): a linear recurrence
over time with one state number a channel, in place of attention.

In order, for C channels in B blocks: y = gelu_tanh(h Wy^T + by); u = a causal convolution over time
of h Wx^T + bx on each channel of its own (`taps` taps with a bias, the last tap the current token's,
zeros before a sequence's start, no activation); in every block g, with u_g its C/B channels,
r = sigmoid(Ra_g u_g + ra_g), i = sigmoid(Ri_g u_g + ri_g); log a = -8 r softplus(lam);
S <- a S + sqrt(1 - a^2) i u; out = (S y) Wo^T.

A sequence's state is S [C] and the convolution's last taps - 1 inputs; both start at zero and are
carried from step to step, so a sequence may be fed in any portions. Everything that enters the
recurrence is float32; the products run in the run's type with float32 sums (the gates' products of
blocks on the tensor cores: ops.kernels.gemm_tc_blocks). Wy and Wx are one product, and so are both
gates of all blocks.
"""
from __future__ import annotations

import torch
import torch.nn.functional as F

from ..ops import kernels as K
from .base import need, register_part
from .linear import Linear

DECAY_POWER = 8.0        # the c of log a = -c r softplus(lam)


@register_part("mixer", "real_gated_lru")
class RealGatedLRU:
    graph_safe = True

    @staticmethod
    def _sizes(p):
        return tuple(int(need(p, k, "real_gated_lru")) for k in ("hidden_size", "channels", "blocks", "taps"))

    @classmethod
    def tensors(cls, spec):
        D, C, B, taps = cls._sizes(spec.params)
        pre, bs = spec.prefix, C // B
        return {f"{pre}.y": ((C, D), "matrix"), f"{pre}.y.b": ((C,), "matrix"),
                f"{pre}.x": ((C, D), "matrix"), f"{pre}.x.b": ((C,), "matrix"),
                f"{pre}.conv": ((C, taps), "matrix"), f"{pre}.conv.b": ((C,), "matrix"),
                f"{pre}.ra": ((B, bs, bs), "matrix"), f"{pre}.ra.b": ((B, bs), "matrix"),
                f"{pre}.ri": ((B, bs, bs), "matrix"), f"{pre}.ri.b": ((B, bs), "matrix"),
                f"{pre}.lam": ((C,), "matrix"), f"{pre}.o": ((D, C), "matrix")}

    def __init__(self, spec, weights, runtime):
        self.runtime = runtime
        self.D, self.C, self.B, self.taps = self._sizes(spec.params)
        if self.C % self.B:
            raise ValueError(f"{self.C} channels do not divide into {self.B} blocks")
        if not 1 <= self.taps <= 16:
            raise ValueError(f"a convolution of {self.taps} taps: this kernel takes 1 to 16")
        self.bs = self.C // self.B
        pre = spec.prefix
        f32 = lambda n: weights[n].to(device=runtime.device, dtype=torch.float32).contiguous()
        self.proj = Linear.stacked([weights[f"{pre}.y"], weights[f"{pre}.x"]], runtime)     # columns [y | x]
        self.o = Linear(weights[f"{pre}.o"], runtime)
        self.y_b, self.x_b = f32(f"{pre}.y.b"), f32(f"{pre}.x.b")
        self.conv_w = f32(f"{pre}.conv").t().contiguous()      # [taps, channels]: a tap's weights lie together
        self.conv_b = f32(f"{pre}.conv.b")
        self.r_b, self.i_b = f32(f"{pre}.ra.b").reshape(-1), f32(f"{pre}.ri.b").reshape(-1)
        self.lam = (-DECAY_POWER * F.softplus(f32(f"{pre}.lam"))).contiguous()
        # both gates' matrices of a block below one another, the blocks below one another
        ra, ri = weights[f"{pre}.ra"], weights[f"{pre}.ri"]
        gates = torch.cat([ra, ri.to(ra.dtype)], dim=1)         # [B, 2 bs, bs]
        self.tensor_cores = not runtime.is_f32 and gates.dtype == torch.bfloat16 and self.bs % 8 == 0
        self.pitch = 2 * self.bs
        if self.tensor_cores:
            pad = -self.pitch % K.GROUP_ROW_PAD                 # a tile of the product lies in one block
            gates = F.pad(gates, (0, 0, 0, pad))
            self.pitch += pad
        gates = gates.reshape(self.B * self.pitch, self.bs).contiguous()
        self.gates = K.tile_weight(gates) if self.tensor_cores else gates

    def cache_need(self):
        return None

    def state_shape(self):
        """One float32 row a sequence: S [C], then the convolution's last inputs [taps - 1, C]."""
        return ((self.taps, self.C), torch.float32)

    adds_residual = True      # forward takes `residual` and may add its update to it in place
    takes_factor = True       # ... times `factor`, a number a column of the stream

    def forward(self, y, ctx, entry, residual=None, factor=None):
        store = entry.state()
        u = self.proj(y, split_ok=True)                        # float32 [y | x], possibly partial sums
        conv_state = store[:, 1:] if self.taps > 1 else None
        x = K.conv_silu(u, self.C, self.C, self.conv_w, self.conv_b, conv_state, ctx.tok_seq, ctx.cu_q, ctx.seq_slot,
                        ctx.B, ctx.is_decode, in_bias=self.x_b, silu=False, also_bf16=self.tensor_cores)
        if self.tensor_cores:
            x, x16 = x
            z = K.gemm_tc_blocks(x16, self.gates, self.pitch)
        else:
            z = K.block_product(x, self.gates, self.B)
        v = K.rglru(x, z, self.pitch, self.bs, self.r_b, self.i_b, self.lam, u, 0, self.y_b, store[:, 0], ctx.cu_q,
                    ctx.seq_slot, ctx.B, self.runtime.dtype)
        return self.o(v, split_ok=True, add_to=residual, factor=factor)
