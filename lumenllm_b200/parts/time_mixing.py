"""Time mixing ("time_mixing", RWKV-style): a recurrence over time with a matrix state per head whose
inputs each read a mix of the token's row and the row before it.

In order, for H heads of d channels, y' the row of the token before (zeros before a sequence's first):
every s of r, k, v, g, w reads x_s = y + (y' - y) mu_s; r, k, v = x_r Wr^T, x_k Wk^T, x_v Wv^T (H d wide),
gate = silu(x_g Wg^T); a decay for every key channel, w = exp(-exp(tanh(x_w W1^T) W2^T + w0)); per head
o = (S + diag(u) k v^T)^T r, then S <- diag(w) S + k v^T (S is d x d; a token's own value counts with the
bonus u instead of through the state); every head's o divided by its root mean square, all heads times
the weight `.norm` (H d values) times the gate; out = that Wo^T. Tensors: `<prefix>.mu.r` .. `.mu.w` [D],
`.r`, `.k`, `.v`, `.g` [H d, D], `.w1` [rank, D], `.w2` [H d, rank], `.w0` [H d], `.u` [H, d], `.norm` [H d],
`.o` [D, H d].

A sequence's state is one float32 row: y of its last token, then S of every head ([H, d, d]); it starts at
zero and is carried from step to step, so a sequence may be fed in any portions. Decays (the product with
W2 included), bonus, state, sums and norm are float32. The five products that read the mixes are one
block-diagonal product (block s reads x_s) with float32 sums: on the tensor cores in a bfloat16 run.
"""
from __future__ import annotations

import torch
import torch.nn.functional as F

from ..ops import kernels as K
from .base import need, register_part
from .linear import Linear

SOURCES = ("r", "k", "v", "g", "w")


@register_part("mixer", "time_mixing")
class TimeMixing:
    """Parameters: hidden_size, num_heads, head_dim, decay_rank, norm_eps."""
    graph_safe = True

    @staticmethod
    def _sizes(p):
        return tuple(int(need(p, k, "time_mixing")) for k in ("hidden_size", "num_heads", "head_dim", "decay_rank"))

    @classmethod
    def tensors(cls, spec):
        D, H, d, rank = cls._sizes(spec.params)
        pre, C = spec.prefix, H * d
        t = {f"{pre}.mu.{s}": ((D,), "matrix") for s in SOURCES}
        t.update({f"{pre}.{s}": ((C, D), "matrix") for s in "rkvg"})
        t.update({f"{pre}.w1": ((rank, D), "matrix"), f"{pre}.w2": ((C, rank), "matrix"), f"{pre}.w0": ((C,), "matrix"),
                  f"{pre}.u": ((H, d), "matrix"), f"{pre}.norm": ((C,), "norm"), f"{pre}.o": ((D, C), "matrix")})
        return t

    def __init__(self, spec, weights, runtime):
        self.runtime = runtime
        self.D, self.H, self.d, self.rank = self._sizes(spec.params)
        if self.d > K.linear_attn_max_dim():
            raise ValueError(f"head size {self.d}: the recurrence takes up to {K.linear_attn_max_dim()}")
        self.eps = float(need(spec.params, "norm_eps", "time_mixing"))
        pre = spec.prefix
        f32 = lambda n: weights[n].to(device=runtime.device, dtype=torch.float32).contiguous()
        self.mu = torch.stack([f32(f"{pre}.mu.{s}") for s in SOURCES]).contiguous()
        mats = [weights[f"{pre}.{s}"] for s in "rkvg"] + [weights[f"{pre}.w1"]]
        self.tensor_cores = not runtime.is_f32 and all(m.dtype == torch.bfloat16 for m in mats) and self.D % 8 == 0
        # rows of a block: all alike, the last one (the decays' first product) shorter on the tensor cores
        self.pitch = max(self.H * self.d, self.rank)
        if self.tensor_cores:
            self.pitch += -self.pitch % K.GROUP_ROW_PAD         # a tile of the product lies in one block
        rows = [self.pitch] * 4 + [self.rank + -self.rank % 64 if self.tensor_cores else self.pitch]
        dt = torch.bfloat16 if all(m.dtype == torch.bfloat16 for m in mats) else torch.float32
        w = torch.cat([F.pad(m.to(dt), (0, 0, 0, n - m.shape[0])) for m, n in zip(mats, rows)]).contiguous()
        self.proj = K.tile_weight(w) if self.tensor_cores else w
        self.w2 = f32(f"{pre}.w2").t().contiguous()             # [rank, H d]: a rank's numbers lie together
        self.w0, self.u, self.norm_w = f32(f"{pre}.w0"), f32(f"{pre}.u"), f32(f"{pre}.norm")
        self.o = Linear(weights[f"{pre}.o"], runtime)
        self.state_at = self.D + -self.D % 4                    # S begins on 16 bytes

    def cache_need(self):
        return None

    def state_shape(self):
        return ((self.state_at + self.H * self.d * self.d,), torch.float32)

    adds_residual = True      # forward takes `residual` and may add its update to it in place

    def forward(self, y, ctx, entry, residual=None):
        store = entry.state()
        x = K.shift_mix(y, self.mu, store[:, :self.D], ctx.tok_seq, ctx.cu_q, ctx.seq_slot)
        # float32 [r | k | v | g | w1], a block's columns `pitch` apart, possibly partial sums
        if self.tensor_cores:
            u = K.gemm_tc_blocks(x, self.proj, self.pitch)
        else:
            u = K.block_product(x.float(), self.proj, len(SOURCES))
        P = self.pitch
        decay, bonus = K.low_rank_decay(u, 4 * P, self.w2, self.w0, twice=True, bonus=(self.u, 0, P))
        S = store[:, self.state_at:].unflatten(1, (self.H, self.d, self.d))
        o = K.linear_attn(u, 0, P, 2 * P, False, decay, S, ctx.cu_q, ctx.seq_slot, ctx.B, self.H, self.d, self.d, bonus=bonus)
        v = K.head_norm_gate(o, self.norm_w, self.eps, u, 3 * P, self.H, self.runtime.dtype, silu=True)
        return self.o(v, split_ok=True, add_to=residual)
