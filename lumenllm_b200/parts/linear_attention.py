"""Linear attention with decay: a recurrence over time with a matrix state per head, in place of a
softmax over cached keys. "decay_linear_attention" has a fixed decay a head, "gated_linear_attention"
(at the end of this file) a decay that every token brings for every key channel.

In order, for H heads with keys of d and values of dv channels: q = act(y Wq^T), k = act(y Wk^T)
(H d wide), v = act(y Wv^T) (H dv wide), act = SiLU (`activation` "silu") or nothing ("none"); per
head S <- decay_h S + k v^T, o = S^T q (S is d x dv; o sees the token's own write; no other
scale); the heads' o side by side are divided by their root mean square over all H dv channels,
times the weight `.norm` (H dv values), times sigmoid(y Wg^T) when `output_gate`; out = that Wo^T.
`decay` is one number a head, from the configuration.

A sequence's state is S of every head (float32, kept [H, d, dv]); it starts at zero and is carried
from step to step, so a sequence may be fed in any portions. Activations, state, sums, norm and
gate are float32; the projections run in the run's type, and the ones that read y are one product.
"""
from __future__ import annotations

import torch

from ..ops import kernels as K
from .base import need, register_part
from .linear import Linear


@register_part("mixer", "decay_linear_attention")
class DecayLinearAttention:
    graph_safe = True

    @staticmethod
    def _sizes(p):
        return tuple(int(need(p, k, "decay_linear_attention")) for k in ("hidden_size", "num_heads", "head_dim", "value_dim"))

    @classmethod
    def tensors(cls, spec):
        D, H, d, dv = cls._sizes(spec.params)
        pre = spec.prefix
        t = {f"{pre}.q": ((H * d, D), "matrix"), f"{pre}.k": ((H * d, D), "matrix"), f"{pre}.v": ((H * dv, D), "matrix"),
             f"{pre}.norm": ((H * dv,), "norm"), f"{pre}.o": ((D, H * dv), "matrix")}
        if spec.params.get("output_gate", True):
            t[f"{pre}.g"] = ((H * dv, D), "matrix")
        return t

    def __init__(self, spec, weights, runtime):
        p = spec.params
        self.runtime = runtime
        self.D, self.H, self.d, self.dv = self._sizes(p)
        if self.d > K.linear_attn_max_dim():
            raise ValueError(f"key size {self.d}: the recurrence takes up to {K.linear_attn_max_dim()}")
        decay = [float(x) for x in need(p, "decay", "decay_linear_attention")]
        if len(decay) != self.H:
            raise ValueError(f"{len(decay)} decays for {self.H} heads")
        act = p.get("activation", "silu")
        if act not in ("silu", "none"):
            raise ValueError(f"decay_linear_attention: activation {act!r} (known: 'silu', 'none')")
        self.silu = act == "silu"
        self.eps = float(need(p, "norm_eps", "decay_linear_attention"))
        self.gated = bool(p.get("output_gate", True))
        pre = spec.prefix
        f32 = lambda n: weights[n].to(device=runtime.device, dtype=torch.float32).contiguous()
        self.decay = torch.tensor(decay, dtype=torch.float32, device=runtime.device)
        mats = [weights[f"{pre}.{n}"] for n in ("q", "k", "v") + (("g",) if self.gated else ())]
        # `external_projection`: whoever runs this part makes the product (stacked with others that read
        # the same rows) and hands its result, and the column where this part's begin, to forward
        self.input_mats = mats if p.get("external_projection", False) else None
        self.proj = None if self.input_mats is not None else Linear.stacked(mats, runtime)
        self.norm_w = f32(f"{pre}.norm")
        self.o = Linear(weights[f"{pre}.o"], runtime)
        self.k_col, self.v_col = self.H * self.d, 2 * self.H * self.d
        self.g_col = self.v_col + self.H * self.dv

    def cache_need(self):
        return None

    def state_shape(self):
        """The heads' states [H, d, dv], float32."""
        return ((self.H, self.d, self.dv), torch.float32)

    adds_residual = True      # forward takes `residual` and may add its update to it in place

    projects_input = True         # may be built with `external_projection` and fed `projected`

    def forward(self, y, ctx, entry, residual=None, projected=None, col0=0):
        S = entry.state()
        # float32 [... | q | k | v | g | ...] from column col0, possibly partial sums
        u = projected if projected is not None else self.proj(y, split_ok=True)
        o = K.linear_attn(u, col0, col0 + self.k_col, col0 + self.v_col, self.silu, self.decay, S, ctx.cu_q, ctx.seq_slot,
                          ctx.B, self.H, self.d, self.dv)
        dt = self.runtime.dtype
        v = K.cols_rmsnorm(o, 0, self.H * self.dv, self.norm_w, self.eps, dt, gate=u if self.gated else None,
                           gate_col=col0 + self.g_col)
        return self.o(v, split_ok=True, add_to=residual)


@register_part("mixer", "gated_linear_attention")
class GatedLinearAttention:
    """In order, for H heads with keys of d and values of dv channels: q = y Wq^T d^-1/2, k = y Wk^T (H d
    wide), v = y Wv^T (H dv wide); a decay for every key channel, alpha = sigmoid(z)^(1/tau) with
    z = Wa2 (Wa1 y) + b (a product of rank `decay_rank`); per head S <- diag(alpha) S + k v^T, o = S^T q
    (S is d x dv; the decay acts on the rows of the key channels; o sees the token's own write); every
    head's o is divided by its root mean square over dv, times the weight `.norm` (dv values, one for all
    heads), and all heads are multiplied by silu(y Wg^T); out = that Wo^T.

    A sequence's state is S of every head (float32, kept [H, d, dv]); it starts at zero and is carried
    from step to step. Decays (their product of low rank included), state, sums, norm and gate are
    float32; the projections run in the run's type, and the ones that read y are one product."""
    graph_safe = True

    @staticmethod
    def _sizes(p):
        return tuple(int(need(p, k, "gated_linear_attention")) for k in
                     ("hidden_size", "num_heads", "head_dim", "value_dim", "decay_rank"))

    @classmethod
    def tensors(cls, spec):
        D, H, d, dv, r = cls._sizes(spec.params)
        pre = spec.prefix
        return {f"{pre}.q": ((H * d, D), "matrix"), f"{pre}.k": ((H * d, D), "matrix"), f"{pre}.v": ((H * dv, D), "matrix"),
                f"{pre}.g": ((H * dv, D), "matrix"), f"{pre}.a1": ((r, D), "matrix"), f"{pre}.a2": ((H * d, r), "matrix"),
                f"{pre}.a2.b": ((H * d,), "matrix"), f"{pre}.norm": ((dv,), "norm"), f"{pre}.o": ((D, H * dv), "matrix")}

    def __init__(self, spec, weights, runtime):
        p = spec.params
        self.runtime = runtime
        self.D, self.H, self.d, self.dv, self.rank = self._sizes(p)
        if self.d > K.linear_attn_max_dim():
            raise ValueError(f"key size {self.d}: the recurrence takes up to {K.linear_attn_max_dim()}")
        self.tau = float(need(p, "tau", "gated_linear_attention"))
        self.eps = float(need(p, "norm_eps", "gated_linear_attention"))
        pre = spec.prefix
        f32 = lambda n: weights[n].to(device=runtime.device, dtype=torch.float32).contiguous()
        mats = [weights[f"{pre}.{n}"] for n in ("q", "k", "v", "g", "a1")]
        self.input_mats = mats if p.get("external_projection", False) else None    # as in DecayLinearAttention
        self.proj = None if self.input_mats is not None else Linear.stacked(mats, runtime)
        self.a2 = f32(f"{pre}.a2").t().contiguous()             # [rank, H d]: a rank's numbers lie together
        self.a2_b, self.norm_w = f32(f"{pre}.a2.b"), f32(f"{pre}.norm")
        self.o = Linear(weights[f"{pre}.o"], runtime)
        self.k_col, self.v_col = self.H * self.d, 2 * self.H * self.d
        self.g_col = self.v_col + self.H * self.dv
        self.a_col = self.g_col + self.H * self.dv

    def cache_need(self):
        return None

    def state_shape(self):
        """The heads' states [H, d, dv], float32."""
        return ((self.H, self.d, self.dv), torch.float32)

    adds_residual = True      # forward takes `residual` and may add its update to it in place

    projects_input = True         # may be built with `external_projection` and fed `projected`

    def forward(self, y, ctx, entry, residual=None, projected=None, col0=0):
        # float32 [... | q | k | v | g | a1 | ...] from column col0, possibly partial sums
        u = projected if projected is not None else self.proj(y, split_ok=True)
        alpha = K.low_rank_decay(u, col0 + self.a_col, self.a2, self.a2_b, self.tau)
        o = K.linear_attn(u, col0, col0 + self.k_col, col0 + self.v_col, False, alpha, entry.state(), ctx.cu_q,
                          ctx.seq_slot, ctx.B, self.H, self.d, self.dv, o_scale=self.d ** -0.5)
        v = K.head_norm_gate(o, self.norm_w, self.eps, u, col0 + self.g_col, self.H, self.runtime.dtype, silu=True)
        return self.o(v, split_ok=True, add_to=residual)
