"""The attention mixers: grouped-query causal attention over the cache.

"gqa_attention" (GQAttention) norms each head, "wide_norm_attention" (WideNormAttention)
norms a whole projection at once, has biases, a short convolution over time, a value norm, values of
their own width, a learned sink in the softmax and an output gate,
"head_norm_attention" (HeadNormAttention, at the end of this file) norms each head, has biases,
values of their own width, capped scores, chunks, a sink in the softmax and an output gate; all
hand their queries to `causal_attention`, which picks the kernel.

In order (crates/aegisllm-cuda/src/executor/attention.rs:139-202,241-250,341-352,
413-425; prompt twin executor/prefill/layer.rs:472-636,810-823,967-1047):
q, k, v = y Wq^T, y Wk^T, y Wv^T; optional per-head RMSNorm of q and k with a
weight of head_dim values; rotation of q and k; k, v appended to the cache at the
token's position; for query head h the kv head is h // (heads / kv_heads)
(attention_decode_common.cuh:112-115), scores scaled by `softmax_scale`, a query
at position p sees keys j <= p (and p - j < window if a window is set); o = ctx Wo^T.
Softmax, norms and angles are float32.
"""
from __future__ import annotations

import torch

from ..cache.kv import CacheNeed
from ..ops import kernels as K
from .base import build_part, need, part_tensors, register_part
from .linear import Linear


# Batches of a decode step for which the attention kernel does the rotary kernel's work itself
# (ops.kernels.attn_decode_qkv; the same bits either way). It saves a kernel and its wait on the
# step's path, and costs every block of a sequence's segments the making of its query heads:
# at the 8B shape 2,455 against 2,424 tokens/s at batch 8 and 4,428 against 4,372 at 16, but
# 6,985 against 7,083 at 32 and 10,290 against 10,600 at 64; at batch 1 338 against 340.
FUSED_DECODE_ROWS = (4, 16)


@register_part("mixer", "gqa_attention")
class GQAttention:
    graph_safe = True

    @classmethod
    def tensors(cls, spec):
        p = spec.params
        H, nq, nkv, d = (int(need(p, k, "gqa_attention")) for k in
                         ("hidden_size", "num_heads", "num_kv_heads", "head_dim"))
        t = {f"{spec.prefix}.q_proj.weight": ((nq * d, H), "matrix"),
             f"{spec.prefix}.o_proj.weight": ((H, nq * d), "matrix")}
        if not p.get("shares_cache", False):
            t[f"{spec.prefix}.k_proj.weight"] = ((nkv * d, H), "matrix")
            t[f"{spec.prefix}.v_proj.weight"] = ((nkv * d, H), "matrix")
        if p.get("qk_norm", False):
            t[f"{spec.prefix}.q_norm.weight"] = ((d,), "norm")
            if not p.get("shares_cache", False):
                t[f"{spec.prefix}.k_norm.weight"] = ((d,), "norm")
        t.update(part_tensors("position", p["position"]))
        return t

    def __init__(self, spec, weights, runtime):
        p = spec.params
        self.runtime = runtime
        self.H = int(p["hidden_size"])
        self.nq, self.nkv, self.d = int(p["num_heads"]), int(p["num_kv_heads"]), int(p["head_dim"])
        if self.nq % self.nkv:
            raise ValueError(f"{self.nq} heads are not a multiple of {self.nkv} kv heads")
        if self.d % 16 or self.d > 256:
            raise ValueError(f"head_dim {self.d}: the attention kernels take multiples of 16 up to 256")
        self.window = int(p.get("window", 0) or 0)
        self.scale = float(need(p, "softmax_scale", "gqa_attention"))
        self.shares_cache = bool(p.get("shares_cache", False))
        self.position = build_part("position", p["position"], weights, runtime)
        pre = spec.prefix
        mats = [weights[f"{pre}.q_proj.weight"]]
        if not self.shares_cache:
            mats += [weights[f"{pre}.k_proj.weight"], weights[f"{pre}.v_proj.weight"]]
        self.qkv = Linear.stacked(mats, runtime)
        # a run that reads another run's cache projects queries only
        self.q_only = self.qkv if self.shares_cache else self.qkv.first_rows(self.nq * self.d)
        self.o = Linear(weights[f"{pre}.o_proj.weight"], runtime)
        self.q_norm = self.k_norm = None
        self.qk_eps = float(p.get("qk_norm_eps", 0.0))
        if p.get("qk_norm", False):
            off = float(p.get("qk_norm_weight_offset", 0.0))
            f32 = lambda n: (weights[n].to(device=runtime.device, dtype=torch.float32) + off).contiguous()
            self.q_norm = f32(f"{pre}.q_norm.weight")
            if not self.shares_cache:
                self.k_norm = f32(f"{pre}.k_norm.weight")

    def cache_need(self):
        return CacheNeed(self.nkv, self.d, self.window)

    def state_shape(self):
        return None

    adds_residual = True      # forward takes `residual` and may add its update to it in place

    def forward(self, y, ctx, entry, residual=None):
        kc, vc, table = entry.cache()
        writes = entry.writes_cache and not self.shares_cache
        if (writes and not self.qkv.f32 and entry.layout == K.LAYOUT_SW128 and y.is_contiguous()
                and K.gemm_tc_qkv_takes(y.shape[0], self.qkv.out_features, self.qkv.in_features, self.nq,
                                        self.nkv, self.d, self.position.rotary_dim)):
            # a prompt with heads of 128: norm, rotation and cache write in the product's epilogue
            q = K.gemm_tc_qkv(y, self.qkv.weight, self.q_norm, self.k_norm, self.qk_eps,
                              self.position.angles(ctx), self.position.rotary_dim, ctx.cache_pos,
                              ctx.tok_seq, table, kc, vc, self.nq, self.nkv)
            out = self.attend(q, kc, vc, table, ctx, entry.layout)
            return self.o(out.view(-1, self.nq * self.d), split_ok=True, add_to=residual)
        # float32 [N, (nq + 2 nkv) d], possibly as S partial sums
        qkv = self.qkv(y, split_ok=True) if writes else self.q_only(y, split_ok=True)
        if (writes and ctx.is_decode and FUSED_DECODE_ROWS[0] <= ctx.B <= FUSED_DECODE_ROWS[1]
                and entry.layout == K.LAYOUT_SW128 and self.d == 128
                and self.nq // self.nkv <= 16 and self.position.rotary_dim in (0, 128)
                and kc.dtype == torch.bfloat16):
            # one token a sequence, heads of 128: the attention blocks make their query heads and
            # the new key and value themselves, from the projection's partial sums
            out = K.attn_decode_qkv(qkv, self.q_norm, self.k_norm, self.qk_eps, self.position.angles(ctx),
                                    self.position.rotary_dim, kc, vc, table, ctx.cache_pos, self.window,
                                    self.scale, self.nq, self.nkv)
            return self.o(out.view(-1, self.nq * self.d), split_ok=True, add_to=residual)
        nkv_new = self.nkv if writes else 0
        q = K.qk_norm_rope_store(qkv, self.q_norm, self.k_norm, self.qk_eps,
                                 self.position.angles(ctx), self.position.rotary_dim,
                                 ctx.cache_pos, ctx.tok_seq, table,
                                 kc if nkv_new else None, vc if nkv_new else None,
                                 self.nq, nkv_new, self.d, self.runtime.dtype, layout=entry.layout)
        out = self.attend(q, kc, vc, table, ctx, entry.layout)
        return self.o(out.view(-1, self.nq * self.d), split_ok=True, add_to=residual)

    def attend(self, q, kc, vc, table, ctx, layout):
        return causal_attention(q, kc, vc, table, ctx, layout, layout, self.window, self.scale)


def causal_attention(q, kc, vc, table, ctx, k_layout, v_layout, window, scale, chunk=0, softcap=0.0,
                     sink=False, gate=None, gate_col=0, head_gate=False, keep_first=0, key_dim=None, value_dim=None):
    """Chooses the kernel by the step's shape: the split-KV kernel when every sequence
    brings one token, the flash kernel for prompts, and the general kernel for the
    32-bit path and for head sizes the fast kernels do not take. All agree within rounding.
    q [N, nq, d], as wide as the cache's keys; key_dim and value_dim say how much of keys and values is
    used where the cache's rows are padded. `chunk`, `softcap`, `sink`, `gate` and `keep_first` are the
    options of ops.kernels.attn_generic_opt."""
    nq, d = q.shape[1], q.shape[2]
    nkv, dv = kc.shape[1], vc.shape[3]
    opts = dict(chunk=chunk, softcap=softcap, sink=sink, gate=gate, gate_col=gate_col, head_gate=head_gate,
                keep_first=keep_first, value_dim=value_dim)
    fast = (k_layout == K.LAYOUT_SW128 and v_layout == K.LAYOUT_SW128 and q.dtype == torch.bfloat16
            and max(d, dv) <= K.ATTN_FAST_MAX and nq // nkv <= 16)
    if fast and ctx.is_decode:
        return K.attn_decode(q, kc, vc, table, ctx.cache_pos, window, scale, **opts)
    if fast:
        # a captured step is replayed for other divisions of its tokens than the one it was
        # captured with: the kernel then takes the division from the device alone
        q_lens = None if ctx.extras.get("captured") else ctx.q_lens
        return K.attn_prefill(q, kc, vc, table, ctx.cu_q, ctx.seq_start, q_lens, window, scale, n_seqs=ctx.B,
                              key_dim=key_dim, **opts)
    if chunk or softcap or (sink is not None and sink is not False) or gate is not None or keep_first or value_dim:
        return K.attn_generic_opt(q, kc, vc, table, ctx.tok_seq, ctx.cache_pos, window, scale, layout=k_layout,
                                  v_layout=v_layout, **opts)
    return K.attn_generic(q, kc, vc, table, ctx.tok_seq, ctx.cache_pos, window, scale, layout=k_layout,
                          v_layout=v_layout)


@register_part("mixer", "wide_norm_attention")
class WideNormAttention:
    """q, k, v = y Wq^T + bq, y Wk^T + bk, y Wv^T + bv (biases when `bias`, the default); with `taps` n > 0
    each column then goes through a causal convolution over time (n taps, no bias, the last tap the
    current token's, zeros before a sequence's start); ONE RMS norm over the whole query
    projection (all heads at once, a weight of heads x dim values) and one over the whole key
    projection; then the position part's rotation of the first `rotary_dim` values of every
    query and key head (value i with value i + rotary_dim/2, or 2i with 2i + 1 when
    `interleaved_rotation`); every value head divided by its own root mean square (no weight) and
    cached so when `value_norm`; a query at position p sees key j if 0 <= p - j < window
    (window 0: every earlier key); weights exp(s_j) / (sum exp(s_j) + exp(sink_h)) with s = scale * q . k,
    the last term, one learned number a query head, only when `sink`; query head h reads kv head
    h // (heads / kv_heads); with `output_gate` the heads' outputs are multiplied by sigmoid(y Wg^T)
    element by element; o = ctx Wo^T, without a bias. Keys are `head_dim` wide, values `value_dim`.
    Convolution, norms, angles, scores and weights are float32. A sequence's state is the convolution's
    last taps - 1 inputs. Tensors: `<prefix>.q`, `.k`, `.v` (each with `.b` when `bias` and `.conv`
    [channels, taps] when `taps`), `.q.norm`, `.k.norm`, `.sink` [heads], `.g`, `.o`. Parameters:
    hidden_size, num_heads, num_kv_heads, head_dim, value_dim, softmax_scale, window, norm_eps, position
    (a PartSpec) and the options above."""
    graph_safe = True

    @staticmethod
    def _sizes(p):
        return tuple(int(need(p, k, "wide_norm_attention")) for k in
                     ("hidden_size", "num_heads", "num_kv_heads", "head_dim", "value_dim"))

    @classmethod
    def tensors(cls, spec):
        p = spec.params
        D, H, G, d, dv = cls._sizes(p)
        pre, taps = spec.prefix, int(p.get("taps", 0) or 0)
        t = {f"{pre}.q.norm": ((H * d,), "norm"), f"{pre}.k.norm": ((G * d,), "norm"), f"{pre}.o": ((D, H * dv), "matrix")}
        for n, width in (("q", H * d), ("k", G * d), ("v", G * dv)):
            t[f"{pre}.{n}"] = ((width, D), "matrix")
            if p.get("bias", True):
                t[f"{pre}.{n}.b"] = ((width,), "matrix")
            if taps:
                t[f"{pre}.{n}.conv"] = ((width, taps), "matrix")
        if p.get("sink", False):
            t[f"{pre}.sink"] = ((H,), "matrix")
        if p.get("output_gate", False):
            t[f"{pre}.g"] = ((H * dv, D), "matrix")
        t.update(part_tensors("position", p["position"]))
        return t

    def __init__(self, spec, weights, runtime):
        p = spec.params
        self.runtime = runtime
        _, self.H, self.G, self.d, self.dv = self._sizes(p)
        if self.H % self.G:
            raise ValueError(f"{self.H} heads are not a multiple of {self.G} kv heads")
        if self.d > 512 or self.dv > 512:
            raise ValueError(f"key size {self.d}, value size {self.dv}: the attention kernels take up to 512")
        self.window = int(p.get("window", 0) or 0)
        self.scale = float(need(p, "softmax_scale", "wide_norm_attention"))
        self.eps = float(need(p, "norm_eps", "wide_norm_attention"))
        self.value_norm = bool(p.get("value_norm", False))
        self.interleaved = bool(p.get("interleaved_rotation", False))
        self.position = build_part("position", p["position"], weights, runtime)
        pre = spec.prefix
        f32 = lambda n: weights[n].to(device=runtime.device, dtype=torch.float32).contiguous()
        mats = [weights[f"{pre}.{n}"] for n in "qkv"]
        self.gated = bool(p.get("output_gate", False))
        if self.gated:
            mats.append(weights[f"{pre}.g"])       # the gate reads the same rows: one product for all four
        # `external_projection`: as in HeadNormAttention
        self.input_mats = mats if p.get("external_projection", False) else None
        self.proj = None if self.input_mats is not None else Linear.stacked(mats, runtime)
        self.width = self.H * self.d + self.G * (self.d + self.dv)      # columns of q, k and v; the gate's follow
        self.qkv_bias = torch.cat([f32(f"{pre}.{n}.b") for n in "qkv"]).contiguous() if p.get("bias", True) else None
        self.taps = int(p.get("taps", 0) or 0)
        if self.taps > 16:
            raise ValueError(f"a convolution of {self.taps} taps: this kernel takes 1 to 16")
        # [taps, channels]: a tap's weights lie together
        self.conv_w = torch.cat([f32(f"{pre}.{n}.conv") for n in "qkv"]).t().contiguous() if self.taps else None
        self.q_norm, self.k_norm = f32(f"{pre}.q.norm"), f32(f"{pre}.k.norm")
        self.sink = f32(f"{pre}.sink") if p.get("sink", False) else None
        self.o = Linear(weights[f"{pre}.o"], runtime)

    def cache_need(self):
        return CacheNeed(self.G, self.d, self.window, v_dim=0 if self.dv == self.d else self.dv)

    def state_shape(self):
        """The convolution's last inputs [taps - 1, channels], float32."""
        return ((self.taps - 1, self.width), torch.float32) if self.taps > 1 else None

    adds_residual = True      # forward takes `residual` and may add its update to it in place

    projects_input = True         # may be built with `external_projection` and fed `projected`
    needs_first_columns = True    # its kernels read q, k, v (and the gate) from column 0 of the projection's rows

    def forward(self, y, ctx, entry, residual=None, projected=None, col0=0):
        kc, vc, table = entry.cache()
        if projected is not None and col0 != 0:
            raise ValueError("wide_norm_attention reads its columns from the start of the projection's rows")
        # float32 [q | k | v | gate | ...], possibly partial sums
        u = projected if projected is not None else self.proj(y, split_ok=True)
        rot = self.position.rotary_dim
        conv = None
        if self.taps:
            conv = (self.conv_w, entry.state() if self.taps > 1 else None, ctx.cu_q, ctx.seq_slot, ctx.B, ctx.is_decode)
        q = K.qkv_bias_norm_store(u, self.qkv_bias, self.q_norm, self.k_norm, self.eps, ctx.cache_pos,
                                  ctx.tok_seq, table, kc, vc, self.H, self.G, self.d, self.dv, self.runtime.dtype,
                                  k_layout=entry.layout, v_layout=entry.v_layout,
                                  cs=self.position.angles(ctx) if rot else None, rotary_dim=rot,
                                  value_unit_eps=self.eps if self.value_norm else None, interleaved=self.interleaved,
                                  conv=conv)
        out = causal_attention(q, kc, vc, table, ctx, entry.layout, entry.v_layout, self.window, self.scale,
                               sink=self.sink, gate=u if self.gated else None, gate_col=self.width)
        return self.o(out.view(-1, self.H * self.dv), split_ok=True, add_to=residual)


@register_part("mixer", "head_norm_attention")
class HeadNormAttention:
    """q, k, v = y Wq^T (+ bq), y Wk^T (+ bk), y Wv^T (+ bv); every query head and every key head
    RMS-normed over its `head_dim` values with ONE weight of that size for all heads (plain weight);
    then the position part's rotation of the first `rotary_dim` values of every query and key head
    (value i with value i + rotary_dim/2, or 2i with 2i + 1 when `interleaved_rotation`); with
    `query_temperature` (coef, every) queries times 1 + coef ln(floor((p + 1) / every) + 1) at position p;
    score = softmax_scale * q . k, and with `softcap` c > 0 then c * tanh(score / c); a query at
    position p sees key j <= p, with `chunk` n > 0 only where p // n == j // n, with `window` w > 0
    only where p - j < w or j < `keep_first`; weights exp(s_j) / (sink + sum exp(s_j)) with sink = 1 when `sink` is set
    (a key of score 0 without a value) and 0 otherwise; query head h reads kv head
    h // (heads / kv_heads); with `output_gate` the heads' outputs are multiplied by
    sigmoid(y Wg^T) element by element, with `output_gate` "head" by one number a head (Wg has `heads` rows);
    o = ctx Wo^T without a bias. Keys are `head_dim` wide, values `value_dim`; with `padded_cache` the
    bfloat16 cache keeps both as wide as the next multiple of 64, so that the tensor-core kernels take any
    width up to 256. `qk_norm` "unit": heads are divided by their root mean square without a weight (a
    rotation keeps lengths, so this is the same before it as after it). Norms, angles, scores and weights are float32. Tensors: `<prefix>.q`, `.k`,
    `.v` (each with `.b` when `bias`), `.q.norm`, `.k.norm` (when `qk_norm` is True, the default), `.g`
    (when `output_gate`), `.o`."""
    graph_safe = True

    @staticmethod
    def _sizes(p):
        return tuple(int(need(p, k, "head_norm_attention")) for k in
                     ("hidden_size", "num_heads", "num_kv_heads", "head_dim", "value_dim"))

    @classmethod
    def tensors(cls, spec):
        p = spec.params
        D, H, G, d, dv = cls._sizes(p)
        pre = spec.prefix
        t = {f"{pre}.q": ((H * d, D), "matrix"), f"{pre}.k": ((G * d, D), "matrix"),
             f"{pre}.v": ((G * dv, D), "matrix"), f"{pre}.o": ((D, H * dv), "matrix")}
        if p.get("bias", False):
            t.update({f"{pre}.q.b": ((H * d,), "matrix"), f"{pre}.k.b": ((G * d,), "matrix"),
                      f"{pre}.v.b": ((G * dv,), "matrix")})
        if p.get("qk_norm", True) is True:
            t.update({f"{pre}.q.norm": ((d,), "norm"), f"{pre}.k.norm": ((d,), "norm")})
        if p.get("output_gate", False):
            t[f"{pre}.g"] = ((H if p["output_gate"] == "head" else H * dv, D), "matrix")
        t.update(part_tensors("position", p["position"]))
        return t

    def __init__(self, spec, weights, runtime):
        p = spec.params
        self.runtime = runtime
        _, self.H, self.G, self.d, self.dv = self._sizes(p)
        if self.H % self.G:
            raise ValueError(f"{self.H} heads are not a multiple of {self.G} kv heads")
        if self.d > 512 or self.dv > 512:
            raise ValueError(f"key size {self.d}, value size {self.dv}: the attention kernels take up to 512")
        self.window = int(p.get("window", 0) or 0)
        self.chunk = int(p.get("chunk", 0) or 0)
        self.softcap = float(p.get("softcap", 0.0) or 0.0)
        self.sink = (torch.zeros((self.H,), dtype=torch.float32, device=runtime.device) if p.get("sink", False) else None)
        self.keep_first = int(p.get("keep_first", 0) or 0) if self.window or self.chunk else 0
        self.padded = bool(p.get("padded_cache", False))
        self.interleaved = bool(p.get("interleaved_rotation", False))
        self.temperature = p.get("query_temperature")
        if self.temperature is not None:
            self.temperature = tuple(float(x) for x in self.temperature)
            if len(self.temperature) != 2 or self.temperature[1] <= 0:
                raise ValueError(f"head_norm_attention: query_temperature {self.temperature} is not (coef, every > 0)")
        self.scale = float(need(p, "softmax_scale", "head_norm_attention"))
        self.eps = float(need(p, "norm_eps", "head_norm_attention"))
        self.position = build_part("position", p["position"], weights, runtime)
        pre = spec.prefix
        f32 = lambda n: weights[n].to(device=runtime.device, dtype=torch.float32).contiguous()
        mats = [weights[f"{pre}.q"], weights[f"{pre}.k"], weights[f"{pre}.v"]]
        self.gated, self.head_gate = bool(p.get("output_gate", False)), p.get("output_gate") == "head"
        if self.gated:
            mats.append(weights[f"{pre}.g"])       # the gate reads the same rows: one product for all four
        # `external_projection`: whoever runs this part makes the product (stacked with others that read
        # the same rows) and hands its result to forward; these are the matrices, in the order of the columns
        self.input_mats = mats if p.get("external_projection", False) else None
        self.proj = None if self.input_mats is not None else Linear.stacked(mats, runtime)
        self.bias = (torch.cat([f32(f"{pre}.q.b"), f32(f"{pre}.k.b"), f32(f"{pre}.v.b")]).contiguous()
                     if p.get("bias", False) else None)
        self.q_norm = self.k_norm = None
        qk_norm = p.get("qk_norm", True)
        if qk_norm == "unit":
            self.q_norm = self.k_norm = torch.ones((self.d,), dtype=torch.float32, device=runtime.device)
        elif qk_norm:
            self.q_norm, self.k_norm = f32(f"{pre}.q.norm"), f32(f"{pre}.k.norm")
        self.gate_col = self.H * self.d + self.G * (self.d + self.dv)
        self.o = Linear(weights[f"{pre}.o"], runtime)

    def cache_need(self):
        return CacheNeed(self.G, self.d, self.window, v_dim=0 if self.dv == self.d else self.dv, chunk=self.chunk,
                         keep_first=self.keep_first, padded=self.padded)

    def state_shape(self):
        return None

    adds_residual = True      # forward takes `residual` and may add its update to it in place

    projects_input = True         # may be built with `external_projection` and fed `projected`
    needs_first_columns = True    # its kernels read q, k, v (and the gate) from column 0 of the projection's rows

    def forward(self, y, ctx, entry, residual=None, projected=None, col0=0):
        kc, vc, table = entry.cache()
        if projected is not None and col0 != 0:
            raise ValueError("head_norm_attention reads its columns from the start of the projection's rows")
        # float32 [q | k | v | gate | ...], possibly partial sums
        u = projected if projected is not None else self.proj(y, split_ok=True)
        rot = self.position.rotary_dim
        q = K.qkv_head_norm_store(u, self.bias, self.q_norm, self.k_norm, self.eps,
                                  self.position.angles(ctx) if rot else None, rot, ctx.cache_pos, ctx.tok_seq, table,
                                  kc, vc, self.H, self.G, self.d, self.dv, self.runtime.dtype,
                                  k_layout=entry.layout, v_layout=entry.v_layout, interleaved=self.interleaved,
                                  temperature=self.temperature, positions=ctx.rope_pos)
        out = causal_attention(q, kc, vc, table, ctx, entry.layout, entry.v_layout, self.window, self.scale,
                               chunk=self.chunk, softcap=self.softcap, sink=self.sink,
                               gate=u if self.gated else None, gate_col=self.gate_col, head_gate=self.head_gate,
                               keep_first=self.keep_first, key_dim=self.d,
                               value_dim=self.dv if self.dv != vc.shape[3] else None)
        return self.o(out.view(-1, self.H * self.dv), split_ok=True, add_to=residual)
