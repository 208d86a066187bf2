"""Mefatar in the engine against the plain implementation (tests/plain_mefatar.py): every mechanism
alone, then whole prompts, prompts in portions, decoding token by token, batches of unequal requests,
slots, pages and state that are used again, and greedy generation through the library's entry point."""
import json
import math

import pytest
import torch

import plain_mefatar as P
from mefatar_models import SMALL, config, layer, left, make_weights, parallel, right, unit, write_model

pytestmark = pytest.mark.gpu

F32, BF16 = torch.float32, torch.bfloat16
DTYPES = ["float32", "bfloat16"]


def tol(dtype):
    return 3e-5 if dtype in (F32, "float32") else 3e-2


def close(got, ref, dtype, what=""):
    got, ref = got.detach().float().cpu(), ref.float()
    assert got.shape == ref.shape, (what, got.shape, ref.shape)
    assert torch.isfinite(got).all(), what
    err, scale = float((got - ref).abs().max()), max(1.0, float(ref.abs().max()))
    assert err <= tol(dtype) * scale, f"{what}: {err:.3e} > {tol(dtype) * scale:.3e}"


def runtime(dtype):
    from lumenllm_b200.parts import Runtime
    return Runtime(torch.device("cuda", 0), dtype)


def tokens_of(cfg, lengths, seed):
    g = torch.Generator().manual_seed(seed)
    return [torch.randint(0, cfg["vocab"], (n,), generator=g).tolist() for n in lengths]


def rows(T, D, dtype, seed, std=1.0):
    return (torch.randn(T, D, generator=torch.Generator().manual_seed(seed)) * std).to(dtype).float()


def pieces(y, sizes):
    out, at = [], 0
    for n in sizes:
        out.append(y[at:at + n])
        at += n
    assert at == y.shape[0]
    return out


def total(update, D):
    """An update of the stream, however it is handed on, as one float32 tensor on the host."""
    from lumenllm_b200.ops import kernels as K
    from lumenllm_b200.parts.norm import ShapedUpdate
    if isinstance(update, ShapedUpdate):
        h = torch.zeros(update.groups[0][0].shape[-2], D, device="cuda")
        K.add_shaped_rmsnorm(h, update.groups, None, 0.0, F32)
        return h.cpu()
    return (update.sum(0) if update.dim() == 3 else update).float().cpu()


def mixer_part(m, D, dtype, seed, child=None, edit=None, eps=1e-6):
    """A one-layer model's mixer, built as the engine builds it (`child` 0 or 1: one side of two
    mixers side by side, alone); its weights as the plain implementation reads them."""
    from lumenllm_b200.config import config_from_dict
    from lumenllm_b200.parts import build_part
    cfg = config(8, D, eps, [layer(m)])
    w = make_weights(cfg, seed)
    if edit is not None:
        edit(w)
    spec = config_from_dict(cfg).model_spec().layers[0].mixer
    if child is not None:
        spec = spec.params["parts"][child]["mixer"]
    part = build_part("mixer", spec, {k: v.cuda() for k, v in w.items()}, runtime(dtype))
    return part, {k: v.float() for k, v in w.items()}


def run_mixer(mixer, rt, pieces_by_seq, twice=False):
    """Feeds sequences' rows piece by piece through a mixer alone. pieces_by_seq: for each sequence
    a list of row blocks (an empty block: the sequence pauses that step). With `twice` everything
    runs a second time on the slots, pages and state rows that the first run gave back. Returns
    each sequence's updates in order."""
    from lumenllm_b200.cache import KVCache
    from lumenllm_b200.engine.context import EntryView, StepEntry, build_context
    need, shape = mixer.cache_need(), mixer.state_shape()
    cache = KVCache({0: need} if need is not None else {}, 4096, 4, 4096, dtype=rt.dtype, device=rt.device,
                    state_shapes={0: shape} if shape is not None else None)
    for _ in range(2 if twice else 1):
        slots = [cache.alloc_slot() for _ in pieces_by_seq]
        outs = [[] for _ in pieces_by_seq]
        for step in range(max(len(p) for p in pieces_by_seq)):
            live = [b for b, p in enumerate(pieces_by_seq) if step < len(p) and p[step].shape[0]]
            if not live:
                continue
            ctx, _ = build_context(cache, rt, [StepEntry(slots[b], [0] * pieces_by_seq[b][step].shape[0]) for b in live])
            y = torch.cat([pieces_by_seq[b][step] for b in live]).to(rt.dtype).cuda()
            out = total(mixer.forward(y, ctx, EntryView(ctx, 0, 0 if need is not None else None, True)), y.shape[1])
            at = 0
            for b in live:
                n = pieces_by_seq[b][step].shape[0]
                outs[b].append(out[at:at + n])
                cache.commit(slots[b], n)
                at += n
        for s in slots:
            cache.free_slot(s)
        cache.check()
    return [torch.cat(o) for o in outs]


PORTIONS = {150: [(150,), (64, 64, 22), (2, 2, 61, 1, 84), (1,) * 150], 70: [(70,), (3, 67), (69, 1), (2,) * 35]}


def in_any_portions(part, rt, plain_of, D, dtype, seed, std=1.0):
    """Two sequences of 150 and 70 rows, fed whole, in portions down to two rows and row by row, side
    by side in one batch, twice on the same slots: always the plain implementation's update."""
    ya, yb = rows(150, D, dtype, seed, std), rows(70, D, dtype, seed + 1, std)
    ra, rb = plain_of(ya), plain_of(yb)
    for pa, pb in zip(PORTIONS[150], PORTIONS[70]):
        ga, gb = run_mixer(part, rt, [pieces(ya, pa), pieces(yb, pb)], twice=True)
        close(ga, ra, dtype, f"{pa[:3]}")
        close(gb, rb, dtype, f"{pb[:3]}")


# ------------------------------------------------------------------ kernels alone

@pytest.mark.parametrize("dtype", [F32, BF16])
@pytest.mark.parametrize("width", [64, 50, 1032])
@pytest.mark.parametrize("N", [37, 400])
def test_rms_norm_with_shaped_updates(dtype, width, N):
    """The stream plus groups of partial sums: a factor a column, a norm before the sum, both, neither; the
    norm of the sum; rows gathered; the stream left alone on request; more groups than one launch takes."""
    from lumenllm_b200.ops import kernels as K
    g = torch.Generator().manual_seed(width)
    rn = lambda *s: torch.randn(*s, generator=g)
    h, w = rn(N, width), 1 + 0.1 * rn(width)
    groups = [(rn(3, N, width), 0.5, rn(width), 1 + 0.1 * rn(width), 1e-5), (rn(N, width), -1.25, None, 1 + 0.1 * rn(width), 1e-3),
              (rn(2, N, width), 1.0, rn(width), None, 0.0), (rn(7, N, width), 0.3, None, None, 0.0)]

    def value(d, s, c, nw, eps):
        d = d.sum(0) if d.dim() == 3 else d
        d = P.rms_norm(d, nw, eps) if nw is not None else d
        return s * (d if c is None else c * d)

    x = h + sum(value(*gr) for gr in groups)
    dev = [tuple(v.cuda() if isinstance(v, torch.Tensor) else v for v in gr) for gr in groups]
    hd = h.clone().cuda()
    close(K.add_shaped_rmsnorm(hd, dev, w.cuda(), 1e-6, dtype), P.rms_norm(x, w, 1e-6), dtype, "norm")
    close(hd, x, F32, "stream")
    want = torch.tensor([5, 0, 36, 5], dtype=torch.int32)
    hd = h.clone().cuda()
    y = K.add_shaped_rmsnorm(hd, dev, w.cuda(), 1e-6, dtype, rows=want.cuda(), write_h=False)
    close(y, P.rms_norm(x, w, 1e-6)[want.long()], dtype, "gathered rows")
    assert torch.equal(hd.cpu(), h)
    hd = h.clone().cuda()
    assert K.add_shaped_rmsnorm(hd, dev + dev[:2], None, 0.0, dtype) is None          # six groups, two launches
    close(hd, x + value(*groups[0]) + value(*groups[1]), F32, "adding only")


def test_dynamic_tanh_takes_a_shaped_update():
    """The other norm, behind a layer whose updates have factors a column."""
    from lumenllm_b200.config.spec import PartSpec
    from lumenllm_b200.parts import build_part
    from lumenllm_b200.parts.norm import ShapedUpdate
    g = torch.Generator().manual_seed(3)
    h, d, c = torch.randn(9, 40, generator=g), torch.randn(2, 9, 40, generator=g), torch.randn(40, generator=g)
    w = {"n": torch.ones(40), "n.b": torch.zeros(40), "n.alpha": torch.tensor(0.5)}
    norm = build_part("norm", PartSpec("dynamic_tanh", {"size": 40, "tensor": "n"}), w, runtime(F32))
    y = norm.forward(h.cuda(), ShapedUpdate.of(d.cuda(), c.cuda()), F32)
    close(y, torch.tanh(0.5 * (h + c * d.sum(0))), F32)


@pytest.mark.parametrize("blocks,bs", [(3, 64), (2, 128), (5, 24), (4, 200), (2, 320)])
@pytest.mark.parametrize("N", [1, 9, 100, 300, 2100])
def test_block_diagonal_product(blocks, bs, N):
    """On the tensor cores in every orientation they have (few rows with k split, narrow tiles, two SMs a
    tile), blocks of one, a part of one and several tiles; and in 32-bit."""
    from lumenllm_b200.ops import kernels as K
    g = torch.Generator().manual_seed(blocks * bs)
    x = torch.randn(N, blocks * bs, generator=g)
    w = torch.randn(blocks, 2 * bs, bs, generator=g) * bs ** -0.5
    pad = -2 * bs % K.GROUP_ROW_PAD
    R = 2 * bs + pad
    w16 = torch.nn.functional.pad(w, (0, 0, 0, pad)).to(BF16)
    x16 = x.to(BF16)
    ref = torch.einsum("ngk,grk->ngr", x16.double().view(N, blocks, bs), w16.double())
    got = K.gemm_tc_blocks(x16.cuda(), K.tile_weight(w16.reshape(blocks * R, bs).cuda().contiguous()), R).sum(0)
    close(got, ref.reshape(N, blocks * R), F32, "tensor cores")
    ref = torch.einsum("ngk,grk->ngr", x.double().view(N, blocks, bs), w.double()).reshape(N, -1)
    close(K.block_product(x.cuda(), w.reshape(-1, bs).cuda().contiguous(), blocks), ref, F32, "32-bit")
    K.check_error_flags()


def test_products_with_a_factor_a_column_and_with_gelu():
    from lumenllm_b200.ops import kernels as K
    g = torch.Generator().manual_seed(4)
    M, N, D = 2304, 2320, 192
    x, w = torch.randn(M, D, generator=g).to(BF16), (torch.randn(N, D, generator=g) * D ** -0.5).to(BF16)
    f, h = torch.randn(N, generator=g), torch.randn(M, N, generator=g)
    assert K.gemm_tc_adds(M, N)
    prod = (x.cuda().double() @ w.cuda().double().T).float().cpu()
    hd = h.clone().cuda()
    K.gemm_tc(x.cuda(), K.tile_weight(w.cuda()), add_to=hd, col_scale=f.cuda())
    close(hd, h + f * prod, F32, "added in place")
    for m in (2304, 130, 7):
        for act, fn in (("gelu", P.gelu_tanh), ("silu", P.silu)):
            p = prod[:m].view(m, N // 2, 2)
            ref = fn(p[..., 0]) * p[..., 1]
            got = K.gemm_tc(x[:m].cuda().contiguous(), K.tile_weight(w.cuda()), silu_interleaved=True, act=act)
            close(got, ref, BF16, f"{act} epilogue, {m} rows")
            parts = torch.stack([prod[:m] * 0.25, prod[:m] * 0.75]).cuda()
            close(K.silu_mul(parts, F32, interleaved=True, act=act), ref, F32, f"{act} kernel, {m} rows")
            halves = torch.cat([parts[..., 0::2], parts[..., 1::2]], dim=-1).contiguous()
            close(K.silu_mul(halves, BF16, act=act), ref, BF16, f"{act} kernel, halves, {m} rows")
    K.check_error_flags()


def gla(q, k, v, alpha, S):
    """q, k, alpha [T, H, d], v [T, H, dv] -> (o [T, H, dv], final state)."""
    out = []
    for t in range(q.shape[0]):
        S = alpha[t][:, :, None] * S + k[t][:, :, None] * v[t][:, None, :]
        out.append(torch.einsum("hde,hd->he", S, q[t]))
    return torch.stack(out), S


@pytest.mark.parametrize("per_channel", [True, False])
@pytest.mark.parametrize("H,d,dv,lens", [(2, 8, 40, ([150, 1, 33], [1, 40, 2])), (1, 72, 96, ([130, 70, 40], [3, 1, 1])),
                                         (3, 128, 32, ([600, 520, 700], [512, 600, 530])),
                                         (2, 30, 10, ([540, 700, 513], [2, 1, 4])), (1, 200, 24, ([1300, 1, 513], [1, 1, 1])),
                                         (1, 512, 16, ([600, 512, 600], [1, 2, 1]))])
def test_linear_attention_kernel(H, d, dv, lens, per_channel):
    """Three sequences in one launch, then each again from the state the first launch left: walked token by
    token, from staged runs, and in chunks side by side; a decay a token and channel or a fixed one a head;
    partial sums and one sum; a slot that is not the sequence's index."""
    from lumenllm_b200.ops import kernels as K
    g = torch.Generator().manual_seed(d + dv)
    W = 2 * H * d + H * dv + 8
    fixed = torch.rand(H, generator=g) * 0.2 + 0.8
    for S in (2, 1):
        state = torch.zeros(5, H, d, dv).cuda()
        slots = torch.tensor([3, 0, 4], dtype=torch.int32).cuda()
        plain = [torch.zeros(H, d, dv, dtype=torch.float64) for _ in range(3)]
        for ls in lens:
            u = torch.randn(S, sum(ls), W, generator=g) * 0.6
            al = torch.sigmoid(torch.randn(sum(ls), H * d, generator=g) + 2) ** 0.125 if per_channel else None
            cu = torch.tensor([0] + torch.tensor(ls).cumsum(0).tolist(), dtype=torch.int32).cuda()
            out = K.linear_attn(u.cuda(), 4, 4 + H * d, 4 + 2 * H * d, False, (al if per_channel else fixed).cuda(), state,
                                cu, slots, 3, H, d, dv, o_scale=0.3).cpu()
            x = u.sum(0).double()
            for b, (o, xb) in enumerate(zip(pieces(out, ls), pieces(x, ls))):
                T = xb.shape[0]
                q, k = (xb[:, 4 + i * H * d:4 + (i + 1) * H * d].view(T, H, d) for i in (0, 1))
                v = xb[:, 4 + 2 * H * d:4 + 2 * H * d + H * dv].view(T, H, dv)
                a = pieces(al.double(), ls)[b].view(T, H, d) if per_channel else fixed.double()[None, :, None].expand(T, H, d)
                ref, plain[b] = gla(q, k, v, a, plain[b])
                close(o, 0.3 * ref.reshape(T, H * dv), F32, f"sequence {b} of {T}")
                close(state[int(slots[b])], plain[b], F32, f"state {b}")
        assert float(state[1].abs().max()) == 0.0 and float(state[2].abs().max()) == 0.0


@pytest.mark.parametrize("rank,C,N", [(5, 32, 3), (16, 300, 40), (130, 70, 17), (1, 8, 1)])
def test_decays_of_low_rank(rank, C, N):
    from lumenllm_b200.ops import kernels as K
    g = torch.Generator().manual_seed(rank)
    u, w, b = torch.randn(2, N, rank + 7, generator=g), torch.randn(rank, C, generator=g) * 3, torch.randn(C, generator=g) * 9
    z = (u.sum(0)[:, 3:3 + rank].double() @ w.double() + b.double())
    for tau in (1.0, 16.0):
        ref = torch.exp(torch.nn.functional.logsigmoid(z) / tau)
        close(K.low_rank_decay(u.cuda(), 3, w.cuda(), b.cuda(), tau), ref, F32, f"tau {tau}")


@pytest.mark.parametrize("C,B,pad", [(40, 5, 0), (96, 1, 64), (130, 2, 0), (300, 3, 56)])
def test_recurrent_unit_kernel(C, B, pad):
    """Three sequences in one launch (also of one token and of more than a chunk), then each again from the
    state the first launch left; partial sums; blocks with padding between them."""
    from lumenllm_b200.ops import kernels as K
    g = torch.Generator().manual_seed(C)
    rn = lambda *s: torch.randn(*s, generator=g)
    bs = C // B
    pitch = 2 * bs + pad
    br, bi, by, lam = rn(C), rn(C), rn(C), -8 * torch.nn.functional.softplus(rn(C) * 2 - 3)
    store = torch.zeros(5, 3, C).cuda()
    slots = torch.tensor([3, 0, 4], dtype=torch.int32).cuda()
    S = [torch.zeros(C, dtype=torch.float64) for _ in range(3)]
    for lens in ([150, 1, 64], [1, 2, 1], [65, 129, 2], [3, 1, 9]):
        N = sum(lens)
        u, z, y = rn(N, C), rn(2, N, B * pitch), rn(3, N, C + 5)
        cu = torch.tensor([0] + torch.tensor(lens).cumsum(0).tolist(), dtype=torch.int32).cuda()
        got = K.rglru(u.cuda(), z.cuda(), pitch, bs, br.cuda(), bi.cuda(), lam.cuda(), y.cuda(), 2, by.cuda(), store[:, 1],
                      cu, slots, 3, F32).cpu()
        zs, ys = z.sum(0).double().view(N, B, pitch), y.sum(0).double()[:, 2:2 + C]
        r, i = torch.sigmoid(zs[..., :bs].reshape(N, C) + br), torch.sigmoid(zs[..., bs:2 * bs].reshape(N, C) + bi)
        a = torch.exp(lam.double() * r)
        x = torch.sqrt(1 - a * a) * i * u
        out = P.gelu_tanh(ys + by)
        for b, (t0, t1) in enumerate(zip(cu.tolist(), cu.tolist()[1:])):
            for t in range(t0, t1):
                S[b] = a[t] * S[b] + x[t]
                out[t] *= S[b]
            close(store[int(slots[b]), 1], S[b], F32, f"state {b}")
        close(got, out, F32, f"{lens}")
    assert float(store[:, 0].abs().max()) == 0.0 and float(store[:, 2].abs().max()) == 0.0 and float(store[1].abs().max()) == 0.0


@pytest.mark.parametrize("taps", [1, 2, 3, 4, 6])
def test_convolution_with_an_input_bias(taps):
    """Zeros (not the bias) before the start; no activation; the bfloat16 copy; runs inside a sequence,
    over a border of two, and single tokens."""
    from lumenllm_b200.ops import kernels as K
    g = torch.Generator().manual_seed(taps)
    C, lens = 70, [21, 3, 40]
    w, b, ib = torch.randn(C, taps, generator=g), torch.randn(C, generator=g), torch.randn(C, generator=g)
    state = torch.zeros(4, taps - 1, C).cuda() if taps > 1 else None
    slots = torch.tensor([2, 0, 3], dtype=torch.int32).cuda()
    xs = [torch.randn(n + 30, C, generator=g) for n in lens]
    at, outs = [0, 0, 0], [[], [], []]
    for step in (lens, [1, 1, 1], [2, 1, 5], [1, 1, 1]):
        N = sum(step)
        u = torch.zeros(1, N, C + 9)
        u[0, :, 4:4 + C] = torch.cat([x[a:a + n] for x, a, n in zip(xs, at, step)])
        cu = torch.tensor([0] + torch.tensor(step).cumsum(0).tolist(), dtype=torch.int32).cuda()
        seq = torch.repeat_interleave(torch.arange(3), torch.tensor(step)).int().cuda()
        y, y16 = K.conv_silu(u.cuda(), 4, C, w.t().contiguous().cuda(), b.cuda(), state, seq, cu, slots, 3,
                             step == [1, 1, 1], in_bias=ib.cuda(), silu=False, also_bf16=True)
        assert torch.equal(y16, y.to(BF16))
        for k, o in enumerate(pieces(y.cpu(), step)):
            outs[k].append(o)
            at[k] += step[k]
    for k in range(3):
        ref = P.causal_conv(xs[k][:at[k]] + ib, w, b)
        close(torch.cat(outs[k]), ref, F32, f"sequence {k}")


# ------------------------------------------------------------------ mixers alone

LEFT = [left(4, 2, 16, 24, 0.3, 4, rot=8, base=5000.0, scaling=(4.0, 1.0, 4.0, 64)),
        left(3, 3, 32, 8, 0.25, 2, rot=32, base=500.0),
        left(6, 2, 64, 64, 0.12, 1),
        left(4, 1, 128, 128, 0.09, 3, rot=64, base=1e5, scaling=(16.0, 2.0, 16.0, 128)),
        left(2, 1, 10, 6, 0.4, 6, rot=6)]
RIGHT = [right(2, 16, 24, 8.0, 5), right(1, 72, 96, 2.0, 7), right(3, 128, 32, 16.0, 16), right(5, 8, 40, 1.0, 2)]
UNITS = [unit(40, 5, 2), unit(48, 1, 4), unit(128, 2, 3), unit(30, 3, 1), unit(256, 2, 5)]
ANY_LEFT, ANY_RIGHT = LEFT[1], RIGHT[0]


@pytest.mark.parametrize("dtype", [F32, BF16])
@pytest.mark.parametrize("m", LEFT)
def test_softmax_side_in_any_portions(m, dtype):
    D = 64
    part, w = mixer_part(parallel(m, ANY_RIGHT), D, dtype, seed=11, child=0)
    in_any_portions(part, runtime(dtype),
                    lambda y: P.softmax_attention(y, w, "l0.mix.left", m, 1e-6, torch.arange(y.shape[0])), D, dtype, seed=12)


@pytest.mark.parametrize("dtype", [F32, BF16])
@pytest.mark.parametrize("m", [LEFT[0], LEFT[1], left(4, 2, 32, 16, 0.2, 3, rot=20, base=100.0)])
def test_softmax_side_in_prompts_that_take_several_tokens_a_block(m, dtype):
    """Sequences of 301, 1, 2 and 150 rows in one step, each continued by a prompt of 310, 5, 2 and 1: blocks
    of tokens over the borders of sequences, first tokens that read the state, both sides of every edge."""
    D = 48
    part, w = mixer_part(parallel(m, ANY_RIGHT), D, dtype, seed=41, child=0)
    ys = [rows(n, D, dtype, 42 + n) for n in (611, 6, 4, 151)]
    got = run_mixer(part, runtime(dtype), [pieces(y, c) for y, c in zip(ys, ((301, 310), (1, 5), (2, 2), (150, 1)))], twice=True)
    for y, o in zip(ys, got):
        close(o, P.softmax_attention(y, w, "l0.mix.left", m, 1e-6, torch.arange(y.shape[0])), dtype, f"{y.shape[0]} rows")


@pytest.mark.parametrize("dtype", [F32, BF16])
@pytest.mark.parametrize("m", RIGHT)
def test_linear_side_in_any_portions(m, dtype):
    D = 48
    part, w = mixer_part(parallel(ANY_LEFT, m), D, dtype, seed=13, child=1)
    assert part.cache_need() is None and part.state_shape()[0] == (m["heads"], m["dim"], m["vdim"])
    in_any_portions(part, runtime(dtype), lambda y: P.gated_linear_attention(y, w, "l0.mix.right", m, 1e-6), D, dtype, seed=14)


@pytest.mark.parametrize("dtype", [F32, BF16])
@pytest.mark.parametrize("m", UNITS)
def test_recurrent_unit_in_any_portions(m, dtype):
    D = 48
    part, w = mixer_part(m, D, dtype, seed=15)
    assert part.cache_need() is None and part.state_shape()[0] == (m["conv"], m["width"])
    assert part.tensor_cores == (dtype == BF16 and (m["width"] // m["blocks"]) % 8 == 0)
    in_any_portions(part, runtime(dtype), lambda y: P.recurrent_unit(y, w, "l0.mix", m), D, dtype, seed=16)


@pytest.mark.parametrize("dtype", [F32, BF16])
def test_two_mixers_side_by_side(dtype):
    """One product for both sides, one cache entry, one state row in two pieces, and half the sum of the
    normed updates."""
    D = 64
    m = parallel(LEFT[0], right(5, 7, 9, 4.0, 3))
    part, w = mixer_part(m, D, dtype, seed=17)
    C = 4 * 16 + 2 * (16 + 24)
    assert part.cache_need().n_kv == 2 and part.state_shape()[0] == (3 * C + 5 * 7 * 9 + 1,)       # 315 rounded up to 316
    assert part.proj is not None and part.col0 == [0, C + 4 * 24] and part.mixers[0].proj is None
    in_any_portions(part, runtime(dtype), lambda y: P.side_by_side(y, w, "l0.mix", m, 1e-6, torch.arange(y.shape[0])),
                    D, dtype, seed=18)


@pytest.mark.parametrize("dtype", [F32, BF16])
@pytest.mark.parametrize("size", [16, 64, 128])
def test_sinks_of_every_size(dtype, size):
    """A sink far above every score silences its head, one far below leaves the softmax as it is, one among
    them takes its share; for the general kernel and the tensor-core ones, in prompts and decoded."""
    D, m = 64, left(4, 2, size, size, size ** -0.5, 2, rot=8)

    def edit(w):
        w["l0.mix.left.sink"] = torch.tensor([12.0, -40.0, 0.5, 2.0], dtype=BF16)

    part, w = mixer_part(parallel(m, ANY_RIGHT), D, dtype, seed=19, child=0, edit=edit)
    y = rows(200, D, dtype, 20)
    ref = P.softmax_attention(y, w, "l0.mix.left", m, 1e-6, torch.arange(200))
    other = dict(w, **{"l0.mix.left.sink": torch.full((4,), -40.0)})
    assert float((P.softmax_attention(y, other, "l0.mix.left", m, 1e-6, torch.arange(200)) - ref).abs().max()) > 0.3
    for cut in ((200,), (190,) + (1,) * 10, (1,) * 200):
        (got,) = run_mixer(part, runtime(dtype), [pieces(y, cut)])
        close(got, ref, dtype, f"{cut[:2]}")


FAR = (0, 1, 63, 64, 65, 127, 128, 191, 192, 298)


@pytest.mark.parametrize("decode", [False, True])
@pytest.mark.parametrize("dtype", [F32, BF16])
def test_one_loud_key_far_back_and_at_page_borders(dtype, decode):
    """Key heads made of the query heads' weights with their columns moved on by one, the convolutions
    alike and nearly silent but for the current token, and one earlier row equal to the last row moved the
    same way: that key equals the last query, and its score stands out among 300, wherever it lies, for a
    prompt's last row and for a row decoded alone."""
    D, T = 64, 300
    m = left(4, 2, 32, 16, 1.0, 3, rot=8, base=1e4)

    def edit(w):
        pre = "l0.mix.left."
        q = w[pre + "q"].view(4, 32, D).clone()
        q[1], q[3] = q[0], q[2]                     # the query heads of a group alike, so that every head hears the key
        w[pre + "q"] = q.reshape(128, D)
        w[pre + "k"] = torch.roll(torch.stack([q[0], q[2]]), -1, dims=2).reshape(64, D).clone()
        for n in "qkv":
            w[f"{pre}{n}.conv"] = torch.tensor([0.02, -0.03, 1.0], dtype=BF16).repeat(w[pre + n].shape[0], 1)
        for n in "qk":
            w[f"{pre}{n}.norm"] = torch.ones_like(w[f"{pre}{n}.norm"])
        w[pre + "sink"] = torch.full((4,), 3.0, dtype=BF16)

    part, w = mixer_part(parallel(m, ANY_RIGHT), D, dtype, seed=21, child=0, edit=edit)
    rt = runtime(dtype)
    for j0 in FAR:
        y = rows(T, D, dtype, seed=22 + j0)
        y[j0] = torch.roll(y[T - 1], -1)
        ref = P.softmax_attention(y, w, "l0.mix.left", m, 1e-6, torch.arange(T))
        quiet = y.clone()
        quiet[j0] = -quiet[j0]
        assert float((P.softmax_attention(quiet, w, "l0.mix.left", m, 1e-6, torch.arange(T))[-1] - ref[-1]).abs().max()) > 0.1
        (got,) = run_mixer(part, rt, [pieces(y, (T - 1, 1) if decode else (T,))])
        close(got[-1:], ref[-1:], dtype, f"key {j0}")


@pytest.mark.parametrize("dtype", [F32, BF16])
def test_convolutions_reach_back_over_every_cut(dtype):
    """One loud row at place 100, with taps that differ a lot: the four rows that see it through the
    convolution are right however the sequence is cut around it, for both mixers that convolve."""
    D = 48
    for m, child, plain in ((LEFT[0], 0, lambda y, w: P.softmax_attention(y, w, "l0.mix.left", LEFT[0], 1e-6, torch.arange(len(y)))),
                            (UNITS[1], None, lambda y, w: P.recurrent_unit(y, w, "l0.mix", UNITS[1]))):
        part, w = mixer_part(parallel(m, ANY_RIGHT) if child == 0 else m, D, dtype, seed=23, child=child)
        y = rows(112, D, dtype, seed=24)
        y[100] *= 10
        ref = plain(y, w)
        for cut in ((112,), (100, 12), (101, 11), (101, 1, 10), (102, 2, 8), (103, 9), (100,) + (1,) * 12):
            (got,) = run_mixer(part, runtime(dtype), [pieces(y, cut)])
            close(got[99:], ref[99:], dtype, f"{cut[:3]}")


@pytest.mark.parametrize("dtype", [F32, BF16])
def test_states_remember_far_back_and_forget_by_channel(dtype):
    """A loud first token, then 400 quiet ones fed in portions: what decays slowly still carries it at the
    end (the plain result without it is far off), what decays fast has lost it."""
    D, T = 48, 401
    m = right(2, 16, 8, 16.0, 4)

    def slow(w):
        w["l0.mix.right.a2.b"] = torch.cat([torch.full((16,), 12.0), torch.full((16,), -3.0)]).to(BF16)

    def lasting(w):
        w["l0.mix.lam"] = torch.cat([torch.full((40,), -8.0), torch.full((8,), 2.0)]).to(BF16)

    y = rows(T, D, dtype, seed=26, std=0.5)
    y[0] = (y[0] * 40).to(dtype).float()
    quiet = y.clone()
    quiet[0] = 0.0
    for part, w, plain in (mixer_part(parallel(ANY_LEFT, m), D, dtype, seed=25, child=1, edit=slow)
                           + (lambda x, w: P.gated_linear_attention(x, w, "l0.mix.right", m, 1e-6),),
                           mixer_part(UNITS[1], D, dtype, seed=25, edit=lasting)
                           + (lambda x, w: P.recurrent_unit(x, w, "l0.mix", UNITS[1]),)):
        ref = plain(y, w)
        assert float((plain(quiet, w)[-1] - ref[-1]).abs().max()) > 0.05
        (got,) = run_mixer(part, runtime(dtype), [pieces(y, (1, 199, 2, 198, 1))])
        close(got, ref, dtype)


@pytest.mark.parametrize("dtype", [F32, BF16])
@pytest.mark.parametrize("N", [1, 9, 150, 600])
def test_feed_forward(dtype, N):
    from lumenllm_b200.config import config_from_dict
    from lumenllm_b200.parts import build_part
    D = 64
    cfg = config(8, D, 1e-6, [layer(UNITS[0], 88)])
    w = make_weights(cfg, seed=27)
    part = build_part("ffn", config_from_dict(cfg).model_spec().layers[0].ffn, {k: v.cuda() for k, v in w.items()}, runtime(dtype))
    y = rows(N, D, dtype, seed=28)
    close(total(part.forward(y.to(dtype).cuda(), None), D), P.gated_ff(y, {k: v.float() for k, v in w.items()}, "l0.mlp"), dtype)


# ------------------------------------------------------------------ the model in the engine

@pytest.fixture(scope="module")
def models(tmp_path_factory):
    root = tmp_path_factory.mktemp("mefatar")
    return {name: write_model(cfg, root / name, seed=3 + i) for i, (name, cfg) in enumerate(SMALL.items())}


@pytest.fixture(scope="module")
def plain(models):
    return {name: P.load_model(folder) + ({},) for name, folder in models.items()}


def plain_logits(plain, name, tokens):
    cfg, w, memo = plain[name]
    key = tuple(tokens)
    if key not in memo:
        memo[key] = P.forward(cfg, w, tokens)
    return memo[key]


def engine_of(models, name, dtype, **kw):
    from lumenllm_b200.engine import Engine
    kw.setdefault("max_tokens", 2048)
    return Engine.from_folder(models[name], dtype=dtype, **kw)


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("name", list(SMALL))
def test_whole_prompts(name, dtype, models, plain):
    from lumenllm_b200.engine import StepEntry
    eng = engine_of(models, name, dtype)
    for toks in tokens_of(SMALL[name], (1, 2, 65, 200), seed=30):
        slot = eng.alloc_slot()
        close(eng.step([StepEntry(slot, toks, list(range(len(toks))))]), plain_logits(plain, name, toks), dtype, f"{len(toks)} tokens")
        eng.free_slot(slot)
    eng.cache.check()
    eng.check_kernels()


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("name", list(SMALL))
def test_residual_stream_after_every_layer_run(name, dtype, models, plain):
    from lumenllm_b200.engine import StepEntry
    from lumenllm_b200.engine.context import EntryView
    from lumenllm_b200.ops import kernels as K
    cfg, w, _ = plain[name]
    toks = tokens_of(cfg, (40,), seed=31)[0]
    ref = []
    P.forward(cfg, w, toks, ref)
    eng = engine_of(models, name, dtype)
    ctx = eng.build_context([StepEntry(eng.alloc_slot(), toks, [])])
    m = eng.model
    assert len(m.schedule) == len(ref)
    h, pending = m.embedding.forward(ctx.tokens, ctx), None
    for i, e in enumerate(m.schedule):
        h, pending = m.blocks[e.layer].forward(h, pending, ctx, EntryView(ctx, i, i if i in ctx.cache.group_of else None, True))
        x = h.clone()
        if pending is not None:
            K.add_shaped_rmsnorm(x, pending.groups, None, 0.0, F32)
        close(x, ref[i], dtype, f"after run {i} (layer {e.layer})")


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("name", list(SMALL))
def test_prompt_in_portions_and_decoded_token_by_token(name, dtype, models, plain):
    from lumenllm_b200.engine import StepEntry
    toks = tokens_of(SMALL[name], (171,), seed=32)[0]
    ref = plain_logits(plain, name, toks)
    eng = engine_of(models, name, dtype, max_slots=2)
    for cuts in ((64, 2, 62, 3), (1, 127), (130,)):
        slot = eng.alloc_slot()
        got, at = [], 0
        for n in cuts:
            got.append(eng.step([StepEntry(slot, toks[at:at + n], list(range(n)))]))
            at += n
        got += [eng.step([StepEntry(slot, [toks[t]], [0])]) for t in range(at, len(toks))]
        close(torch.cat(got), ref, dtype, f"{cuts}")
        eng.free_slot(slot)
    eng.cache.check()
    eng.check_kernels()


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("name", list(SMALL))
def test_a_batch_of_unequal_requests_equals_each_alone(name, dtype, models, plain):
    """Prompts of 1, 2, 64, 65 and 131 tokens in one batch, decoded together while the shorter ones
    end; then the slots, pages and state rows they gave back serve the same requests in another order."""
    from lumenllm_b200.engine import StepEntry
    lens = (65, 1, 131, 2, 64)
    prompts = tokens_of(SMALL[name], [n + k for k, n in enumerate(lens)], seed=33)      # request k decodes k tokens
    refs = [plain_logits(plain, name, p) for p in prompts]
    eng = engine_of(models, name, dtype, max_slots=5)
    for order in ((0, 1, 2, 3, 4), (4, 2, 0, 3, 1)):
        slots = {k: eng.alloc_slot() for k in order}
        got = eng.step([StepEntry(slots[k], prompts[k][:lens[k]], list(range(lens[k]))) for k in order])
        close(got, torch.cat([refs[k][:lens[k]] for k in order]), dtype, "prompts")
        for t in range(4):
            live = [k for k in order if k > t]
            got = eng.step([StepEntry(slots[k], [prompts[k][lens[k] + t]], [0]) for k in live])
            close(got, torch.stack([refs[k][lens[k] + t] for k in live]), dtype, f"decoded {t}")
            for k in order:
                if k == t + 1:
                    eng.free_slot(slots[k])
        eng.free_slot(slots[0])
        eng.cache.check()
    eng.check_kernels()


@pytest.mark.parametrize("dtype", DTYPES)
def test_long_decoding_over_page_borders(dtype, models, plain):
    from lumenllm_b200.cache import PAGE
    from lumenllm_b200.engine import StepEntry
    toks = tokens_of(SMALL["Z"], (3 * PAGE + 20,), seed=34)[0]
    ref = plain_logits(plain, "Z", toks)
    eng = engine_of(models, "Z", dtype, max_tokens=6 * PAGE, max_slots=2)
    slot = eng.alloc_slot()
    got = [eng.step([StepEntry(slot, toks[:5], list(range(5)))])]
    got += [eng.step([StepEntry(slot, [toks[t]], [0])]) for t in range(5, len(toks))]
    close(torch.cat(got), ref, dtype)
    eng.free_slot(slot)
    eng.cache.check()
    eng.check_kernels()


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("width", [44, 50])
def test_a_model_whose_rows_are_no_multiples_of_16_bytes(dtype, width, tmp_path):
    """Widths 44 and 50, heads of 6 keys and 10 values, a recurrence of 7 key channels, units of 30 channels
    in blocks of 10: no row of any matrix is a multiple of 16 bytes, so the products and the row kernels go
    the ways that need no alignment."""
    from lumenllm_b200.engine import Engine, StepEntry
    cfg = config(61, width, 1e-5, [
        layer(parallel(left(3, 1, 6, 10, 0.4, 4, rot=4, scaling=(2.0, 1.0, 3.0, 32)), right(2, 7, 5, 3.0, 3)), 9),
        layer(unit(30, 3, 3)), layer(unit(22, 1, 2), 13)], loop=(1, 3, 2))
    folder = write_model(cfg, tmp_path / "m", seed=90)
    _, w = P.load_model(folder)
    toks = tokens_of(cfg, (390,), seed=91)[0]
    ref = P.forward(cfg, w, toks)
    eng = Engine.from_folder(folder, dtype=dtype, max_tokens=1024, max_slots=2)
    slot = eng.alloc_slot()
    got = [eng.step([StepEntry(slot, toks[:370], list(range(370)))])]
    got += [eng.step([StepEntry(slot, [toks[t]], [0])]) for t in range(370, 390)]
    close(torch.cat(got), ref, dtype)
    eng.check_kernels()


def test_a_long_wide_prompt(tmp_path):
    """A prompt long and wide enough for the tensor-core kernels of every product (the output products with
    factors a column add into the stream by themselves), of the softmax side (keys and values of 128), of
    the block-diagonal product on pairs of SMs, and for the chunks of both recurrences."""
    from lumenllm_b200.engine import Engine, StepEntry
    cfg = config(64, 1024, 1e-6, [
        layer(parallel(left(4, 2, 128, 128, 0.09, 4, rot=64, scaling=(6.0, 1.0, 4.0, 512)), right(4, 64, 64, 16.0, 16)), 512),
        layer(unit(1536, 6, 4), 640)], loop=(0, 2, 2))
    T = 2300
    folder = write_model(cfg, tmp_path / "wide", seed=70)
    toks = tokens_of(cfg, (T,), seed=71)[0]
    want = [0, 1, 63, 64, 255, 256, 1023, 1024, 2047, 2048, T - 2, T - 1]
    _, w = P.load_model(folder)
    ref = P.forward(cfg, w, toks)[want]
    eng = Engine.from_folder(folder, dtype="bfloat16", max_tokens=4096)
    slot = eng.alloc_slot()
    close(eng.step([StepEntry(slot, toks, want)]), ref, "bfloat16")
    eng.check_kernels()


@pytest.mark.parametrize("dtype", DTYPES)
def test_greedy_generation_through_the_entry_point(dtype, models, plain):
    """build(EngineConfig).generate: batches, the scheduler's run-ahead and captured steps."""
    from lumenllm_b200 import EngineConfig, GenerateRequest, build
    name = "Z"
    cfg, w, _ = plain[name]
    built = build(EngineConfig(model_path=str(models[name]), dtype=dtype, context_size=512, max_batch=3))
    assert built.engine.model.graph_safe
    prompts = tokens_of(cfg, (70, 3, 29, 130), seed=40)
    outs = built.generate([GenerateRequest(p, 10) for p in prompts], eos_token_ids=[])
    for p, o in zip(prompts, outs):
        assert o.finish_reason == "length" and len(o.tokens) == 10
        lg = P.forward(cfg, w, list(p) + o.tokens)
        for k, tok in enumerate(o.tokens):
            row = lg[len(p) - 1 + k]
            gap = float(row.max() - row[tok])     # 0 where the plain choice was made
            assert gap <= (1e-4 if dtype == "float32" else 0.05 * max(1.0, float(row.abs().max()))), (k, gap)
        if dtype == "float32":
            assert o.tokens == P.greedy(cfg, w, p, 10)
    built.engine.check_kernels()


def test_command_line_generates(models, capsys):
    from lumenllm_b200.cli import main
    rc = main(["generate", "--model", str(models["X"]), "--prompt-tokens", "5,6,7", "--prompt-tokens", "1",
               "--max-tokens", "4", "--ctx-size", "128", "--format", "json", "--dtype", "float32"])
    assert rc == 0
    outs = json.loads(capsys.readouterr().out.strip().splitlines()[-1])
    cfg, w = P.load_model(models["X"])
    assert [o["tokens"] for o in outs] == [P.greedy(cfg, w, p, 4) for p in ([5, 6, 7], [1])]


def test_random_weights_mode_builds_and_steps():
    """A configuration alone is enough for an engine with random weights (the throughput runs use it)."""
    from lumenllm_b200.engine import Engine, StepEntry
    eng = Engine.from_random(SMALL["Z"], seed=1, std=0.05, max_tokens=512)
    slot = eng.alloc_slot()
    lg = eng.step([StepEntry(slot, list(range(40)), [39])])
    assert lg.shape == (1, SMALL["Z"]["vocab"]) and torch.isfinite(lg).all()
    eng.check_kernels()


def test_trace_replay_writes_the_wanted_logits(models, plain, tmp_path):
    """bin/trace_run as a user starts it: a batch of two prompts, decoded together, one request
    ending early; the files hold the plain logits at the wanted places."""
    import subprocess
    import sys
    from pathlib import Path
    import numpy as np
    name = "X"
    cfg = SMALL[name]
    a, b = tokens_of(cfg, (40, 9), seed=50)
    steps = [{"step": 0, "entries": [{"id": "a", "tokens": a[:30], "want": [0, 29]},
                                     {"id": "b", "tokens": b[:8], "want": [7]}], "end": []},
             {"step": 1, "entries": [{"id": "a", "tokens": [a[30]], "want": []},
                                     {"id": "b", "tokens": [b[8]], "want": [0]}], "end": ["b"]}]
    steps += [{"step": 2 + t, "entries": [{"id": "a", "tokens": [a[31 + t]], "want": [0]}],
               "end": ["a"] if t == 8 else []} for t in range(9)]
    runner = Path(__file__).resolve().parent.parent / "bin" / "trace_run"
    out = tmp_path / "out"
    done = subprocess.run([sys.executable, str(runner), "--model", str(models[name]), "--dtype", "float32",
                           "--out", str(out), "--max-tokens", "128"],
                          input="".join(json.dumps(s) + "\n" for s in steps), capture_output=True, text=True, timeout=600)
    assert done.returncode == 0, done.stderr[-2000:]
    assert [l for l in done.stdout.splitlines() if l.startswith("done ")] == [f"done {s['step']}" for s in steps]
    ra, rb = plain_logits(plain, name, a), plain_logits(plain, name, b)
    read = lambda s: torch.from_numpy(np.fromfile(out / f"{s}.f32", dtype="<f4").reshape(-1, cfg["vocab"]).copy())
    close(read(0), torch.stack([ra[0], ra[29], rb[7]]), F32, "prompts")
    close(read(1), rb[8:9], F32, "the short request's last token")
    for t in range(9):
        close(read(2 + t), ra[31 + t:32 + t], F32, f"decoded {t}")
