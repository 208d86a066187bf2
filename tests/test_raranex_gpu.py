"""Raranex in the engine against the plain implementation (tests/plain_raranex.py): every mechanism alone, then
whole prompts, prompts in portions, decoding token by token, batches of unequal requests, slots, pages and
state that are used again, and greedy generation through the library's entry point."""
import json

import pytest
import torch

import plain_raranex as P
from raranex_models import (SMALL, all_experts, attention, config, layer, left, make_weights, moe, parallel, right,
                            write_model)

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
        g = update.groups[0]
        h = torch.zeros(g[6][0].shape[0] if len(g) > 6 else g[0].shape[-2], D, device="cuda")
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
def test_two_norms_of_one_stream_with_every_kind_of_update(dtype, width, N):
    """Groups with a factor a row, normed ones, rows picked from anywhere with weights of their own, a base in
    place of the stream; two norms, one norm, and the stream itself cast into a wider matrix."""
    from lumenllm_b200.ops import kernels as K
    g = torch.Generator().manual_seed(width + N)
    rn = lambda *s: torch.randn(*s, generator=g)
    h, base, w1, w2, wn = rn(N, width), rn(width), 1 + 0.2 * rn(width), 1 + 0.2 * rn(width), 1 + 0.2 * rn(width)
    a, b, rowf = rn(3, N, width), rn(N, width), torch.rand(N, generator=g)
    rows, pw = rn(2 * N, width), torch.rand(N, 3, generator=g)
    place = torch.randint(-1, 2 * N, (N, 3), generator=g).int()
    c = lambda t: None if t is None else t.cuda().contiguous()
    groups = [(c(a), 0.5, None, c(wn), 1e-5), (c(b), 1.0, None, None, 0.0, c(rowf)),
              (c(rows), 1.0, None, None, 0.0, None, (c(place), c(pw)))]
    picked = (rows[place.clamp(min=0).long()] * (pw * (place >= 0))[:, :, None]).sum(1)
    update = 0.5 * P.rms_norm(a.sum(0), wn, 1e-5) + rowf[:, None] * b + picked
    for start in (None, base):
        x = update + (h if start is None else start)
        hc = c(h).clone()
        y1, y2 = K.add_shaped_rmsnorm(hc, groups, c(w1), 1e-6, dtype, base=c(start), weight2=c(w2))
        close(hc, x, F32, "stream")
        close(y1, P.rms_norm(x, w1, 1e-6), dtype, "first norm")
        close(y2, P.rms_norm(x, w2, 1e-6), dtype, "second norm")
        wide = torch.full((N, 2 * width), 7.0, dtype=dtype, device="cuda")
        hc = c(h).clone()
        assert K.add_shaped_rmsnorm(hc, groups, None, 0.0, None, base=c(start), cast_to=wide[:, width:], write_h=False) is None
        close(wide[:, width:], x, dtype, "cast")
        assert torch.equal(hc, c(h)) and bool((wide[:, :width] == 7).all())
        want = torch.tensor([N - 1, 0, 3], dtype=torch.int32).cuda()
        y = K.add_shaped_rmsnorm(c(h).clone(), groups, c(w1), 1e-6, dtype, rows=want, write_h=False, base=c(start))
        close(y, P.rms_norm(x, w1, 1e-6)[want.cpu().long()], dtype, "wanted rows")


@pytest.mark.parametrize("dtype", [F32, BF16])
@pytest.mark.parametrize("D,E,top,count,keep", [(64, 16, 3, 4, 2), (50, 6, 2, 3, 1), (256, 64, 6, 8, 4), (96, 200, 5, 40, 3),
                                                (40, 3, 1, 3, 2), (72, 40, 4, 1, 1), (64, 5, 5, 1, 1)])
@pytest.mark.parametrize("N", [1, 9, 300, 1200])
def test_router_in_groups(dtype, D, E, top, count, keep, N):
    """The choice in the best groups, normalised weights and the token's gate, whatever kernel instance the
    step's size takes: the same choices and weights for a row alone and in a batch."""
    from lumenllm_b200.ops import kernels as K
    g = torch.Generator().manual_seed(E + N)
    y = torch.randn(N, D, generator=g).to(dtype)
    w = torch.randn(E + 1, D, generator=g) * 2 * D ** -0.5
    corr = torch.randn(E, generator=g)
    idx, wt, gate = K.moe_route_x(y.cuda(), w.cuda(), corr.cuda(), top, 1.5, mode="sigmoid", groups=count, keep=keep,
                                  normalize=True, token_gate=True)
    z = y.double() @ w.double().T
    s = torch.sigmoid(z[:, :E])
    ref = P.choose(s, corr.double(), top, {"count": count, "keep": keep})
    c = s + corr.double()
    same = (idx.cpu().sort(dim=1).values == ref.sort(dim=1).values).all(dim=1)
    for t in (~same).nonzero().flatten().tolist():        # only where the plain scores tie to within rounding
        lost = torch.tensor(sorted(set(ref[t].tolist()) ^ set(idx[t].tolist())))
        by = c[t].view(count, -1).topk(min(2, E // count), dim=1).values.sum(1).sort(descending=True).values
        assert float(c[t][lost].max() - c[t][lost].min()) < 1e-5 or (count > 1 and float(by[keep - 1] - by[min(keep, count - 1)]) < 1e-5)
    chosen = torch.gather(s, 1, idx.cpu().long())
    close(wt, 1.5 * chosen / (chosen.sum(1, keepdim=True) + 1e-20), F32, "weights")
    close(gate, torch.sigmoid(z[:, E]), F32, "gate")
    one = K.moe_route_x(y[N // 2:N // 2 + 1].cuda(), w.cuda(), corr.cuda(), top, 1.5, mode="sigmoid", groups=count, keep=keep,
                        normalize=True, token_gate=True)
    assert torch.equal(one[0][0], idx[N // 2]) and torch.equal(one[1][0], wt[N // 2]) and torch.equal(one[2][0], gate[N // 2])
    i2, w2 = K.moe_route(z[:, :E].float().cuda(), corr.cuda(), top, 1.0, mode="sigmoid", groups=count, keep=keep, normalize=True)
    close(w2, torch.gather(s, 1, i2.cpu().long()) / torch.gather(s, 1, i2.cpu().long()).sum(1, keepdim=True), F32, "by logits")


@pytest.mark.parametrize("E,K_,F_,N,top", [(4, 128, 96, 300, 2), (3, 200, 256, 700, 1), (6, 64, 40, 50, 3), (5, 1024, 320, 2000, 2),
                                           (2, 8, 8, 5, 2)])
def test_products_of_rows_sorted_by_expert(E, K_, F_, N, top):
    """Places, gathered rows, and both grouped tcgen05 products, with experts that get many rows, few and none."""
    from lumenllm_b200.ops import kernels as K
    g = torch.Generator().manual_seed(E + N)
    lean = torch.tensor([2.0 ** -e for e in range(E)])
    lean[-1] = 0.0 if E > top else 1.0                    # the last expert is never chosen
    idx = torch.stack([torch.multinomial(lean, top, generator=g) for _ in range(N)]).int()
    idx[N // 3, 0] = E                                    # an entry that no expert takes
    y = torch.randn(N, K_, generator=g).to(BF16)
    gate_up, down = (torch.randn(E, r, c, generator=g).div(c ** 0.5).to(BF16) for r, c in ((2 * F_, K_), (K_, F_)))
    place = K.moe_place(idx.cuda(), E)
    p, used = place[0].cpu(), idx < E
    assert bool((p[~used] == -1).all()) and p[used].unique().numel() == int(used.sum())
    assert torch.equal(place[1].cpu()[(p[used] // K.MOE_PLACE_ROWS).long()], idx[used])
    assert int(place[2]) == sum(-(-int((idx == e).sum()) // K.MOE_PLACE_ROWS) for e in range(E))
    x = K.moe_gather(y.cuda(), place[0], place[3])
    token = torch.arange(N)[:, None].expand(N, top)
    assert torch.equal(x.cpu()[p[used].long()], y[token[used]])
    z = K.moe_product_placed(x, K.expert_weight(gate_up.cuda(), True), place)
    o = K.moe_product_placed(z, K.expert_weight(down.cuda(), False), place)
    W = gate_up.float()[idx[used].long()]
    gu = torch.einsum("nrc,nc->nr", W, y.float()[token[used]])
    ref = P.silu(gu[:, :F_]) * gu[:, F_:]
    got = z.cpu()[p[used].long()].float()
    close(got, ref, BF16, "gate/up")
    close(o.cpu()[p[used].long()], torch.einsum("nrc,nc->nr", down.float()[idx[used].long()], got), F32 if F_ < 64 else BF16, "down")


@pytest.mark.parametrize("E,N,top", [(16, 4097, 4), (300, 500, 6), (256, 40, 2), (1, 700, 1)])
def test_places_of_many_entries_and_experts(E, N, top):
    from lumenllm_b200.ops import kernels as K
    g = torch.Generator().manual_seed(E)
    idx = torch.randint(0, E + (E > 1), (N, top), generator=g).int()
    place, tile_expert, n_tiles, rows = K.moe_place(idx.cuda(), E)
    p, used = place.cpu(), idx < E
    assert bool((p[~used] == -1).all()) and p[used].unique().numel() == int(used.sum()) and int(p.max()) < rows
    assert torch.equal(tile_expert.cpu()[(p[used] // K.MOE_PLACE_ROWS).long()], idx[used])
    assert int(n_tiles) == sum(-(-int((idx == e).sum()) // K.MOE_PLACE_ROWS) for e in range(E))
    for e in range(min(E, 3)):                     # an expert's rows are its first ones, without a gap
        mine = p[idx == e].sort().values
        assert mine.numel() == 0 or torch.equal(mine, torch.arange(int(mine[0]), int(mine[0]) + mine.numel()).int())


@pytest.mark.parametrize("dtype", [F32, BF16])
@pytest.mark.parametrize("C", [64, 20, 1032])
def test_token_shift(dtype, C):
    """Rows mixed with the row before them, over steps whose sequences begin, go on and pause, on slots that are
    not the sequences' indices."""
    from lumenllm_b200.ops import kernels as K
    g = torch.Generator().manual_seed(C)
    mu = torch.rand(5, C, generator=g)
    lens = [[1, 40, 2], [3, 1, 1], [1, 1, 1], [17, 2, 5]]
    xs = [torch.randn(sum(l[b] for l in lens), C, generator=g).to(dtype) for b in range(3)]
    store, slots = torch.zeros(5, C + 4).cuda(), torch.tensor([4, 0, 2], dtype=torch.int32).cuda()
    at, outs = [0, 0, 0], [[], [], []]
    for step in lens:
        y = torch.cat([x[a:a + n] for x, a, n in zip(xs, at, step)]).cuda()
        cu = torch.tensor([0] + torch.tensor(step).cumsum(0).tolist(), dtype=torch.int32).cuda()
        seq = torch.repeat_interleave(torch.arange(3), torch.tensor(step)).int().cuda()
        for b, o in enumerate(pieces(K.shift_mix(y, mu.cuda(), store[:, :C], seq, cu, slots).cpu(), step)):
            outs[b].append(o)
            at[b] += step[b]
    for b in range(3):
        x = xs[b].float()
        before = torch.cat([torch.zeros(1, C), x[:-1]])
        ref = (x[:, None] + (before - x)[:, None] * mu).reshape(-1, 5 * C)
        close(torch.cat(outs[b]), ref, dtype, f"sequence {b}")
        close(store[int(slots[b]), :C], x[-1], F32, "state")
    assert float(store[:, C:].abs().max()) == 0.0 and float(store[[1, 3]].abs().max()) == 0.0


@pytest.mark.parametrize("rank,H,d,N", [(5, 2, 16, 3), (16, 3, 100, 40), (130, 1, 70, 17), (1, 4, 2, 1), (64, 5, 64, 300)])
def test_decays_and_bonuses(rank, H, d, N):
    from lumenllm_b200.ops import kernels as K
    g = torch.Generator().manual_seed(rank + N)
    C = H * d
    u, w, b, ub = torch.randn(3, N, 2 * C + rank + 9, generator=g), torch.randn(rank, C, generator=g) / rank, \
        torch.randn(C, generator=g) - 1, torch.randn(H, d, generator=g)
    out, bonus = K.low_rank_decay(u.cuda(), 2 * C + 4, w.cuda(), b.cuda(), twice=True, bonus=(ub.cuda(), 2, C + 2))
    x = u.sum(0).double()
    z = torch.tanh(x[:, 2 * C + 4:2 * C + 4 + rank]) @ w.double() + b.double()
    close(out, torch.exp(-torch.exp(z)), F32, "decay")
    r, k = x[:, 2:2 + C].view(N, H, d), x[:, C + 2:2 * C + 2].view(N, H, d)
    close(bonus, (r * ub.double() * k).sum(-1), F32, "bonus")


@pytest.mark.parametrize("H,d,lens", [(2, 8, ([150, 1, 33], [1, 40, 2])), (1, 72, ([130, 70, 40], [3, 1, 1])),
                                      (3, 64, ([600, 520, 700], [512, 600, 530])), (2, 30, ([540, 700, 513], [2, 1, 4])),
                                      (1, 128, ([300, 5, 600], [1, 1, 1])), (1, 200, ([1300, 1, 513], [1, 1, 1]))])
def test_recurrence_that_reads_before_it_writes(H, d, lens):
    """Three sequences in one launch, then each again from the state the first launch left: token by token,
    from staged runs, and in chunks side by side; partial sums and one sum."""
    from lumenllm_b200.ops import kernels as K
    g = torch.Generator().manual_seed(d)
    C, W = H * d, 3 * H * d + 8
    ub = torch.randn(H, d, generator=g, dtype=torch.float64)
    for S in (2, 1):
        state, slots = torch.zeros(5, H, d, d).cuda(), torch.tensor([3, 0, 4], dtype=torch.int32).cuda()
        seen = [([], [], [], []) for _ in range(3)]
        outs = [[], [], []]
        for ls in lens:
            u = torch.randn(S, sum(ls), W, generator=g) * 0.6
            al = torch.exp(-torch.exp(torch.randn(sum(ls), C, generator=g) - 3))
            x = u.sum(0).double()
            r, k, v = (x[:, 4 + i * C:4 + (i + 1) * C].view(-1, H, d) for i in range(3))
            bonus = (r * ub * k).sum(-1).float()
            cu = torch.tensor([0] + torch.tensor(ls).cumsum(0).tolist(), dtype=torch.int32).cuda()
            out = K.linear_attn(u.cuda(), 4, 4 + C, 4 + 2 * C, False, al.cuda(), state, cu, slots, 3, H, d, d, bonus=bonus.cuda())
            for b in range(3):
                outs[b].append(pieces(out.cpu(), ls)[b])
                for kept, t in zip(seen[b], (r, k, v, al.double().view(-1, H, d))):
                    kept.append(pieces(t, ls)[b])
        for b in range(3):
            r, k, v, a = (torch.cat(t) for t in seen[b])
            close(torch.cat(outs[b]), P.bonus_recurrence(r, k, v, a, ub).reshape(-1, C), F32, f"sequence {b}")
        assert float(state[1].abs().max()) == 0.0 and float(state[2].abs().max()) == 0.0


# ------------------------------------------------------------------ mixers alone

ATTENTION = [attention(4, 2, 16, 24, 1.5, size=9, keep=3, rot=8, base=5000.0), attention(3, 3, 20, 12, 2.0, size=40, keep=1, rot=20),
             attention(6, 2, 64, 64, 2.0, size=70, keep=66, rot=64), attention(4, 1, 128, 128, 1.2, size=100, keep=5, rot=30),
             attention(2, 1, 10, 6, 1.4), attention(5, 1, 72, 136, 1.1, size=1, keep=2, rot=72), attention(2, 2, 136, 40, 1.0, size=65)]
LEFT = [left(4, 2, 16, 24, 0.3, 6.0, 0.4, 16), left(3, 3, 32, 8, 0.25), left(6, 2, 64, 64, 0.12, None, 0.6, 33), left(4, 1, 128, 160, 0.09, 15.0),
        left(2, 1, 10, 6, 0.4, 4.0, 0.9, 2.5), left(4, 4, 200, 256, 0.07, 20.0, 0.1, 7), left(18, 1, 16, 24, 0.3, 9.0, 0.2, 20)]
RIGHT = [right(2, 16, 5), right(1, 72, 7), right(3, 64, 16), right(5, 8, 40), right(1, 20, 1), right(2, 30, 3)]
ANY_LEFT, ANY_RIGHT = LEFT[1], RIGHT[0]


@pytest.mark.parametrize("dtype", [F32, BF16])
@pytest.mark.parametrize("m", ATTENTION)
def test_windowed_attention_in_any_portions(m, dtype):
    D = 64
    part, w = mixer_part(m, D, dtype, seed=11)
    in_any_portions(part, runtime(dtype), lambda y: P.windowed_attention(y, w, "l0.mix", m, 1e-6, torch.arange(y.shape[0])), D,
                    dtype, seed=12)


@pytest.mark.parametrize("dtype", [F32, BF16])
@pytest.mark.parametrize("m", LEFT)
def test_tempered_attention_in_any_portions(m, dtype):
    D = 64
    part, w = mixer_part(parallel(m, ANY_RIGHT), D, dtype, seed=13, child=0)
    in_any_portions(part, runtime(dtype), lambda y: P.tempered_attention(y, w, "l0.mix.left", m, 1e-6, torch.arange(y.shape[0])), D,
                    dtype, seed=14)


@pytest.mark.parametrize("dtype", [F32, BF16])
@pytest.mark.parametrize("D", [48, 50])
@pytest.mark.parametrize("m", RIGHT)
def test_time_mixing_in_any_portions(m, D, dtype):
    part, w = mixer_part(parallel(ANY_LEFT, m), D, dtype, seed=15, child=1)
    assert part.tensor_cores == (dtype == BF16 and D == 48)
    in_any_portions(part, runtime(dtype), lambda y: P.time_mixing(y, w, "l0.mix.right", m, 1e-6), D, dtype, seed=16)


@pytest.mark.parametrize("dtype", [F32, BF16])
def test_two_mixers_side_by_side(dtype):
    D, m = 64, parallel(LEFT[0], right(5, 7, 3))
    part, w = mixer_part(m, D, dtype, seed=17)
    assert part.cache_need().n_kv == 2 and part.state_shape()[0] == (64 + 5 * 7 * 7,)
    in_any_portions(part, runtime(dtype), lambda y: P.side_by_side(y, w, "l0.mix", m, 1e-6, torch.arange(y.shape[0])),
                    D, dtype, seed=18)


def loud_pair(w, pre, H, G, d, D):
    """Every query head of a kv head alike, and that kv head's key weights the same with their columns moved on
    by one: a row equal to another moved the same way has a key equal to the other's query."""
    q = w[pre + "q"].view(H, d, D).clone()
    for h in range(H):
        q[h] = q[h // (H // G) * (H // G)]
    w[pre + "q"] = q.reshape(H * d, D)
    w[pre + "k"] = torch.roll(q[::H // G], -1, dims=2).reshape(G * d, D).clone()


WINDOWS = [(32, 24, 20, 3), (32, 24, 64, 64), (64, 64, 20, 3), (64, 64, 65, 70), (128, 160, 130, 2), (24, 24, 1, 1), (64, 64, 64, 0)]


@pytest.mark.parametrize("decode", [False, True])
@pytest.mark.parametrize("dtype", [F32, BF16])
@pytest.mark.parametrize("d,dv,size,keep", WINDOWS)
def test_a_loud_key_at_every_edge(d, dv, size, keep, dtype, decode):
    """One key that equals the last query, placed at the first token, on both sides of the kept tokens' end, of the
    window's start and of every page border, and next to the query: it is heard where it is in sight, and where
    it is not nothing of it is (the plain result with it in sight is far off)."""
    D, T = 64, 300
    m = attention(4, 2, d, dv, 6.0 / d, size=size, keep=keep)
    part, w = mixer_part(m, D, dtype, seed=21, edit=lambda w: loud_pair(w, "l0.mix.", 4, 2, d, D))
    rt, pos, p = runtime(dtype), torch.arange(T), T - 1
    places = {0, keep - 1, keep, p - size, p - size + 1, p - 1, 63, 64, 127, 128, 191, 192}
    for j0 in sorted(x for x in places if 0 <= x < p):
        y = rows(T, D, dtype, seed=22 + j0)
        y[j0] = torch.roll(y[p], -1)
        ref = P.windowed_attention(y, w, "l0.mix", m, 1e-6, pos)
        quiet = y.clone()
        quiet[j0] = -quiet[j0]
        moved = float((P.windowed_attention(quiet, w, "l0.mix", m, 1e-6, pos)[-1] - ref[-1]).abs().max())
        assert moved > 0.1 if p - j0 < size or j0 < keep else moved == 0.0
        (got,) = run_mixer(part, rt, [pieces(y, (T - 1, 1) if decode else (T,))])
        close(got[-1:], ref[-1:], dtype, f"key {j0}")


@pytest.mark.parametrize("decode", [False, True])
@pytest.mark.parametrize("dtype", [F32, BF16])
@pytest.mark.parametrize("d,dv", [(32, 16), (64, 64), (128, 160)])
def test_a_loud_key_far_back_under_a_cap_and_a_temperature(d, dv, dtype, decode):
    """The same without a window: capped scores and queries that grow with the position, at every page border."""
    D, T = 64, 300
    m = left(4, 2, d, dv, 3.0 / d, 9.0, 0.8, 40)

    def edit(w):
        loud_pair(w, "l0.mix.left.", 4, 2, d, D)
        for n in "qk":
            w[f"l0.mix.left.{n}.norm"] = torch.ones_like(w[f"l0.mix.left.{n}.norm"])

    part, w = mixer_part(parallel(m, ANY_RIGHT), D, dtype, seed=23, child=0, edit=edit)
    rt = runtime(dtype)
    plain = lambda y, mm=m: P.tempered_attention(y, w, "l0.mix.left", mm, 1e-6, torch.arange(T))
    for j0 in (0, 1, 63, 64, 65, 127, 128, 191, 192, 298):
        y = rows(T, D, dtype, seed=24 + j0)
        y[j0] = torch.roll(y[T - 1], -1)
        ref = plain(y)
        quiet = y.clone()
        quiet[j0] = -quiet[j0]
        for other in (plain(quiet), plain(y, dict(m, softcap=None)), plain(y, dict(m, q_temp=None))):
            assert float((other[-1] - ref[-1]).abs().max()) > 0.06
        (got,) = run_mixer(part, rt, [pieces(y, (T - 1, 1) if decode else (T,))])
        close(got[-1:], ref[-1:], dtype, f"key {j0}")


@pytest.mark.parametrize("dtype", [F32, BF16])
def test_temperature_changes_at_its_period(dtype):
    """Positions just before and at the multiples of the period, in a prompt and decoded one by one."""
    D, m = 64, left(4, 2, 64, 64, 0.4, None, 4.0, 10)
    part, w = mixer_part(parallel(m, ANY_RIGHT), D, dtype, seed=25, child=0)
    y = rows(45, D, dtype, seed=26)
    ref = P.tempered_attention(y, w, "l0.mix.left", m, 1e-6, torch.arange(45))
    late = P.tempered_attention(y, w, "l0.mix.left", m, 1e-6, torch.arange(45) - 1)
    assert float((late - ref)[[9, 19, 29]].abs().amax(1).min()) > 0.05
    for cut in ((45,), (8,) + (1,) * 37):
        (got,) = run_mixer(part, runtime(dtype), [pieces(y, cut)])
        close(got, ref, dtype, f"{cut[:2]}")


@pytest.mark.parametrize("dtype", [F32, BF16])
def test_a_loud_row_around_every_cut_of_the_shift(dtype):
    D, m = 48, RIGHT[0]
    part, w = mixer_part(parallel(ANY_LEFT, m), D, dtype, seed=27, child=1)
    y = rows(112, D, dtype, seed=28)
    y[100] *= 10
    ref = P.time_mixing(y, w, "l0.mix.right", m, 1e-6)
    for cut in ((112,), (100, 12), (101, 11), (101, 1, 10), (102, 2, 8), (100,) + (1,) * 12):
        (got,) = run_mixer(part, runtime(dtype), [pieces(y, cut)])
        close(got[99:], ref[99:], dtype, f"{cut[:3]}")


@pytest.mark.parametrize("dtype", [F32, BF16])
def test_states_remember_far_back_and_forget_by_channel(dtype):
    """A loud first token, then 400 quiet ones in portions: what decays slowly still carries it at the end, what
    decays fast has lost it."""
    D, T, m = 48, 401, right(2, 16, 4)

    def slow(w):
        w["l0.mix.right.w0"] = torch.cat([torch.full((16,), -9.0), torch.full((16,), 1.5)]).to(BF16)

    y = rows(T, D, dtype, seed=30, std=0.5)
    y[0] = (y[0] * 40).to(dtype).float()
    quiet = y.clone()
    quiet[0] = 0.0
    part, w = mixer_part(parallel(ANY_LEFT, m), D, dtype, seed=29, child=1, edit=slow)
    ref = P.time_mixing(y, w, "l0.mix.right", m, 1e-6)
    assert float((P.time_mixing(quiet, w, "l0.mix.right", m, 1e-6)[-1] - ref[-1]).abs().max()) > 0.05
    (got,) = run_mixer(part, runtime(dtype), [pieces(y, (1, 199, 2, 198, 1))])
    close(got, ref, dtype)


MIXTURES = [moe(40, 6, 2, 3, 2, shared=24), moe(24, 8, 3, 4, 2), moe(64, 4, 1, 2, 1, shared=100), moe(20, 5, 5, shared=12), moe(16, 3, 2, 3, 3)]


@pytest.mark.parametrize("dtype", [F32, BF16])
@pytest.mark.parametrize("D", [64, 50])
@pytest.mark.parametrize("N", [1, 9, 150, 900])
@pytest.mark.parametrize("m", MIXTURES)
def test_expert_mixture(m, N, D, dtype):
    """On equal inputs, choices and all; sizes that go to the tcgen05 product, to the short tiles and, at width 50,
    to the 32-bit product."""
    from lumenllm_b200.config import config_from_dict
    from lumenllm_b200.parts import build_part
    cfg = config(8, D, 1e-6, [layer(ANY_ATTENTION, m)])
    w = make_weights(cfg, 31)
    part = build_part("ffn", config_from_dict(cfg).model_spec().layers[0].ffn, {k: v.cuda() for k, v in w.items()}, runtime(dtype))
    y = rows(N, D, dtype, seed=32)
    close(total(part.forward(y.to(dtype).cuda(), None), D), P.expert_mixture(y, {k: v.float() for k, v in w.items()}, "l0.mlp", m), dtype)


ANY_ATTENTION = ATTENTION[0]


@pytest.mark.parametrize("dtype", [F32, BF16])
@pytest.mark.parametrize("D,N", [(64, 5), (50, 5), (64, 300), (256, 700)])
def test_a_pass_makes_the_stream_anew(D, N, dtype):
    """Twice in a row, with an update pending before each, and the next layer's pair of norms behind it."""
    from types import SimpleNamespace
    from lumenllm_b200.config.spec import PartSpec
    from lumenllm_b200.parts import build_part
    from lumenllm_b200.parts.norm import ShapedUpdate, rmsnorm_pair
    g = torch.Generator().manual_seed(D)
    w = {"loop.in": torch.randn(D, 2 * D, generator=g).mul((2 * D) ** -0.5).to(BF16), "loop.step": torch.randn(2, D, generator=g).to(BF16),
         "a": torch.ones(D), "b": 1 + 0.1 * torch.randn(D, generator=g)}
    rt = runtime(dtype)
    cuda = {k: v.cuda() for k, v in w.items()}
    part = build_part("stream", PartSpec("loop_input", {"hidden_size": D, "times": 2, "tensor": "loop.in", "step_tensor": "loop.step"}), cuda, rt)
    norms = [build_part("norm", PartSpec("rmsnorm", {"size": D, "eps": 1e-6, "tensor": n}), cuda, rt) for n in "ab"]
    x0, u = torch.randn(N, D, generator=g).to(BF16).float(), torch.randn(3, N, D, generator=g)
    x, h, ctx = x0, x0.cuda(), SimpleNamespace(extras={})
    part.start(h, ctx)
    plain = {k: v.float() for k, v in w.items()}
    for t, pending in ((0, u.cuda()), (1, ShapedUpdate([(u[0].cuda(), 0.5, None, None, 0.0)]))):
        x = P.loop_entry(x + (u.sum(0) if t == 0 else 0.5 * u[0]), x0, plain, t)
        h, pending = part.forward(h, pending, ctx, t)
        y1, y2 = rmsnorm_pair(*norms, h, pending, dtype)
        close(h, x, dtype, f"pass {t}")
        close(y1, P.rms_norm(x, plain["a"], 1e-6), dtype, "first norm")
        close(y2, P.rms_norm(x, plain["b"], 1e-6), dtype, "second norm")


# ------------------------------------------------------------------ the model in the engine

# what a run of a type is compared on: in bfloat16 the form in which every expert is chosen (raranex_models.all_experts)
FORMS = {"float32": lambda c: c, "bfloat16": all_experts}


@pytest.fixture(scope="module")
def models(tmp_path_factory):
    root = tmp_path_factory.mktemp("raranex")
    return {(name, dt): write_model(form(cfg), root / f"{name}_{dt}", seed=3 + i)
            for i, (name, cfg) in enumerate(SMALL.items()) for dt, form in FORMS.items()}


@pytest.fixture(scope="module")
def plain(models):
    return {key: P.load_model(folder) + ({},) for key, folder in models.items()}


def plain_logits(plain, key, tokens):
    cfg, w, memo = plain[key]
    tokens_key = tuple(tokens)
    if tokens_key not in memo:
        memo[tokens_key] = P.forward(cfg, w, tokens)
    return memo[tokens_key]


def engine_of(models, name, dtype, **kw):
    from lumenllm_b200.engine import Engine
    kw.setdefault("max_tokens", 2048)
    return Engine.from_folder(models[name, dtype], dtype=dtype, **kw)


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("name", list(SMALL))
def test_whole_prompts(name, dtype, models, plain):
    from lumenllm_b200.engine import StepEntry
    eng = engine_of(models, name, dtype)
    for toks in tokens_of(SMALL[name], (1, 2, 65, 200), seed=30):
        slot = eng.alloc_slot()
        close(eng.step([StepEntry(slot, toks, list(range(len(toks))))]), plain_logits(plain, (name, dtype), toks), dtype, f"{len(toks)} tokens")
        eng.free_slot(slot)
    eng.cache.check()
    eng.check_kernels()


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("name", list(SMALL))
def test_residual_stream_after_every_layer_run(name, dtype, models, plain):
    from lumenllm_b200.engine import StepEntry
    from lumenllm_b200.engine.context import EntryView
    from lumenllm_b200.ops import kernels as K
    from lumenllm_b200.parts.norm import ShapedUpdate
    cfg, w, _ = plain[name, dtype]
    toks = tokens_of(cfg, (40,), seed=31)[0]
    ref = []
    P.forward(cfg, w, toks, ref)
    eng = engine_of(models, name, dtype)
    ctx = eng.build_context([StepEntry(eng.alloc_slot(), toks, [])])
    m = eng.model
    assert len(m.schedule) == len(ref)
    h, pending = m.embedding.forward(ctx.tokens, ctx), None
    for part in m.stream_parts:
        part.start(h, ctx)
    for i, e in enumerate(m.schedule):
        if e.before is not None:
            h, pending = m.stream_parts[e.before].forward(h, pending, ctx, e.before_index)
        h, pending = m.blocks[e.layer].forward(h, pending, ctx, EntryView(ctx, i, i if i in ctx.cache.group_of else None, True))
        x = h.clone()
        if pending is not None:
            K.add_shaped_rmsnorm(x, ShapedUpdate.groups_of(pending), None, 0.0, F32)
        close(x, ref[i], dtype, f"after run {i} (layer {e.layer})")


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("name", list(SMALL))
def test_prompt_in_portions_and_decoded_token_by_token(name, dtype, models, plain):
    from lumenllm_b200.engine import StepEntry
    toks = tokens_of(SMALL[name], (171,), seed=32)[0]
    ref = plain_logits(plain, (name, dtype), toks)
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
    refs = [plain_logits(plain, (name, dtype), p) for p in prompts]
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
    ref = plain_logits(plain, ("Z", dtype), toks)
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
    """Widths 44 and 50, heads of 6 keys and 10 values, heads of 7 channels, experts of 9: no row of any matrix is a
    multiple of 16 bytes, so the products and the row kernels go the ways that need no alignment."""
    from lumenllm_b200.engine import Engine, StepEntry
    cfg = FORMS[dtype](config(61, width, 1e-5, [
        layer(parallel(left(3, 1, 6, 10, 0.4, 7.0, 0.3, 30), right(2, 7, 3)), moe(9, 4, 2, 2, 1, shared=11)),
        layer(attention(3, 1, 6, 10, 1.4, size=50, keep=3, rot=4), moe(13, 3, 1, 3, 2))], loop=(0, 2, 2)))
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
    """A prompt long and wide enough for the tensor-core kernels of every product (the experts' over rows sorted by
    expert, the attention's output product into the stream in place), of both attentions, and for the chunks of
    the recurrence."""
    from lumenllm_b200.engine import Engine, StepEntry
    cfg = all_experts(config(64, 1024, 1e-6, [
        layer(attention(4, 2, 128, 128, 0.1, size=600, keep=5, rot=128), moe(128, 4, 2, 2, 1, shared=256)),
        layer(parallel(left(4, 2, 64, 96, 0.12, 20.0, 0.2, 500), right(4, 64, 16)), moe(192, 3, 1, shared=320))], loop=(0, 2, 2)))
    T = 2300
    folder = write_model(cfg, tmp_path / "wide", seed=70)
    toks = tokens_of(cfg, (T,), seed=71)[0]
    want = [0, 1, 4, 5, 63, 64, 599, 600, 604, 605, 1023, 1024, 2047, 2048, T - 2, T - 1]
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
    cfg, w, _ = plain[name, dtype]
    built = build(EngineConfig(model_path=str(models[name, dtype]), dtype=dtype, context_size=512, max_batch=3))
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
    rc = main(["generate", "--model", str(models["X", "float32"]), "--prompt-tokens", "5,6,7", "--prompt-tokens", "1",
               "--max-tokens", "4", "--ctx-size", "128", "--format", "json", "--dtype", "float32"])
    assert rc == 0
    outs = json.loads(capsys.readouterr().out.strip().splitlines()[-1])
    cfg, w = P.load_model(models["X", "float32"])
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
    done = subprocess.run([sys.executable, str(runner), "--model", str(models[name, "float32"]), "--dtype", "float32",
                           "--out", str(out), "--max-tokens", "128"],
                          input="".join(json.dumps(s) + "\n" for s in steps), capture_output=True, text=True, timeout=600)
    assert done.returncode == 0, done.stderr[-2000:]
    assert [l for l in done.stdout.splitlines() if l.startswith("done ")] == [f"done {s['step']}" for s in steps]
    ra, rb = (plain_logits(plain, (name, "float32"), x) for x in (a, b))
    read = lambda s: torch.from_numpy(np.fromfile(out / f"{s}.f32", dtype="<f4").reshape(-1, cfg["vocab"]).copy())
    close(read(0), torch.stack([ra[0], ra[29], rb[7]]), F32, "prompts")
    close(read(1), rb[8:9], F32, "the short request's last token")
    for t in range(9):
        close(read(2 + t), ra[31 + t:32 + t], F32, f"decoded {t}")
