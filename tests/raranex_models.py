"""Small Raranex configurations and seeded weights for the tests. The sizes differ from one another in
everything that can differ: heads against kv heads (ratio 1, 2, 3, 4, 17), key size against value size, widths
that fill a tile of the tensor-core attention and that do not, rotation over a part of a head, over all of it
and none; windows shorter and longer than a cache page, kept first tokens of none, a few, a window's worth
and more than a page; query temperatures of short and long periods and none, caps and none; time mixing of
one to five heads, ranks of 1 to 24; experts in one to four groups, of which one to all are kept, one to five
choices, with and without a shared expert; layers without a feed-forward; loops over the first layers, over
the last, over both kinds, of one pass and several, and none; widths that are multiples of 16, of 8, of 4 and
of 2 only.
"""
import copy
import json
from pathlib import Path

import torch


def attention(heads, kv_heads, dim, vdim, scale, size=None, keep=0, rot=None, base=10000.0):
    m = {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "scale": scale}
    if size is not None:
        m["mask"] = {"size": size, "keep_first": keep}
    if rot is not None:
        m["rot"] = {"base": base, "dims": rot}
    return m


def left(heads, kv_heads, dim, vdim, scale, softcap=None, coef=None, every=None):
    m = {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "scale": scale}
    if softcap is not None:
        m["softcap"] = softcap
    if coef is not None:
        m["q_temp"] = {"coef": coef, "every": every}
    return m


def right(heads, dim, rank):
    return {"heads": heads, "dim": dim, "decay_rank": rank}


def parallel(a, b):
    return {"left": a, "right": b}


def moe(ff, experts, top, count=1, keep=1, shared=None):
    m = {"kind": "moe", "expert": {"ff": ff},
         "router": {"experts": experts, "top": top, "groups": {"count": count, "keep": keep}}}
    if shared is not None:
        m["shared"] = {"ff": shared}
    return m


def layer(mixer, mlp=None):
    return {"type": "parallel" if "left" in mixer else "attention", "mixer": mixer, "mlp": mlp}


def config(vocab, width, eps, layers, loop=None):
    c = {"architecture": "Raranex", "vocab": vocab, "width": width, "norm": {"eps": eps}, "layers": layers}
    if loop is not None:
        c["loop"] = dict(zip(("start", "stop", "times"), loop))
    return c


SMALL = {
    # values wider than keys and narrower; a loop over both kinds of layers in the middle
    "X": config(97, 64, 1e-6, [
        layer(attention(4, 2, 16, 24, 0.4, size=9, keep=3, rot=8, base=5000.0), moe(40, 6, 2, 3, 2, shared=24)),
        layer(parallel(left(4, 2, 16, 20, 0.3, 6.0, 0.4, 16), right(3, 12, 5)), moe(24, 8, 3, 4, 2, shared=16)),
        layer(attention(3, 3, 20, 12, 0.3, size=40, keep=1, rot=20)),
        layer(parallel(left(3, 1, 24, 40, 0.25), right(1, 20, 1)), moe(16, 5, 5, shared=40))], loop=(1, 3, 3)),
    # no loop; no window and no rotation in one layer; more kept tokens than a page holds; no shared expert
    "Y": config(160, 96, 1e-5, [
        layer(parallel(left(6, 2, 32, 48, 0.2, 12.0, 0.7, 5.5), right(5, 8, 24)), moe(56, 4, 1, 2, 1)),
        layer(attention(6, 2, 48, 32, 0.2, size=33, keep=70, rot=16, base=300.0), moe(20, 12, 4, 4, 4, shared=72)),
        layer(attention(4, 4, 8, 8, 0.5), moe(32, 6, 2, 2, 2))]),
    # widths that fill the tensor-core attention's tiles and that do not; a loop over the last layers
    "Z": config(211, 128, 3e-6, [
        layer(attention(4, 2, 64, 64, 0.2, size=100, keep=2, rot=64, base=2e5), moe(64, 8, 2, 2, 1, shared=96)),
        layer(attention(6, 2, 128, 128, 0.1, size=70, keep=6, rot=32, base=1e5), moe(48, 4, 2, shared=32)),
        layer(parallel(left(4, 1, 128, 160, 0.09, 25.0, 0.2, 50), right(2, 64, 16)), moe(40, 9, 3, 3, 2, shared=48)),
        layer(parallel(left(3, 1, 72, 56, 0.12, None, 0.5, 30), right(4, 32, 8)))], loop=(1, 4, 2)),
    # a single layer, run twice; more query heads a kv head than the tensor-core attention takes
    "V": config(64, 80, 1e-5, [layer(parallel(left(17, 1, 16, 16, 0.25, 8.0, 0.3, 9), right(1, 72, 7)),
                                     moe(48, 3, 2, 3, 2, shared=16))], loop=(0, 1, 2)),
    # one pass over the first layers: the stream is made anew once
    "U": config(73, 52, 1e-5, [layer(attention(2, 1, 12, 20, 0.4, size=130, keep=4, rot=12), moe(12, 4, 1, 2, 2, shared=8)),
                               layer(attention(2, 2, 12, 12, 0.35, size=5, keep=5, rot=2))], loop=(0, 1, 1)),
}


def all_experts(cfg):
    """The same model with every mixture using all its experts. A choice among experts is not continuous: where
    two scores nearly tie, the rounding of a bfloat16 stream decides, and the token then goes another way. Whole
    models are therefore compared in 32-bit as they are and in bfloat16 in this form."""
    c = copy.deepcopy(cfg)
    for L in c["layers"]:
        if L["mlp"] is not None:
            r = L["mlp"]["router"]
            r["top"], r["groups"]["keep"] = r["experts"], r["groups"]["count"]
    return c


def make_weights(cfg, seed):
    """Seeded bfloat16 tensors by the design's names, of a size that keeps activations of order one; decays slow
    enough to remember; router rows large enough for choices to be clear of ties in 32-bit."""
    g = torch.Generator().manual_seed(seed)
    rn = lambda *shape, std=1.0: torch.randn(shape, generator=g) * std
    D, t = cfg["width"], {}
    mat = lambda rows, cols: rn(rows, cols, std=cols ** -0.5)

    def heads(q, a):
        H, G, d, dv = a["heads"], a["kv_heads"], a["dim"], a["vdim"]
        t[q + "q"], t[q + "k"], t[q + "v"] = mat(H * d, D), mat(G * d, D), mat(G * dv, D)
        t[q + "g"], t[q + "o"] = mat(H, D), mat(D, H * dv)

    t["embed"], t["head"], t["final.norm"] = rn(cfg["vocab"], D), mat(cfg["vocab"], D), 1 + rn(D, std=0.1)
    if cfg.get("loop"):
        t["loop.in"], t["loop.step"] = mat(D, 2 * D), rn(cfg["loop"]["times"], D, std=0.5)
    for i, L in enumerate(cfg["layers"]):
        m, p = L["mixer"], f"l{i}."
        t[p + "norm1"] = 1 + rn(D, std=0.1)
        if L["type"] == "parallel":
            a, b, q = m["left"], m["right"], p + "mix.left."
            heads(q, a)
            t[q + "q.norm"], t[q + "k.norm"], t[q + "out"] = 1 + rn(a["dim"], std=0.2), 1 + rn(a["dim"], std=0.2), 1 + rn(D, std=0.1)
            q, C, r = p + "mix.right.", b["heads"] * b["dim"], b["decay_rank"]
            for s in "rkvgw":
                t[f"{q}mu.{s}"] = 0.5 + rn(D, std=0.3)
            for s in "rkvg":
                t[q + s] = mat(C, D)
            # keys that lean towards the receptance, and a positive bonus: at a sequence's first token a head's normed
            # output is v times the sign of sum(r u k), which rounding must not decide
            t[q + "mu.k"], t[q + "k"] = t[q + "mu.r"] + rn(D, std=0.1), 0.8 * t[q + "r"] + 0.6 * t[q + "k"]
            t[q + "w1"], t[q + "w2"], t[q + "w0"] = mat(r, D), mat(C, r), -2.0 + rn(C)
            t[q + "u"], t[q + "norm"] = 0.4 + rn(b["heads"], b["dim"], std=0.7).abs(), 1 + rn(C, std=0.1)
            t[q + "o"], t[q + "out"] = mat(D, C), 1 + rn(D, std=0.1)
        else:
            heads(p + "mix.", m)
        if L["mlp"] is not None:
            f, q = L["mlp"], p + "mlp."
            E = f["router"]["experts"]
            t[p + "norm2"] = 1 + rn(D, std=0.1)
            t[q + "router"], t[q + "correction"] = rn(E, D, std=3.0 * D ** -0.5), rn(E, std=0.3)
            for name, F in [(f"e{e}", f["expert"]["ff"]) for e in range(E)] + ([("shared", f["shared"]["ff"])] if f.get("shared") else []):
                t[f"{q}{name}.gate"], t[f"{q}{name}.up"], t[f"{q}{name}.down"] = mat(F, D), mat(F, D), mat(D, F)
            if f.get("shared"):
                t[q + "shared.sg"] = mat(1, D)
    return {k: v.to(torch.bfloat16) for k, v in t.items()}


def without_ranks(cfg):
    """The configuration as a checkpoint's config.json writes it: the decays' rank is the tensors' matter."""
    c = json.loads(json.dumps(cfg))
    for L in c["layers"]:
        L["mixer"].get("right", {}).pop("decay_rank", None)
    return c


def write_model(cfg, folder, seed):
    from lumenllm_b200.weights.safetensors_io import write_file
    folder = Path(folder)
    folder.mkdir(parents=True, exist_ok=True)
    (folder / "config.json").write_text(json.dumps(without_ranks(cfg)))
    write_file(folder / "model.safetensors", make_weights(cfg, seed))
    return folder
