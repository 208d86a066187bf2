"""Small Mefatar configurations and seeded weights for the tests. The sizes differ from one another in
everything that can differ: heads against kv heads (ratio 1, 2, 3, 4), key size against value size,
rotation over a part of a head, over all of it and none, frequencies stretched by wavelength and plain
ones; convolutions of one to five taps; gated linear attention with one to five heads, key sizes that
fill a lane's share and that do not, decay ranks of 2 to 24, exponents of 1 and not; recurrent units of one
to five blocks, as wide as the model, narrower and wider, blocks that fill a tile of the block-diagonal
product and that do not; layers with and without feed-forward; loops over the first layers, over the last,
over both kinds, and none; widths that are multiples of 16, of 8, of 4 and of 2 only.
"""
import json
from pathlib import Path

import torch


def left(heads, kv_heads, dim, vdim, scale, conv, rot=None, base=10000.0, scaling=None):
    m = {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "conv": conv, "scale": scale}
    if rot is not None:
        m["rot"] = {"base": base, "dims": rot}
        if scaling is not None:
            m["rot"]["scaling"] = dict(zip(("factor", "low", "high", "original"), scaling))
    return m


def right(heads, dim, vdim, tau, rank):
    return {"heads": heads, "dim": dim, "vdim": vdim, "tau": tau, "decay_rank": rank}


def parallel(a, b):
    return {"left": a, "right": b}


def unit(width, blocks, conv):
    return {"width": width, "blocks": blocks, "conv": conv}


def layer(mixer, ff=None):
    return {"type": "parallel" if "left" in mixer else "rglru", "mixer": mixer,
            "mlp": None if ff is None else {"kind": "dense", "ff": ff}}


def config(vocab, width, eps, layers, loop=None):
    c = {"architecture": "Mefatar", "vocab": vocab, "width": width, "norm": {"eps": eps}, "layers": layers}
    if loop is not None:
        c["loop"] = dict(zip(("start", "stop", "times"), loop))
    return c


SMALL = {
    # values wider than keys and narrower; a loop over both kinds of layers in the middle
    "X": config(97, 64, 1e-6, [
        layer(parallel(left(4, 2, 16, 24, 0.3, 4, rot=8, base=5000.0, scaling=(4.0, 1.0, 4.0, 64)),
                       right(2, 16, 24, 8.0, 5)), 80),
        layer(unit(40, 5, 2)),
        layer(parallel(left(3, 3, 32, 8, 0.25, 2, rot=32, base=500.0), right(3, 8, 40, 1.0, 8))),
        layer(unit(48, 1, 4), 56)], loop=(1, 3, 3)),
    # no loop; no rotation in one layer; a convolution of one tap; a feed-forward wider than the model
    "Y": config(160, 96, 1e-5, [
        layer(unit(120, 3, 4), 200),
        layer(parallel(left(6, 2, 32, 32, 0.11, 1), right(1, 40, 24, 16.0, 2)), 72),
        layer(parallel(left(3, 1, 16, 48, 0.2, 5, rot=4, base=1e6, scaling=(8.0, 2.0, 2.0, 128)),
                       right(5, 24, 16, 4.0, 24)))]),
    # sizes that the tensor-core attention kernels take (64, 128), blocks that fill a tile of the
    # block-diagonal product (128) and that do not (64); a loop over the last layers
    "Z": config(211, 128, 3e-6, [
        layer(parallel(left(4, 2, 64, 64, 0.12, 4, rot=32, base=2e5, scaling=(16.0, 1.0, 8.0, 96)),
                       right(2, 64, 64, 12.0, 16)), 160),
        layer(unit(128, 2, 4), 96),
        layer(parallel(left(2, 1, 128, 128, 0.09, 3, rot=128, base=1e5), right(2, 128, 32, 16.0, 8)), 96),
        layer(unit(256, 2, 4))], loop=(2, 4, 2)),
    # a single layer, run twice
    "V": config(64, 80, 1e-5, [layer(parallel(left(5, 1, 16, 16, 0.25, 3, rot=16), right(1, 72, 96, 2.0, 7)), 48)],
                loop=(0, 1, 2)),
}


def make_weights(cfg, seed):
    """Seeded bfloat16 tensors by the design's names, of a size that keeps activations of order one;
    decays slow enough to remember, sinks of both signs."""
    g = torch.Generator().manual_seed(seed)
    rn = lambda *shape, std=1.0: torch.randn(shape, generator=g) * std
    D, t = cfg["width"], {}
    mat = lambda rows, cols: rn(rows, cols, std=cols ** -0.5)
    t["embed"], t["final.norm"] = rn(cfg["vocab"], D), 1 + rn(D, std=0.1)
    for i, L in enumerate(cfg["layers"]):
        m, p = L["mixer"], f"l{i}."
        t[p + "norm1"], t[p + "ls1"] = 1 + rn(D, std=0.1), 0.6 + rn(D, std=0.3)
        if L["type"] == "parallel":
            a, b = m["left"], m["right"]
            H, G, d, dv = a["heads"], a["kv_heads"], a["dim"], a["vdim"]
            q = p + "mix.left."
            for name, rows in (("q", H * d), ("k", G * d), ("v", G * dv)):
                t[q + name] = mat(rows, D)
                t[q + name + ".conv"] = rn(rows, a["conv"], std=0.4)
                t[q + name + ".conv"][:, -1] += 1.0
            t[q + "q.norm"], t[q + "k.norm"] = 1 + rn(H * d, std=0.1), 1 + rn(G * d, std=0.1)
            t[q + "sink"] = rn(H, std=1.5)
            t[q + "g"], t[q + "o"], t[q + "out"] = mat(H * dv, D), mat(D, H * dv), 1 + rn(D, std=0.1)
            H, d, dv, r = b["heads"], b["dim"], b["vdim"], b["decay_rank"]
            q = p + "mix.right."
            for name, rows in (("q", H * d), ("k", H * d), ("v", H * dv), ("g", H * dv), ("a1", r)):
                t[q + name] = mat(rows, D)
            t[q + "a2"], t[q + "a2.b"] = mat(H * d, r), 1.5 + rn(H * d)
            t[q + "norm"], t[q + "o"], t[q + "out"] = 1 + rn(dv, std=0.1), mat(D, H * dv), 1 + rn(D, std=0.1)
        else:
            C, B, q = m["width"], m["blocks"], p + "mix."
            t[q + "y"], t[q + "y.b"], t[q + "x"], t[q + "x.b"] = mat(C, D), rn(C, std=0.3), mat(C, D), rn(C, std=0.3)
            t[q + "conv"], t[q + "conv.b"] = rn(C, m["conv"], std=0.5), rn(C, std=0.2)
            for n in ("ra", "ri"):
                t[q + n], t[q + n + ".b"] = rn(B, C // B, C // B, std=(C // B) ** -0.5), rn(B, C // B, std=0.3)
            t[q + "lam"], t[q + "o"] = -3.0 + rn(C, std=1.5), mat(D, C)
        if L["mlp"] is not None:
            F = L["mlp"]["ff"]
            t[p + "norm2"], t[p + "ls2"] = 1 + rn(D, std=0.1), 0.6 + rn(D, std=0.3)
            t[p + "mlp.gate"], t[p + "mlp.up"], t[p + "mlp.down"] = mat(F, D), mat(F, D), mat(D, F)
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
