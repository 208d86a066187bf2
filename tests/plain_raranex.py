"""A plain, slow implementation of the Raranex decoder on the CPU, written from the design's
equations, one function per mechanism. It shares no code with the library: whole sequences only,
no cache, no batching, a Python loop over time for the recurrence. The tests compare the engine
with it.

Notation: a sequence of T tokens, width D. Softmax attention: H query heads, G key/value heads, key
size d, value size dv. Time mixing: H heads of d channels, state S [d, d] a head. Every function takes
float32 (or float64) tensors.
"""
import json
import math
import struct
from pathlib import Path

import torch

F = torch.float32


def read_safetensors(path):
    raw = Path(path).read_bytes()
    (n,) = struct.unpack("<Q", raw[:8])
    head = json.loads(raw[8:8 + n])
    data = memoryview(raw)[8 + n:]
    kinds = {"BF16": torch.bfloat16, "F32": torch.float32, "I32": torch.int32, "F16": torch.float16}
    out = {}
    for name, info in head.items():
        if name == "__metadata__":
            continue
        a, b = info["data_offsets"]
        out[name] = torch.frombuffer(bytearray(data[a:b]), dtype=kinds[info["dtype"]]).reshape(info["shape"])
    return out


def load_model(folder, dtype=F):
    folder = Path(folder)
    cfg = json.loads((folder / "config.json").read_text())
    return cfg, {k: v.to(dtype) for k, v in read_safetensors(folder / "model.safetensors").items()}


# ------------------------------------------------------------------ small pieces

def unit_rms(x, eps):
    return x / torch.sqrt((x * x).mean(dim=-1, keepdim=True) + eps)


def rms_norm(x, w, eps):
    return unit_rms(x, eps) * w


def silu(z):
    return z * torch.sigmoid(z)


def rotate_neighbours(x, positions, base, dims):
    """x [T, heads, n]: coordinates (2i, 2i + 1), i < dims/2, of each head turned by position * base^(-2i/dims)."""
    i = torch.arange(dims // 2, dtype=torch.float64)
    a = positions.double()[:, None] * (float(base) ** (-2.0 * i / max(dims, 1)))[None, :]
    c, s = torch.cos(a)[:, None, :].to(x.dtype), torch.sin(a)[:, None, :].to(x.dtype)
    u, v = x[..., 0:dims:2], x[..., 1:dims:2]
    return torch.cat([torch.stack([u * c - v * s, v * c + u * s], dim=-1).flatten(-2), x[..., dims:]], dim=-1)


def visible(T, size=None, keep_first=0):
    """[T, T] (query, key): no later key; with `size`, only the last `size` keys and the first keep_first."""
    i, j = torch.arange(T)[:, None], torch.arange(T)[None, :]
    seen = j <= i
    return seen if size is None else seen & ((i - j < size) | (j < keep_first))


def attend(q, k, v, scale, seen, softcap=None):
    """q [T, H, d], k [T, G, d], v [T, G, dv]; query head h reads key/value head h // (H / G)."""
    r = q.shape[1] // k.shape[1]
    k, v = k.repeat_interleave(r, dim=1), v.repeat_interleave(r, dim=1)
    s = torch.einsum("thd,shd->hts", q, k) * scale
    if softcap:
        s = softcap * torch.tanh(s / softcap)
    p = torch.softmax(s.masked_fill(~seen, float("-inf")), dim=-1)
    return torch.einsum("hts,shd->thd", p, v)


def temperature(positions, coef, every, dtype):
    return (1.0 + coef * torch.log(torch.floor((positions.double() + 1.0) / every) + 1.0)).to(dtype)


# ------------------------------------------------------------------ mixers

def windowed_attention(h, w, pre, m, eps, positions):
    T = h.shape[0]
    H, G, d, dv = m["heads"], m["kv_heads"], m["dim"], m["vdim"]
    q, k, v = ((h @ w[f"{pre}.{n}"].T).view(T, heads, size) for n, heads, size in (("q", H, d), ("k", G, d), ("v", G, dv)))
    rot = m.get("rot")
    if rot and rot["dims"]:
        q, k = (rotate_neighbours(x, positions, rot["base"], rot["dims"]) for x in (q, k))
    mask = m.get("mask") or {}
    seen = visible(T, mask.get("size"), mask.get("keep_first", 0))
    o = attend(unit_rms(q, eps), unit_rms(k, eps), v, m["scale"], seen)
    o = o * torch.sigmoid(h @ w[pre + ".g"].T)[:, :, None]
    return o.reshape(T, H * dv) @ w[pre + ".o"].T


def tempered_attention(h, w, pre, m, eps, positions):
    T = h.shape[0]
    H, G, d, dv = m["heads"], m["kv_heads"], m["dim"], m["vdim"]
    q = rms_norm((h @ w[pre + ".q"].T).view(T, H, d), w[pre + ".q.norm"], eps)
    k = rms_norm((h @ w[pre + ".k"].T).view(T, G, d), w[pre + ".k.norm"], eps)
    v = (h @ w[pre + ".v"].T).view(T, G, dv)
    t = m.get("q_temp")
    if t:
        q = q * temperature(positions, t["coef"], t["every"], q.dtype)[:, None, None]
    o = attend(q, k, v, m["scale"], visible(T), m.get("softcap"))
    o = o * torch.sigmoid(h @ w[pre + ".g"].T)[:, :, None]
    return o.reshape(T, H * dv) @ w[pre + ".o"].T


def bonus_recurrence(r, k, v, decay, u):
    """r, k, decay [T, H, d], v [T, H, dv], u [H, d]: o_t = (S + diag(u) k_t v_t^T)^T r_t, then
    S <- diag(decay_t) S + k_t v_t^T, from S = 0."""
    T, H, d = r.shape
    S, o = torch.zeros(H, d, v.shape[-1], dtype=r.dtype), torch.zeros_like(v)
    for t in range(T):
        kv = k[t][:, :, None] * v[t][:, None, :]
        o[t] = torch.einsum("hde,hd->he", S + u[:, :, None] * kv, r[t])
        S = decay[t][:, :, None] * S + kv
    return o


def time_mixing(h, w, pre, m, eps):
    T = h.shape[0]
    H, d = m["heads"], m["dim"]
    before = torch.cat([torch.zeros_like(h[:1]), h[:-1]])
    mix = {s: h + (before - h) * w[f"{pre}.mu.{s}"] for s in "rkvgw"}
    r, k, v = ((mix[s] @ w[f"{pre}.{s}"].T).view(T, H, d) for s in "rkv")
    gate = silu(mix["g"] @ w[pre + ".g"].T)
    z = torch.tanh(mix["w"] @ w[pre + ".w1"].T) @ w[pre + ".w2"].T + w[pre + ".w0"]
    o = bonus_recurrence(r, k, v, torch.exp(-torch.exp(z)).view(T, H, d), w[pre + ".u"])
    return (unit_rms(o, eps).reshape(T, H * d) * w[pre + ".norm"] * gate) @ w[pre + ".o"].T


def side_by_side(h, w, pre, m, eps, positions):
    left = tempered_attention(h, w, pre + ".left", m["left"], eps, positions)
    right = time_mixing(h, w, pre + ".right", m["right"], eps)
    return 0.5 * (rms_norm(left, w[pre + ".left.out"], eps) + rms_norm(right, w[pre + ".right.out"], eps))


# ------------------------------------------------------------------ feed-forward

def gated_unit(h, w, pre):
    return (silu(h @ w[pre + ".gate"].T) * (h @ w[pre + ".up"].T)) @ w[pre + ".down"].T


def choose(s, correction, top, groups=None):
    """s [T, E] scores -> indices [T, top]: the largest s + correction among the experts of the best groups
    (a group's score: the sum of its two largest)."""
    c = s + correction
    if groups:
        T, E = c.shape
        by = c.view(T, groups["count"], E // groups["count"])
        best = by.topk(min(2, by.shape[-1]), dim=-1).values.sum(dim=-1).topk(groups["keep"], dim=-1).indices
        kept = torch.zeros(T, groups["count"], dtype=torch.bool).scatter_(1, best, True)
        c = by.masked_fill(~kept[:, :, None], float("-inf")).view(T, E)
    return c.topk(top, dim=-1).indices


def expert_mixture(h, w, pre, m):
    router = m["router"]
    s = torch.sigmoid(h @ w[pre + ".router"].T)
    idx = choose(s, w[pre + ".correction"], router["top"], router.get("groups"))
    wt = torch.gather(s, 1, idx)
    wt = wt / (wt.sum(dim=-1, keepdim=True) + 1e-20)
    out = torch.zeros_like(h)
    for e in range(router["experts"]):
        rows, place = (idx == e).nonzero(as_tuple=True)
        if rows.numel():
            out[rows] += wt[rows, place][:, None] * gated_unit(h[rows], w, f"{pre}.e{e}")
    if m.get("shared"):
        out = out + torch.sigmoid(h @ w[pre + ".shared.sg"].T) * gated_unit(h, w, pre + ".shared")
    return out


# ------------------------------------------------------------------ model

def runs(cfg):
    """(layer, pass of the loop that begins right before it or None) in the order the layers run."""
    n, loop = len(cfg["layers"]), cfg.get("loop")
    if not loop:
        return [(i, None) for i in range(n)]
    a, b = loop["start"], loop["stop"]
    out = [(i, None) for i in range(a)]
    for t in range(loop["times"]):
        out += [(i, t if i == a else None) for i in range(a, b)]
    return out + [(i, None) for i in range(b, n)]


def loop_entry(x, x0, w, t):
    return torch.cat([x, x0], dim=-1) @ w["loop.in"].T + w["loop.step"][t]


def forward(cfg, w, tokens, layers_out=None):
    """Logits [T, vocab] of one whole sequence. `layers_out`, a list, receives the stream after every
    layer run."""
    eps = cfg["norm"]["eps"]
    tokens = torch.as_tensor(tokens, dtype=torch.long)
    positions = torch.arange(tokens.shape[0])
    x = x0 = w["embed"][tokens]
    for i, t in runs(cfg):
        if t is not None:
            x = loop_entry(x, x0, w, t)
        L, p = cfg["layers"][i], f"l{i}"
        h = rms_norm(x, w[p + ".norm1"], eps)
        if L["type"] == "parallel":
            update = side_by_side(h, w, p + ".mix", L["mixer"], eps, positions)
        else:
            update = windowed_attention(h, w, p + ".mix", L["mixer"], eps, positions)
        if L.get("mlp") is not None:
            update = update + expert_mixture(rms_norm(x, w[p + ".norm2"], eps), w, p + ".mlp", L["mlp"])
        x = x + update
        if layers_out is not None:
            layers_out.append(x.clone())
    return rms_norm(x, w["final.norm"], eps) @ w["head"].T


def greedy(cfg, w, prompt, n_new):
    toks = list(prompt)
    for _ in range(n_new):
        toks.append(int(forward(cfg, w, toks)[-1].argmax()))
    return toks[len(prompt):]
