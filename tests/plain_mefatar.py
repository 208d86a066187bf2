"""A plain, slow implementation of the Mefatar decoder on the CPU, written from the design's
equations, one function per mechanism. It shares no code with the library: whole sequences only,
no cache, no batching, Python loops over time for the recurrences. The tests compare the engine
with it.

Notation: a sequence of T tokens, width D. Softmax attention: H query heads, G key/value heads, key
size d, value size dv. Gated linear attention: H heads, key size d, value size dv, state S [d, dv] a
head. Recurrent unit: C channels in B blocks. Every function takes float32 (or float64) tensors.
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

def rms_norm(x, w, eps):
    return x / torch.sqrt((x * x).mean(dim=-1, keepdim=True) + eps) * w


def silu(z):
    return z * torch.sigmoid(z)


def gelu_tanh(z):
    return 0.5 * z * (1.0 + torch.tanh(math.sqrt(2.0 / math.pi) * (z + 0.044715 * z ** 3)))


def softplus(z):
    return torch.where(z > 20.0, z, torch.log1p(torch.exp(torch.clamp(z, max=20.0))))


def causal_conv(u, w, b=None):
    """y_t = b + sum_j w[:, j] u_(t - taps + 1 + j) a channel, zeros before the start. u [T, C], w [C, taps]."""
    T, taps = u.shape[0], w.shape[1]
    padded = torch.cat([torch.zeros(taps - 1, u.shape[1], dtype=u.dtype), u])
    y = torch.zeros_like(u)
    for j in range(taps):
        y = y + padded[j:j + T] * w[:, j]
    return y if b is None else y + b


def frequencies(base, dims, scaling=None):
    """f_i = base^(-2i/dims), i < dims/2. With `scaling` (factor, low, high, original), by the number of
    turns n_i = original f_i / (2 pi) over the original context: n_i > high keeps f_i, n_i < low gets
    f_i / factor, and between them s f_i + (1 - s) f_i / factor with s = (n_i - low) / (high - low)."""
    i = torch.arange(dims // 2, dtype=torch.float64)
    f = float(base) ** (-2.0 * i / dims)
    if scaling is not None:
        turns = float(scaling["original"]) * f / (2.0 * math.pi)
        low, high, slow = float(scaling["low"]), float(scaling["high"]), f / float(scaling["factor"])
        s = (turns - low) / (high - low) if high != low else torch.zeros_like(f)
        f = torch.where(turns > high, f, torch.where(turns < low, slow, s * f + (1.0 - s) * slow))
    return f


def rotate_neighbours(x, positions, base, dims, scaling=None):
    """x [T, heads, n]: coordinates (2i, 2i + 1), i < dims/2, of each head turned by position * f_i."""
    a = positions.double()[:, None] * frequencies(base, dims, scaling)[None, :]
    c, s = torch.cos(a)[:, None, :].to(x.dtype), torch.sin(a)[:, None, :].to(x.dtype)
    u, v = x[..., 0:dims:2], x[..., 1:dims:2]
    return torch.cat([torch.stack([u * c - v * s, v * c + u * s], dim=-1).flatten(-2), x[..., dims:]], dim=-1)


def sink_softmax(scores, sink):
    """scores [H, T, T] (query, key), sink [H]: causal weights exp(s_j) / (exp(sink) + sum_j exp(s_j))."""
    T = scores.shape[-1]
    s = scores.masked_fill(torch.ones(T, T, dtype=torch.bool).triu(1), float("-inf"))
    top = torch.maximum(s.amax(dim=-1, keepdim=True), sink[:, None, None])
    e = torch.exp(s - top)
    return e / (e.sum(dim=-1, keepdim=True) + torch.exp(sink[:, None, None] - top))


# ------------------------------------------------------------------ mixers

def softmax_attention(h, w, pre, m, eps, positions):
    T = h.shape[0]
    H, G, d, dv = m["heads"], m["kv_heads"], m["dim"], m["vdim"]
    q, k, v = (causal_conv(h @ w[f"{pre}.{n}"].T, w[f"{pre}.{n}.conv"]) for n in "qkv")
    q = rms_norm(q, w[pre + ".q.norm"], eps).view(T, H, d)          # over all heads at once
    k = rms_norm(k, w[pre + ".k.norm"], eps).view(T, G, d)
    v = v.view(T, G, dv)
    rot = m.get("rot")
    if rot and rot["dims"]:
        q, k = (rotate_neighbours(x, positions, rot["base"], rot["dims"], rot.get("scaling")) for x in (q, k))
    k, v = k.repeat_interleave(H // G, dim=1), v.repeat_interleave(H // G, dim=1)
    p = sink_softmax(torch.einsum("thd,shd->hts", q, k) * m["scale"], w[pre + ".sink"])
    o = torch.einsum("hts,shd->thd", p, v).reshape(T, H * dv)
    return (o * torch.sigmoid(h @ w[pre + ".g"].T)) @ w[pre + ".o"].T


def gated_linear_attention(h, w, pre, m, eps):
    T = h.shape[0]
    H, d, dv = m["heads"], m["dim"], m["vdim"]
    q = (h @ w[pre + ".q"].T).view(T, H, d) * d ** -0.5
    k = (h @ w[pre + ".k"].T).view(T, H, d)
    v = (h @ w[pre + ".v"].T).view(T, H, dv)
    z = (h @ w[pre + ".a1"].T) @ w[pre + ".a2"].T + w[pre + ".a2.b"]
    a = (torch.sigmoid(z) ** (1.0 / m["tau"])).view(T, H, d)
    S, o = torch.zeros(H, d, dv, dtype=h.dtype), torch.zeros(T, H, dv, dtype=h.dtype)
    for t in range(T):
        S = a[t][:, :, None] * S + k[t][:, :, None] * v[t][:, None, :]
        o[t] = torch.einsum("hde,hd->he", S, q[t])
    o = rms_norm(o, w[pre + ".norm"], eps).reshape(T, H * dv)
    return (o * silu(h @ w[pre + ".g"].T)) @ w[pre + ".o"].T


def side_by_side(h, w, pre, m, eps, positions):
    left = softmax_attention(h, w, pre + ".left", m["left"], eps, positions)
    right = gated_linear_attention(h, w, pre + ".right", m["right"], eps)
    return 0.5 * (rms_norm(left, w[pre + ".left.out"], eps) + rms_norm(right, w[pre + ".right.out"], eps))


def recurrent_unit(h, w, pre, m):
    T, B = h.shape[0], m["blocks"]
    y = gelu_tanh(h @ w[pre + ".y"].T + w[pre + ".y.b"])
    u = causal_conv(h @ w[pre + ".x"].T + w[pre + ".x.b"], w[pre + ".conv"], w[pre + ".conv.b"])
    ub = u.view(T, B, -1)
    r, i = (torch.sigmoid(torch.einsum("tbj,bkj->tbk", ub, w[f"{pre}.{n}"]) + w[f"{pre}.{n}.b"]).reshape(T, -1)
            for n in ("ra", "ri"))
    log_a = -8.0 * r * softplus(w[pre + ".lam"])
    a, x = torch.exp(log_a), torch.sqrt(-torch.expm1(2.0 * log_a)) * i * u
    S, out = torch.zeros_like(u[0]), torch.zeros_like(u)
    for t in range(T):
        S = a[t] * S + x[t]
        out[t] = S
    return (out * y) @ w[pre + ".o"].T


# ------------------------------------------------------------------ feed-forward and model

def gated_ff(h, w, pre):
    return (gelu_tanh(h @ w[pre + ".gate"].T) * (h @ w[pre + ".up"].T)) @ w[pre + ".down"].T


def runs(cfg):
    """The layers in the order they run: the loop's layers as often as it says, one after the other."""
    n, loop = len(cfg["layers"]), cfg.get("loop")
    if not loop:
        return list(range(n))
    a, b = loop["start"], loop["stop"]
    return list(range(a)) + list(range(a, b)) * loop["times"] + list(range(b, n))


def forward(cfg, w, tokens, layers_out=None):
    """Logits [T, vocab] of one whole sequence. `layers_out`, a list, receives the stream after every
    layer run."""
    eps = cfg["norm"]["eps"]
    tokens = torch.as_tensor(tokens, dtype=torch.long)
    positions = torch.arange(tokens.shape[0])
    x = w["embed"][tokens]
    for i in runs(cfg):
        L, p = cfg["layers"][i], f"l{i}"
        h = rms_norm(x, w[p + ".norm1"], eps)
        if L["type"] == "parallel":
            a = side_by_side(h, w, p + ".mix", L["mixer"], eps, positions)
        else:
            a = recurrent_unit(h, w, p + ".mix", L["mixer"])
        x = x + w[p + ".ls1"] * a
        if L.get("mlp") is not None:
            x = x + w[p + ".ls2"] * gated_ff(rms_norm(x, w[p + ".norm2"], eps), w, p + ".mlp")
        if layers_out is not None:
            layers_out.append(x.clone())
    return rms_norm(x, w["final.norm"], eps) @ w["embed"].T


def greedy(cfg, w, prompt, n_new):
    toks = list(prompt)
    for _ in range(n_new):
        toks.append(int(forward(cfg, w, toks)[-1].argmax()))
    return toks[len(prompt):]
