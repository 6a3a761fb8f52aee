"""A plain, slow implementation of the Sumuvik design: float64, no cache, whole sequences, one function per mechanism.

Written from the design's equations and sharing no code with the package. ``cfg`` is the configuration as a plain
dict (the keys of config.json), ``w`` maps tensor names to float64 tensors.

    layer:   x <- x + mixer(norm_1(x)) + ff(norm_2(x))           (both branches read the same x)
    mixers:  grouped-query attention with biases, neighbouring pairs rotated by rescaled frequencies, a sliding window
             beside the first tokens of the sequence, one added to the softmax's denominator and one sigmoid gate per
             head; and a gated linear recurrence per channel (RG-LRU) behind a short convolution, beside a GELU branch
    ff:      clamped gated unit, dense or as routed experts (sigmoid scores, choice by score + correction within the
             best groups of experts, weights the scores over their sum) beside an expert that every token uses
"""
import json
import math
import os
import struct

import torch

F64 = torch.float64


def rms_norm(x, weight, eps):
    return x / torch.sqrt((x * x).mean(dim=-1, keepdim=True) + eps) * weight


def frequencies(dims, base, scaling=None):
    """Angle of pair i at position p is p * f[i]. ``scaling`` (factor, low, high, original): a pair whose wavelength is
    shorter than original / high keeps its frequency, one longer than original / low has it divided by factor, and
    between the two the frequency is mixed linearly in original / wavelength."""
    out = []
    for i in range(dims // 2):
        f = float(base) ** (-2.0 * i / dims)
        if scaling:
            factor, low, high, original = (float(scaling[k]) for k in ("factor", "low", "high", "original"))
            wave = 2.0 * math.pi / f
            if wave > original / low:
                f = f / factor
            elif wave >= original / high:
                s = (original / wave - low) / (high - low)
                f = (1.0 - s) * f / factor + s * f
        out.append(f)
    return torch.tensor(out, dtype=F64)


def rotate_pairs(x, positions, dims, base, scaling=None):
    """x [tokens, heads, width]: entries 2i and 2i + 1 of every head's first ``dims`` entries are turned together."""
    if dims == 0:
        return x
    ang = positions.to(F64)[:, None] * frequencies(dims, base, scaling)[None, :]
    c, s = ang.cos()[:, None, :], ang.sin()[:, None, :]
    u, v = x[..., 0:dims:2], x[..., 1:dims:2]
    out = x.clone()
    out[..., 0:dims:2] = u * c - v * s
    out[..., 1:dims:2] = v * c + u * s
    return out


def visible(n, window, keep_first):
    """[query, key]: causal, and with a window only its keys or the first ``keep_first`` of the sequence."""
    i = torch.arange(n)[:, None]
    j = torch.arange(n)[None, :]
    seen = j <= i
    if window > 0:
        seen = seen & ((i - j < window) | (j < keep_first))
    return seen


def softmax_plus_one(s, seen):
    """exp(s_j) / (1 + sum exp(s_j)) over the visible keys."""
    s = s.masked_fill(~seen, float("-inf"))
    m = s.amax(dim=-1, keepdim=True).clamp(min=0.0)
    e = torch.exp(s - m)
    return e / (torch.exp(-m) + e.sum(dim=-1, keepdim=True))


def attention(h, m, w, p):
    T = h.shape[0]
    H, G, d, dv = m["heads"], m["kv_heads"], m["dim"], m["vdim"]
    pos = torch.arange(T)
    q = (h @ w[p + "q"].T + w[p + "q.b"]).view(T, H, d)
    k = (h @ w[p + "k"].T + w[p + "k.b"]).view(T, G, d)
    v = (h @ w[p + "v"].T + w[p + "v.b"]).view(T, G, dv)
    rot = m.get("rot") or {}
    turn = (rot.get("dims", 0), rot.get("base", 1.0), rot.get("scaling"))
    q, k = rotate_pairs(q, pos, *turn), rotate_pairs(k, pos, *turn)
    k, v = k.repeat_interleave(H // G, dim=1), v.repeat_interleave(H // G, dim=1)
    mask = m.get("mask") or {}
    s = torch.einsum("ihd,jhd->hij", q, k) * m["scale"]
    a = softmax_plus_one(s, visible(T, mask.get("size", 0), mask.get("keep_first", 0))[None])
    o = torch.einsum("hij,jhd->ihd", a, v)
    o = o * torch.sigmoid(h @ w[p + "g"].T)[:, :, None]
    return o.reshape(T, H * dv) @ w[p + "o"].T


def gelu_tanh(z):
    return 0.5 * z * (1.0 + torch.tanh(math.sqrt(2.0 / math.pi) * (z + 0.044715 * z ** 3)))


def softplus(z):
    return torch.clamp(z, min=0) + torch.log1p(torch.exp(-z.abs()))


def short_conv(x, taps, bias):
    """x [tokens, channels], taps [channels, K], the last tap for the current token; zeros before the start."""
    T, K = x.shape[0], taps.shape[1]
    y = bias.expand(T, -1).clone()
    for lag in range(min(K, T)):
        y[lag:] = y[lag:] + taps[:, K - 1 - lag] * x[: T - lag]
    return y


def block_diagonal(u, mats, bias):
    """u [tokens, blocks * n]; block b of it through mats[b] [n, n]."""
    B, n = mats.shape[0], mats.shape[1]
    return torch.cat([u[:, b * n:(b + 1) * n] @ mats[b].T + bias[b] for b in range(B)], dim=1)


def linear_recurrence(u, r, i, lam):
    """S_t = a S_(t-1) + sqrt(1 - a^2) i u with log a = -8 r softplus(lam), from zero."""
    log_a = -8.0 * r * softplus(lam)
    a, b = torch.exp(log_a), torch.sqrt(-torch.expm1(2.0 * log_a))
    S, out = torch.zeros_like(u[0]), []
    for t in range(u.shape[0]):
        S = a[t] * S + b[t] * i[t] * u[t]
        out.append(S)
    return torch.stack(out)


def rglru(h, m, w, p):
    y = gelu_tanh(h @ w[p + "y"].T + w[p + "y.b"])
    u = short_conv(h @ w[p + "x"].T + w[p + "x.b"], w[p + "conv"], w[p + "conv.b"])
    r = torch.sigmoid(block_diagonal(u, w[p + "ra"], w[p + "ra.b"]))
    i = torch.sigmoid(block_diagonal(u, w[p + "ri"], w[p + "ri.b"]))
    return (linear_recurrence(u, r, i, w[p + "lam"]) * y) @ w[p + "o"].T


def gated_unit(h, w, p, limit):
    g = torch.clamp(h @ w[p + "gate"].T, max=limit)
    u = torch.clamp(h @ w[p + "up"].T, -limit, limit)
    return (g * torch.sigmoid(1.702 * g) * (u + 1.0)) @ w[p + "down"].T


def route(scores, correction, top, groups, scale):
    """One token's scores -> [(expert, weight)]. Groups of neighbours are ranked by the sum of their two largest choice
    scores; experts of the best ``keep`` groups compete."""
    n = scores.shape[0]
    choice = scores + correction
    allowed = list(range(n))
    if groups:
        size = n // groups["count"]
        rank = []
        for g in range(groups["count"]):
            two = sorted(choice[g * size:(g + 1) * size].tolist(), reverse=True)[:2]
            rank.append((-sum(two), g))
        best = {g for _, g in sorted(rank)[: groups["keep"]]}
        allowed = [e for e in allowed if e // size in best]
    chosen = sorted(allowed, key=lambda e: (-float(choice[e]), e))[:top]
    total = sum(float(scores[e]) for e in chosen) + 1e-20
    return [(e, float(scores[e]) / total * scale) for e in chosen]


def experts(h, f, w, p):
    r = f["router"]
    s = torch.sigmoid(h @ w[p + "router"].T)
    out = torch.zeros_like(h)
    for t in range(h.shape[0]):
        for e, weight in route(s[t], w[p + "correction"], r["top"], r.get("groups"), r.get("scale", 1.0)):
            out[t] += weight * gated_unit(h[t:t + 1], w, f"{p}e{e}.", f["expert"]["limit"])[0]
    if f.get("shared"):
        out = out + gated_unit(h, w, p + "shared.", f["shared"]["limit"])
    return out


def feed_forward(h, f, w, p):
    return gated_unit(h, w, p, f["limit"]) if f["kind"] == "dense" else experts(h, f, w, p)


MIXERS = {"attention": attention, "rglru": rglru}


def forward(tokens, cfg, w, residuals=None):
    """Logits [tokens, vocab]; ``residuals`` (a list) gets the stream after every layer."""
    eps = cfg["norm"]["eps"]
    x = w["embed"][torch.as_tensor(tokens)] * cfg["embedding"]["scale"]
    for n, layer in enumerate(cfg["layers"]):
        p = f"l{n}."
        y = MIXERS[layer["type"]](rms_norm(x, w[p + "norm1"], eps), layer["mixer"], w, p + "mix.")
        if layer.get("mlp") is not None:
            y = y + feed_forward(rms_norm(x, w[p + "norm2"], eps), layer["mlp"], w, p + "mlp.")
        x = x + y
        if residuals is not None:
            residuals.append(x.clone())
    return rms_norm(x, w["final.norm"], eps) @ w["head"].T


def load_model_dir(folder):
    """(cfg, weights in float64) of a model folder: config.json and model.safetensors."""
    with open(os.path.join(folder, "config.json")) as f:
        cfg = json.load(f)
    with open(os.path.join(folder, "model.safetensors"), "rb") as f:
        head = json.loads(f.read(struct.unpack("<Q", f.read(8))[0]))
        data = bytearray(f.read())
    kinds = {"BF16": torch.bfloat16, "F32": torch.float32, "F16": torch.float16, "I32": torch.int32}
    w = {}
    for name, e in head.items():
        if name != "__metadata__":
            a, b = e["data_offsets"]
            w[name] = torch.frombuffer(data[a:b], dtype=kinds[e["dtype"]]).reshape(e["shape"]).to(F64)
    return cfg, w
