"""A plain, slow implementation of the Kopatar design: float64, no cache, whole sequences, one function per mechanism.

Written from the design's equations and sharing no code with the package. ``cfg`` is the configuration as a plain
dict (the keys of config.json), ``w`` maps tensor names to float64 tensors.

    block      x <- x + mixer(norm(x)); x <- x + ff(norm(x)), norm an RMS norm with a plain weight per coordinate
    mixers     "channel_delta": a gated delta rule whose decay is a number per head AND key channel, behind short
               causal convolutions, with a low-rank sigmoid gate on the normed heads;
               "retention": a linear recurrence with a fixed decay per head and rotated queries and keys;
               "parallel": softmax attention (normed heads, a window, a gate on every channel of the heads) beside
               a Mamba-2 recurrence (one convolution over x, B and C, a scalar decay per head, a skip D), weighted sum
    ff         W_down act(W_up h), act the xIELU activation with two learned numbers
    loop       layers start .. stop-1 run several times; ahead of pass t the stream takes the embedding output (not
               ahead of the first) and the learned vector of that pass
    head       the embedding table
"""
import json
import os
import struct

import torch

F64 = torch.float64


def rms(x, eps):
    """x divided by its root mean square over the last axis (eps inside the root)."""
    return x / torch.sqrt((x * x).mean(dim=-1, keepdim=True) + eps)


def silu(x):
    return x * torch.sigmoid(x)


def softplus(x):
    return torch.nn.functional.softplus(x, threshold=200.0)


def unit(x, eps=1e-6):
    return x / torch.sqrt((x * x).sum(dim=-1, keepdim=True) + eps)


def short_conv(x, taps, bias=None):
    """x [T, C], taps [C, K]: y_t = sum_j taps[:, K-1-j] x_(t-j) (+ bias), zeros before the start."""
    T, C = x.shape
    K = taps.shape[1]
    padded = torch.cat([x.new_zeros((K - 1, C)), x], dim=0)
    y = x.new_zeros((T, C)) if bias is None else bias.expand(T, C)
    for j in range(K):
        y = y + padded[j: j + T] * taps[:, j]
    return y


def channel_delta(h, m, w, p, eps):
    """Per head with its decay vector g: S <- diag(g) S; u = beta (v - S^T k); S <- S + k u^T; o = S^T q."""
    T = h.shape[0]
    H, G, d, dv = m["heads"], m["kv_heads"], m["dim"], m["vdim"]
    conv = lambda role, n, width: silu(short_conv(h @ w[p + role].T, w[p + role + ".conv"])).view(T, n, width)
    q, k, v = unit(conv("q", G, d)) * d ** -0.5, unit(conv("k", G, d)), conv("v", H, dv)
    beta = torch.sigmoid(h @ w[p + "b"].T)
    a = (h @ w[p + "a1"].T) @ w[p + "a2"].T + w[p + "dt_bias"]
    g = torch.exp(-torch.exp(w[p + "A_log"])[:, None] * softplus(a).view(T, H, d))
    rep = H // G
    q, k = q.repeat_interleave(rep, dim=1), k.repeat_interleave(rep, dim=1)
    S = h.new_zeros((H, d, dv))
    out = h.new_zeros((T, H, dv))
    for t in range(T):
        S = g[t][:, :, None] * S
        u = beta[t][:, None] * (v[t] - torch.einsum("hij,hi->hj", S, k[t]))
        S = S + k[t][:, :, None] * u[:, None, :]
        out[t] = torch.einsum("hij,hi->hj", S, q[t])
    gate = torch.sigmoid((h @ w[p + "g1"].T) @ w[p + "g2"].T)
    return ((rms(out, eps) * w[p + "norm"]).reshape(T, H * dv) * gate) @ w[p + "o"].T


def rotate_halves(x, positions, dims, base):
    """x [T, heads, width]: entry i of a head is paired with entry i + dims/2, for i < dims/2; the rest passes."""
    i = torch.arange(dims // 2, dtype=F64)
    ang = positions.to(F64)[:, None] * (float(base) ** (-2.0 * i / max(dims, 1)))[None, :]
    c, s = ang.cos()[:, None, :], ang.sin()[:, None, :]
    u, v = x[..., : dims // 2], x[..., dims // 2: dims]
    out = x.clone()
    out[..., : dims // 2] = u * c - v * s
    out[..., dims // 2: dims] = v * c + u * s
    return out


def retention(h, m, w, p, eps, positions):
    """Per head: S <- decay S + k v^T; o = S^T q with rotated q and k, k scaled by dim^-1/2."""
    T = h.shape[0]
    H, d, dv = m["heads"], m["dim"], m["vdim"]
    q, k, v = (h @ w[p + "q"].T).view(T, H, d), (h @ w[p + "k"].T).view(T, H, d), (h @ w[p + "v"].T).view(T, H, dv)
    q = rotate_halves(q, positions, m["rot"]["dims"], m["rot"]["base"])
    k = rotate_halves(k, positions, m["rot"]["dims"], m["rot"]["base"]) * d ** -0.5
    decay = torch.tensor(m["decay"], dtype=F64)
    S = h.new_zeros((H, d, dv))
    out = h.new_zeros((T, H, dv))
    for t in range(T):
        S = decay[:, None, None] * S + k[t][:, :, None] * v[t][:, None, :]
        out[t] = torch.einsum("hij,hi->hj", S, q[t])
    return (rms(out, eps).reshape(T, H * dv) * silu(h @ w[p + "g"].T)) @ w[p + "o"].T


def gated_window_attention(h, m, w, p, eps, positions):
    """Softmax attention: heads of q and k normed with a shared weight, a window, a sigmoid gate per channel."""
    T = h.shape[0]
    H, G, d, dv = m["heads"], m["kv_heads"], m["dim"], m["vdim"]
    q = rms((h @ w[p + "q"].T).view(T, H, d), eps) * w[p + "q.norm"]
    k = rms((h @ w[p + "k"].T).view(T, G, d), eps) * w[p + "k.norm"]
    v = (h @ w[p + "v"].T).view(T, G, dv)
    rep = H // G
    k, v = k.repeat_interleave(rep, dim=1), v.repeat_interleave(rep, dim=1)
    s = torch.einsum("ihd,jhd->hij", q, k) * float(m["scale"])
    dist = positions[:, None] - positions[None, :]
    seen = dist >= 0
    size = (m.get("mask") or {}).get("size", 0)
    if size:
        seen = seen & (dist < size)
    a = torch.softmax(s.masked_fill(~seen[None], float("-inf")), dim=-1)
    o = torch.einsum("hij,jhd->ihd", a, v).reshape(T, H * dv)
    return (o * torch.sigmoid(h @ w[p + "g"].T)) @ w[p + "o"].T


def mamba2(h, m, w, p, eps):
    """Per head: S <- exp(-exp(A_log) dt) S + dt B x^T; y = S^T C + D x; gated by silu(z), then normed in parts."""
    T = h.shape[0]
    H, dv, N, G = m["heads"], m["vdim"], m["state"], m["groups"]
    inner = H * dv
    z, xbc, dt = torch.split(h @ w[p + "in"].T, [inner, inner + 2 * G * N, H], dim=1)
    xbc = silu(short_conv(xbc, w[p + "conv"], w[p + "conv.b"]))
    x, B, C = torch.split(xbc, [inner, G * N, G * N], dim=1)
    x, B, C = x.reshape(T, H, dv), B.reshape(T, G, N), C.reshape(T, G, N)
    rep = H // G
    B, C = B.repeat_interleave(rep, dim=1), C.repeat_interleave(rep, dim=1)
    dt = softplus(dt + w[p + "dt_bias"])
    decay = torch.exp(-torch.exp(w[p + "A_log"]) * dt)
    S = h.new_zeros((H, N, dv))
    y = h.new_zeros((T, H, dv))
    for t in range(T):
        S = decay[t][:, None, None] * S + dt[t][:, None, None] * B[t][:, :, None] * x[t][:, None, :]
        y[t] = torch.einsum("hij,hi->hj", S, C[t]) + w[p + "D"][:, None] * x[t]
    y = y.reshape(T, inner) * silu(z)
    y = rms(y.view(T, m["norm_groups"], -1), eps).reshape(T, inner) * w[p + "norm"]
    return y @ w[p + "o"].T


def parallel_mixer(h, m, w, p, eps, positions):
    return float(m["left_scale"]) * gated_window_attention(h, m["left"], w, p + "left.", eps, positions) \
        + float(m["right_scale"]) * mamba2(h, m["right"], w, p + "right.", eps)


def xielu(z, act):
    """z > 0: softplus(p) z^2 + z / 2; z <= 0: (1/2 + softplus(q)) (exp(z) - 1 - z) + z / 2."""
    up, down = softplus(act[0]), 0.5 + softplus(act[1])
    return torch.where(z > 0, up * z * z, down * (torch.expm1(z.clamp(max=0.0)) - z.clamp(max=0.0))) + 0.5 * z


def feed_forward(h, w, p):
    return xielu(h @ w[p + "up"].T, w[p + "act"]) @ w[p + "down"].T


def mixer(h, layer, w, p, eps, positions):
    m = layer["mixer"]
    if layer["type"] == "channel_delta":
        return channel_delta(h, m, w, p, eps)
    if layer["type"] == "retention":
        return retention(h, m, w, p, eps, positions)
    assert layer["type"] == "parallel"
    return parallel_mixer(h, m, w, p, eps, positions)


def layer_order(cfg):
    """(layer, pass number where a pass over the looped stretch begins, else None) in the order they run."""
    n = len(cfg["layers"])
    loop = cfg.get("loop")
    if not loop:
        return [(i, None) for i in range(n)]
    a, b = loop["start"], loop["stop"]
    middle = [(i, t if i == a else None) for t in range(loop["times"]) for i in range(a, b)]
    return [(i, None) for i in range(a)] + middle + [(i, None) for i in range(b, n)]


def forward(tokens, cfg, w, residuals=None):
    """Logits [T, vocab] of one sequence. ``residuals`` (a list) receives the stream after every layer run."""
    eps = float(cfg["norm"]["eps"])
    positions = torch.arange(len(tokens))
    x0 = w["embed"][torch.as_tensor(tokens, dtype=torch.long)]
    x = x0
    for i, begins in layer_order(cfg):
        if begins is not None:
            if begins > 0:
                x = x + x0
            x = x + w["loop.step"][begins]
        p, layer = f"l{i}.", cfg["layers"][i]
        x = x + mixer(rms(x, eps) * w[p + "norm1"], layer, w, p + "mix.", eps, positions)
        if layer.get("mlp") is not None:
            x = x + feed_forward(rms(x, eps) * w[p + "norm2"], w, p + "mlp.")
        if residuals is not None:
            residuals.append(x)
    return (rms(x, eps) * w["final.norm"]) @ w["embed"].T


def load_model_dir(path: str):
    """(cfg, tensors as float64) of a folder with config.json and model.safetensors (own reader: 8-byte length,
    JSON header, data)."""
    with open(os.path.join(path, "config.json")) as f:
        cfg = json.load(f)
    with open(os.path.join(path, "model.safetensors"), "rb") as f:
        (n,) = struct.unpack("<Q", f.read(8))
        header = json.loads(f.read(n))
        data = f.read()
    kinds = {"BF16": torch.bfloat16, "F32": torch.float32, "F16": torch.float16, "I32": torch.int32, "I64": torch.int64}
    w = {}
    for name, info in header.items():
        if name == "__metadata__":
            continue
        lo, hi = info["data_offsets"]
        t = torch.frombuffer(bytearray(data[lo:hi]), dtype=kinds[info["dtype"]]).reshape(info["shape"])
        w[name] = t.to(F64) if t.is_floating_point() else t
    return cfg, w
