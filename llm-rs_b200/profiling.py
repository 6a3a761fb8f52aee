"""Where a step's time goes: every kernel class timed with CUDA events, with the bytes it has to move and the
flops it has to do, and what fraction of the device's peaks that is.

The reference's counterpart is its tracing (``RUST_LOG``, the dump of the first operators of a pass,
llm-core/src/backends/candle.rs:1102-1109) and the timings its command-line tools print
(llm-cli/src/bin/run_model.rs:131-150). Here ``Profiler`` wraps the kernel entry points of ``ops`` while it is
active: every call is bracketed by two CUDA events on the launching stream and by an NVTX range (so that a
timeline tool shows the same names), and classed by kernel and shape. It is meant for eager steps (a replayed
CUDA graph launches nothing through ``ops``): the callers switch graphs off while they profile. Timings taken
this way are serialised launch by launch; they show shares and per-kernel rooflines, not the step's time.

    with Profiler(hbm_gbs=6550, tflops=1660) as prof:
        runner.step(entries)
    print(prof.report())
"""
from __future__ import annotations

import math
from typing import Callable, Dict, List, Optional, Tuple

import torch

from . import ops


def _nbytes(*tensors) -> int:
    return sum(t.numel() * t.element_size() for t in tensors if isinstance(t, torch.Tensor))


# What each wrapped entry point must read and write at the least (bytes) and compute (flops), from its arguments.
def _cost_gemm(x, w, *a, **k) -> Tuple[str, int, float]:
    tokens, K = x.shape
    n = w.size(0)
    width = n // 2 if k.get("epilogue") == "silu_mul" else n
    return f"{n}x{K}", _nbytes(x, w) + tokens * width * 2, 2.0 * tokens * n * K


def _cost_qkv(x, w, q_out, *a, **k):
    tokens, K = x.shape
    return f"{w.size(0)}x{K}", _nbytes(x, w) + tokens * w.size(0) * 2, 2.0 * tokens * w.size(0) * K


def _cost_gemm_f32(x, w, *a, **k):
    return f"{w.size(0)}x{w.size(1)}", _nbytes(x, w) + x.size(0) * w.size(0) * 4, 2.0 * x.size(0) * w.size(0) * w.size(1)


def _cost_library(x, w, *a, **k):
    return f"{w.size(0)}x{w.size(1)}", _nbytes(x, w) + x.size(0) * w.size(0) * 2, 2.0 * x.size(0) * w.size(0) * w.size(1)


def _cost_attn_decode(q, out, cache, dec_reqs, n_dec, q_start, cached_len, block_table, scratch, max_splits, split_keys,
                      n_q_heads, n_kv_heads, head_dim, page_size, window, scale, **k):
    # The keys are counted on the device and read when the report is made: a read here would make the host wait for
    # the device, and the next launch's preparation on the host would then show up as that kernel's time.
    keys = (cached_len[dec_reqs[:n_dec].long()] + 1).clamp(max=window if window > 0 else 1 << 30).sum()
    per_key, fixed = 2 * n_kv_heads * head_dim * cache.element_size(), _nbytes(q, out)
    return (f"{n_dec} requests", lambda: int(keys) * per_key + fixed, lambda: 4.0 * int(keys) * n_q_heads * head_dim)


def _cost_attn_prefill(q, out, cache, tiles, n_tiles, q_start, n_new, cached_len, block_table, n_q_heads, n_kv_heads,
                       head_dim, page_size, window, scale, **k):
    n, c = n_new.double(), cached_len.double()
    pairs = (n * c + n * (n + 1) / 2).sum()             # (query, key) pairs a causal portion sees
    keys, tokens = (n + c).sum(), int(q.size(0))
    per_key, fixed = 2 * n_kv_heads * head_dim * cache.element_size(), _nbytes(q, out)
    return (f"{tokens} tokens", lambda: int(float(keys) * per_key) + fixed,
            lambda: 4.0 * float(pairs) * n_q_heads * head_dim)


def _cost_rows(*tensors_from):
    def cost(*a, **k):
        ts = [a[i] for i in tensors_from if i < len(a) and isinstance(a[i], torch.Tensor)]
        return "", 2 * _nbytes(*ts), 0.0
    return cost


def _cost_grouped(x, w, out, tiles, n_tiles, src, w2=None, **k):
    rows, (G, N, K) = out.size(0), w.shape
    both = 2 if w2 is not None else 1
    # The weights of the experts that got a row are read at least once (rows dealt evenly: G (1 - (1 - 1/G)^rows) of
    # them in expectation); the rows are read and written.
    touched = G * (1.0 - (1.0 - 1.0 / G) ** max(rows, 1))
    return (f"{G}x{N}x{K}{' gated' if w2 is not None else ''}",
            int(touched * N * K * w.element_size() * both) + rows * (K * x.element_size() + N * out.element_size()),
            2.0 * rows * N * K * both)


def _cost_batched(x, w, out, **k):
    M, B, K = x.shape
    N = w.size(1)
    return f"{B}x{N}x{K}", _nbytes(w) + M * B * (K * x.element_size() + N * out.element_size()), 2.0 * M * B * N * K


def _cost_latent_attention(qa, q, gate, cache, table, ctx, out, n_heads, dn, dr, rank, page_size, window, scale, **k):
    pos = ctx.positions.double() + 1
    pairs = (pos.clamp(max=window) if window > 0 else pos).sum()       # (query, key) pairs, counted on the device
    c, n = ctx.cached_len.double(), ctx.n_new.double()
    keys = ((c.clamp(max=window) if window > 0 else c) + n).sum()      # cached rows that must be read at least once
    row = (rank + dr) * cache.element_size()
    return (f"{qa.size(0)} tokens", lambda: int(float(keys) * row) + 2 * _nbytes(qa),
            lambda: 2.0 * float(pairs) * n_heads * (2 * rank + dr))


def _cost_latent_prefill(qa, q, gate, cache, table, ctx, tiles, n_tiles, out, n_heads, dn, dr, rank, page_size, window,
                         scale, **k):
    return _cost_latent_attention(qa, q, gate, cache, table, ctx, out, n_heads, dn, dr, rank, page_size, window, scale)


def _cost_delta_rule(r, k, v, gate, a_raw, decay_raw, decay_bias, a_bias, norm_w, state, ctx, n_heads, d, *a, **kw):
    tokens = r.size(0)
    return (f"{tokens} tokens", tokens * n_heads * d * (6 * r.element_size() + 4) + 2 * ctx.n_requests * n_heads * d * d * 4,
            8.0 * tokens * n_heads * d * d)


def _cost_linear_recurrence(q, k, v, gate, norm_w, state, ctx, n_heads, dk, dv, *a, **kw):
    # q, k, v and the gate are read, the output written; every request's state is read and written once.
    tokens, e = q.size(0), q.element_size()
    return (f"{tokens} tokens", tokens * n_heads * (2 * dk + 3 * dv) * e + 2 * ctx.n_requests * n_heads * dk * dv * 4,
            4.0 * tokens * n_heads * dk * dv)


def _scored_keys(ctx_n_new, ctx_cached, mask, size):
    """((query, key) pairs, keys that must be read at least once) of a step, counted on the device."""
    n, c = ctx_n_new.double(), ctx_cached.double()
    if mask == ops.MASK_CAUSAL:
        return (n * c + n * (n + 1) / 2).sum(), (n + c).sum()
    # Window or chunk: a query sees size keys at most (half of that on average inside a chunk).
    per_query = size if mask == ops.MASK_WINDOW else (size + 1) / 2
    return (n * per_query).sum(), (n + c.clamp(max=size)).sum()


def _cost_scored_prefill(q, out, cache, tiles, n_tiles, ctx, table, n_q_heads, n_kv_heads, dk, dv, page_size, scale,
                         softcap, sink, mask, mask_size, **k):
    pairs, keys = _scored_keys(ctx.n_new, ctx.cached_len, mask, mask_size)
    per_key, fixed = n_kv_heads * (dk + dv) * cache.element_size(), _nbytes(q, out)
    return (f"{q.size(0)} tokens", lambda: int(float(keys) * per_key) + fixed,
            lambda: 2.0 * float(pairs) * n_q_heads * (dk + dv))


def _cost_scored_decode(q, out, cache, dec_reqs, n_dec, ctx, table, max_splits, split_keys, n_q_heads, n_kv_heads, dk,
                        dv, page_size, scale, softcap, sink, mask, mask_size, **k):
    pos = ctx.cached_len[dec_reqs[:n_dec].long()].double()
    if mask == ops.MASK_CHUNK:
        keys = (pos - (pos / mask_size).floor() * mask_size + 1).sum()
    else:
        keys = ((pos + 1).clamp(max=mask_size) if mask == ops.MASK_WINDOW else pos + 1).sum()
    per_key = n_kv_heads * (dk + dv) * cache.element_size()
    return (f"{n_dec} requests", lambda: int(float(keys) * per_key) + n_dec * n_q_heads * (dk + dv) * 2,
            lambda: 2.0 * float(keys) * n_q_heads * (dk + dv))


def _cost_hyper_step(x, write=None, read=None, **k):
    # The streams are read, and written when a branch output is added; that output is read, the normed row written.
    n = _nbytes(x) * (2 if write is not None else 1)
    if write is not None:
        n += _nbytes(write[0])
    if read is not None:
        n += x.size(0) * (x.size(1) // read[0].numel()) * (2 if k.get("act_dtype") == torch.bfloat16 else 4)
    return f"{'write ' if write is not None else ''}{'read' if read is not None else ''}".strip(), n, 0.0


def _cost_hyper_leave(x, streams, write=None, rows=None, **k):
    n_rows = x.size(0) if rows is None else rows.numel()
    width = x.size(1) // streams
    return "", n_rows * width * 4 * (streams + 1) + (n_rows * width * write[0].element_size() if write is not None else 0), 0.0


def _cost_gated_delta(x, gate, taps, ba, a_log, dt_bias, norm_w, state, conv_state, ctx, n_kv_heads, n_heads, dk, dv,
                      *a, **k):
    # The convolutions' inputs and the gate are read, the output written; every request's state is read and written.
    # A decay per key channel is one more float32 row per token.
    tokens, e, decay = x.size(0), x.element_size(), k.get("channel_decay")
    label = f"{tokens} tokens" if decay is None else f"{tokens} tokens, decay per channel"
    return (label, tokens * (x.size(1) + 2 * n_heads * dv) * e + _nbytes(decay) + 2 * ctx.n_requests * n_heads * dk * dv * 4,
            7.0 * tokens * n_heads * dk * dv)


def _cost_ssd(xbc, z, dt_raw, taps, conv_bias, dt_bias, a_log, skip, norm_w, state, conv_state, ctx, n_heads, vdim, n_groups,
              n_state, *a, **k):
    # The convolution's inputs, z and the step sizes are read, the output written; every request's state is read and written.
    tokens, inner, e = xbc.size(0), n_heads * vdim, xbc.element_size()
    return (f"{tokens} tokens", tokens * (xbc.size(1) + 2 * inner + n_heads) * e + 2 * ctx.n_requests * inner * n_state * 4,
            4.0 * tokens * inner * n_state)


def _cost_two_norms(h, d1, d2, w1, w2, *a, **k):
    # The stream is read, and written when something is added to it; the branch outputs are read, the normed rows written.
    rows, act = k.get("rows"), 2 if torch.bfloat16 in a else 4
    n = h.size(0) if rows is None else rows.numel()
    adds = [d for d in (d1, d2) if d is not None]
    per_row = 4 * (2 if adds and rows is None else 1) + sum(d.element_size() for d in adds) + act * (1 if w2 is None else 2)
    return f"{len(adds)} added", n * h.size(1) * per_row, 0.0


def _cost_gates(u, w_r, w_i, *a, **k):
    # Two block-diagonal products over the same rows; a float32 pair per token and channel is written.
    n = w_r.size(1)
    return (f"{w_r.size(0)}x{n}x{n}", _nbytes(u, w_r, w_i) + u.numel() * 8, 4.0 * u.numel() * n)


def _cost_rglru_step(u, w, r_bias, i_bias, rate, y, y_bias, state, ctx):
    n = w.size(1)
    return (f"{u.size(0)} requests, {w.size(0)}x{n}x{n}", _nbytes(w, u, u, u) + u.numel() * 8, 4.0 * u.numel() * n)


WRAPPED: Dict[str, Callable] = {
    "add_two_rmsnorm": _cost_two_norms, "rglru_gates": _cost_gates, "rglru_step": _cost_rglru_step,
    "rglru_scan": lambda ab, y, y_bias, state, ctx: (f"{ab.size(0)} tokens", _nbytes(ab) + ab.size(0) * ab.size(1) * 2 * y.element_size()
                                                     + 2 * ctx.n_requests * ab.size(1) * 4, 0.0),
    "short_conv": _cost_rows(0), "moe_route_groups": _cost_rows(0),
    "hyper_step": _cost_hyper_step, "hyper_leave": _cost_hyper_leave, "gated_delta": _cost_gated_delta,
    "ssd": _cost_ssd, "xielu": _cost_rows(0),
    "enter_pass": lambda h, delta, entered, step: ("", 2 * _nbytes(h) + _nbytes(delta, entered), 0.0),
    "scaled_sum": lambda a, b, *r, **k: ("", 3 * _nbytes(a), 0.0), "poly_norm": _cost_rows(0),
    "bigram_embedding": lambda table, pairs, ctx, prev, copies, *a, **k: (
        "", ctx.token_ids.numel() * table.size(1) * ((1 if pairs is None else 2) * table.element_size() + 4 * copies), 0.0),
    "linear_recurrence": _cost_linear_recurrence, "gate_scan": _cost_rows(0), "post_norm": _cost_rows(0, 1),
    "relu_sq": _cost_rows(0), "scale_": _cost_rows(0), "scored_prepare": _cost_rows(0, 1, 2),
    "scored_prefill": _cost_scored_prefill, "scored_decode": _cost_scored_decode, "moe_route_top": _cost_rows(0),
    "moe_combine_shared": _cost_rows(0, 3),
    "gemm_grouped": _cost_grouped, "gemm_batched": _cost_batched, "latent_attention": _cost_latent_attention,
    "latent_attention_prefill": _cost_latent_prefill,
    "delta_rule": _cost_delta_rule, "token_shift": _cost_rows(0), "outnorm_add": _cost_rows(0, 1),
    "latent_prepare": _cost_rows(0), "tanh_slice": _cost_rows(0), "softcap_": _cost_rows(0),
    "moe_route_table": _cost_rows(0), "moe_sort": _cost_rows(0), "moe_combine": _cost_rows(0),
    "gemm_bf16": _cost_gemm, "gemm_qkv_rope": _cost_qkv, "gemm_f32": _cost_gemm_f32, "library_gemm": _cost_library,
    "attn_decode": _cost_attn_decode, "attn_prefill": _cost_attn_prefill,
    "add_rmsnorm": _cost_rows(0), "embedding": lambda table, ids, *a, **k: ("", ids.numel() * table.size(1) * (table.element_size() + 4), 0.0),
    "silu_mul": _cost_rows(0), "qk_norm_rope_kvwrite": _cost_rows(0, 1, 2), "residual_add": _cost_rows(0, 1),
    "argmax": _cost_rows(0), "sample": _cost_rows(0), "scatter_tokens": _cost_rows(0),
    "outnorm_add_norm": lambda h, y, *a, **k: ("", 2 * _nbytes(h) + 2 * _nbytes(y), 0.0),
    "head_gate": _cost_rows(0), "rmsnorm_rows": _cost_rows(0), "moe_route_biased": _cost_rows(0),
    "moe_combine_identity": lambda rows, row_of, weight_of, expert_of, x, *a, **k: (
        "", _nbytes(rows, x) + x.size(0) * x.size(1) * 4, 0.0),
}


def device_peaks() -> Tuple[float, float]:
    """(GB/s, TFLOP/s) to report against: what a file MEASURED_PEAKS.json in the working directory or beside the
    package says (keys hbm_gbs, bf16_tflops), else the nominal figures of a B200 (7,700 GB/s, 2,250 TFLOP/s)."""
    import json
    import os
    here = os.path.dirname(os.path.abspath(__file__))
    for path in ("MEASURED_PEAKS.json", os.path.join(here, "..", "MEASURED_PEAKS.json")):
        try:
            with open(path) as f:
                m = json.load(f)
            return float(m["hbm_gbs"]), float(m["bf16_tflops"])
        except (OSError, ValueError, KeyError):
            continue
    return 7700.0, 2250.0


class Profiler:
    """Times every call of the wrapped ``ops`` entry points while active (see the module's head)."""

    def __init__(self, hbm_gbs: float, tflops: float, nvtx: bool = True):
        self.hbm_gbs, self.tflops, self.nvtx = float(hbm_gbs), float(tflops), nvtx
        self._saved: Dict[str, Callable] = {}
        self._calls: List[tuple] = []      # (class, bytes, flops, start event, end event); bytes and flops may be callables

    def __enter__(self):
        for name, cost in WRAPPED.items():
            real = getattr(ops, name)
            self._saved[name] = real
            setattr(ops, name, self._wrap(name, real, cost))
        return self

    def __exit__(self, *exc):
        for name, real in self._saved.items():
            setattr(ops, name, real)
        self._saved.clear()
        return False

    def _wrap(self, name, real, cost):
        def timed(*a, **k):
            label, nbytes, flops = cost(*a, **k)
            if name == "gemm_bf16" and k.get("epilogue", "store") != "store":
                label += " " + k["epilogue"]
            cls = f"{name}[{label}]" if label else name
            if self.nvtx:
                torch.cuda.nvtx.range_push(cls)
            start, end = torch.cuda.Event(enable_timing=True), torch.cuda.Event(enable_timing=True)
            start.record()
            try:
                return real(*a, **k)
            finally:
                end.record()
                if self.nvtx:
                    torch.cuda.nvtx.range_pop()
                self._calls.append((cls, nbytes, flops, start, end))
        return timed

    def classes(self) -> List[dict]:
        """Per kernel class: calls, total and mean microseconds, bytes and flops per call, achieved GB/s and
        TFLOP/s and the larger of the two fractions of peak (which bound applies)."""
        torch.cuda.synchronize()
        agg: Dict[str, List[float]] = {}
        for cls, nbytes, flops, start, end in self._calls:
            a = agg.setdefault(cls, [0, 0.0, 0.0, 0.0])
            a[0] += 1
            a[1] += start.elapsed_time(end) * 1e3
            a[2] += int(nbytes() if callable(nbytes) else nbytes)      # (counted on the device: see _cost_attn_decode)
            a[3] += float(flops() if callable(flops) else flops)
        total = sum(a[1] for a in agg.values()) or 1.0
        rows = []
        for cls, (n, us, nbytes, flops) in agg.items():
            gbs, tf = nbytes / us / 1e3, flops / us / 1e6
            f_mem, f_math = gbs / self.hbm_gbs, tf / self.tflops
            rows.append({"class": cls, "calls": n, "us_total": round(us, 1), "us_each": round(us / n, 2),
                         "share": round(us / total, 4), "bytes_each": int(nbytes / n), "flops_each": flops / n,
                         "gb_s": round(gbs, 1), "tflop_s": round(tf, 2), "bound": "hbm" if f_mem >= f_math else "tensor",
                         "frac": round(max(f_mem, f_math), 4)})
        return sorted(rows, key=lambda r: -r["us_total"])

    def report(self) -> str:
        rows = self.classes()
        lines = [f"{'share':>6} {'us total':>10} {'calls':>6} {'us each':>9} {'MB each':>9} {'GFLOP each':>11} "
                 f"{'GB/s':>8} {'TFLOP/s':>8} {'of peak':>8}  kernel class",
                 f"(peaks: {self.hbm_gbs:.0f} GB/s, {self.tflops:.0f} TFLOP/s; serialised launches, CUDA events: where the "
                 f"device waited for the host to prepare a launch, that wait counts, so kernels of tens of us read high)"]
        for r in rows:
            lines.append(f"{100 * r['share']:5.1f}% {r['us_total']:10.1f} {r['calls']:6d} {r['us_each']:9.2f} "
                         f"{r['bytes_each'] / 1e6:9.2f} {r['flops_each'] / 1e9:11.3f} {r['gb_s']:8.1f} {r['tflop_s']:8.2f} "
                         f"{r['frac']:7.3f}{'m' if r['bound'] == 'hbm' else 't'}  {r['class']}")
        return "\n".join(lines)
