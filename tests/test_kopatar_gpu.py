"""The Kopatar design on the GPU against the plain implementation (tests/plain_kopatar.py, float64, no cache): each
mechanism alone (xIELU, what a pass over looped layers adds, window attention with normed heads and gated channels, the
gated delta rule with a decay per key channel, retention, the Mamba-2 recurrence, the parallel mixer), keys at the window's
edge, tokens far back and first tokens made to stand out, then whole models replayed whole, with a tail decoded token by
token, in portions down to one and two tokens and in mixed batches with so few pages and slots that they are used again;
float32 and bfloat16; long decoding beyond the pool; greedy generation through the engine's entry point and scheduler, with
and without CUDA graphs; the trace program and the command line."""
import json
import math
import os
import subprocess
import sys
from types import SimpleNamespace

import numpy as np
import pytest
import torch

import plain_kopatar as P
import replay_util as RU
from kopatar_configs import KOPATAR, shape_weights, write_kopatar_model
from step_util import (CUTS, DEV, close, double, junk_state, make_ctx, make_pages, on_device, planners_of, random_weights,
                       rounded, run_in_cuts)

pytestmark = pytest.mark.gpu

TOL_F32 = 2e-4          # float32 engine against float64: rounding only
TOL_BF16_REL = 0.05     # of the largest logit; a wrong key, window, state or pass moves logits by their own size
LENGTHS = {"A": [2, 19, 40, 77, 131, 260], "B": [1, 9, 33, 70, 128, 161], "C": [5, 31, 66, 150, 300],
           "D": [1, 2, 18, 65, 140, 230], "E": [3, 16, 47, 90, 200], "F": [1, 6, 29, 64, 133, 210]}
MODES = ["whole", "tail", "portions", "mixed"]
BOTH = pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])


@pytest.fixture(scope="module")
def models(tmp_path_factory):
    folder = tmp_path_factory.mktemp("kopatar")
    out = {}
    for name in KOPATAR:
        path = write_kopatar_model(name, str(folder))
        cfg, w = P.load_model_dir(path)
        rng = np.random.default_rng(17 + ord(name))
        reqs = {f"r{i}": rng.integers(0, cfg["vocab"], n).tolist() for i, n in enumerate(LENGTHS[name])}
        ref = {r: P.forward(toks, cfg, w).numpy() for r, toks in reqs.items()}
        out[name] = (path, cfg, w, reqs, ref)
    return out


def _assert_logits(got, ref, dtype, what):
    """float32: every position within TOL_F32 (this pins the logic). bfloat16: three positions in a hundred may exceed
    the tolerance. A wrong key, window, state or pass in a bfloat16 kernel moves every later position."""
    scale = max(float(np.abs(r).max()) for r in ref.values())
    diffs = {k: float(np.abs(row.astype(np.float64) - ref[k[0].replace("again", "")][k[1]]).max())
             for k, row in got.items()}
    assert all(np.isfinite(d) for d in diffs.values()), what
    worst = max(diffs, key=diffs.get)
    if dtype == "float32":
        assert diffs[worst] <= TOL_F32 * max(1.0, scale), f"{what}: max |diff| {diffs[worst]:.3e} at {worst}"
        return
    tol = TOL_BF16_REL * scale
    over = [k for k, d in diffs.items() if d > tol]
    assert len(over) <= max(1, 3 * len(diffs) // 100), \
        f"{what}: max |diff| {diffs[worst]:.3e} at {worst}, {len(over)} of {len(diffs)} over {tol:.3e}: {sorted(over)[:12]}"


# ---- mechanisms alone -----------------------------------------------------------------------------
@BOTH
@pytest.mark.parametrize("rows,width", [(5, 64), (1, 1), (33, 100), (3, 3001)])
def test_xielu_against_plain(rows, width, dtype):
    from llm_rs_b200.parts import Runtime
    from llm_rs_b200.parts.mlp import DenseFF
    from llm_rs_b200 import ops
    g = torch.Generator().manual_seed(width)
    z = rounded(2.0 * torch.randn(rows, width, generator=g), dtype)
    z.view(-1)[: min(8, z.numel())] = torch.tensor([0.0, 1e-4, -1e-4, -1e-2, 30.0, -30.0, -100.0, 1e-2])[: min(8, z.numel())]
    z = rounded(z, dtype)
    act = torch.tensor([0.8, -1.1])
    part = DenseFF(8, 8, "xielu", prefix="f.")
    w = random_weights(part, g)
    w["f.act"] = act
    part.bind(on_device(part, w, dtype), Runtime(torch.device(DEV), dtype, 64))
    got = ops.xielu(z.to(DEV, dtype), part.coeff).float().cpu()
    want = P.xielu(z.double(), act.double())
    # Of each element by itself; the negative branch crosses zero away from z = 0, so its terms count, not their sum.
    tol = 1e-5 if dtype == torch.float32 else 0.005
    assert bool(((got.double() - want).abs() <= tol * (want.abs() + 1e-2 * z.double().abs()) + 1e-12).all())


@BOTH
@pytest.mark.parametrize("rows,width,times", [(7, 50, 3), (1, 1100, 1), (300, 64, 2)])
def test_what_a_pass_adds(rows, width, times, dtype):
    """The embedding output ahead of every pass but the first, the pass's own vector ahead of each, the branch output that
    was not added yet; the embedding output is kept although the stream it came from changes in place."""
    from llm_rs_b200.parts import Runtime
    from llm_rs_b200.parts.embedding import EmbeddingAdd
    g = torch.Generator().manual_seed(rows)
    part = EmbeddingAdd(width, times)
    step = torch.randn(times, width, generator=g)
    part.bind({"loop.step": step.to(DEV)}, Runtime(torch.device(DEV), dtype, 64))
    h0 = torch.randn(rows, width, generator=g)
    ctx, h = SimpleNamespace(stream_copy=None), h0.to(DEV)
    entered, want = part.prepare(h, ctx), h0.clone()
    for t in range(times):
        pending = rounded(torch.randn(rows, width, generator=g), dtype) if t else None
        h = part.forward(h, None if pending is None else pending.to(DEV, dtype), entered, ctx, t)
        if pending is not None:
            want = want + pending
        want = (want + h0 if t else want) + step[t]
        assert torch.allclose(h.cpu(), want, atol=1e-5)
        h.mul_(0.5)      # what the pass's blocks do to the stream
        want = want * 0.5


def _attention(dtype, heads, kv, dk, dv, window, page, n_pages, seed, scale=None, D=56, rot=0):
    from llm_rs_b200.parts import Runtime
    from llm_rs_b200.parts.scored_attention import ScoredAttention
    g = torch.Generator().manual_seed(seed)
    scale = 1.0 / math.sqrt(dk) if scale is None else scale
    part = ScoredAttention(D, heads, kv, dk, dv, scale=scale, mask="window" if window else "causal", mask_size=window,
                           qk_norm="head", norm_eps=1e-5, gated=True, gate_per="channel", rot_dims=rot, rot_base=300.0,
                           prefix="m.")
    w = random_weights(part, g, 1.5)
    part.bind(on_device(part, w, dtype), Runtime(torch.device(DEV), dtype, 4096))
    m = {"heads": heads, "kv_heads": kv, "dim": dk, "vdim": dv, "scale": scale}
    if window:
        m["mask"] = {"size": window}
    return part, w, make_pages(kv, dk, dv, page, n_pages, dtype), m, g, D


@pytest.mark.parametrize("generic", [False, True])
@BOTH
@pytest.mark.parametrize("heads,kv,dk,dv,window,page", [
    (4, 2, 16, 32, 20, 16), (5, 1, 24, 8, 7, 8), (2, 2, 8, 40, 1, 4), (6, 6, 64, 64, 96, 16), (8, 4, 64, 32, 130, 32),
    (3, 3, 128, 128, 0, 64), (4, 4, 128, 128, 33, 16), (6, 1, 48, 32, 75, 16), (7, 1, 40, 40, 151, 16), (12, 3, 80, 48, 16, 16),
    (3, 1, 20, 12, 2, 16), (2, 1, 16, 1, 9, 16)])
def test_gated_window_attention_against_plain(dtype, heads, kv, dk, dv, window, page, generic):
    """The mixer part alone: heads of q and k normed with a shared weight, windows shorter and longer than a page, of one
    token and none, a gate on every channel; on the tensor cores and on the kernel for any type."""
    from llm_rs_b200 import ops
    if generic and dtype == torch.float32:
        pytest.skip("float32 has one kernel")
    part, w, planes, m, g, D = _attention(dtype, heads, kv, dk, dv, window, page, 128, dk + heads)
    seqs = [rounded(torch.randn(n, D, generator=g), dtype) for n in (151, 42)]
    want = [P.gated_window_attention(s.double(), m, double(w), "m.", 1e-5, torch.arange(len(s))) for s in seqs]
    ops.scored_generic_only(generic)
    try:
        got = run_in_cuts(part, planes, {}, seqs, CUTS, page, dtype, g, 128)
    finally:
        ops.scored_generic_only(False)
    for r in range(2):
        close(got[r], want[r], dtype, r)


@BOTH
def test_head_norm_comes_before_a_rotation(dtype):
    """The norm with a shared weight beside a partial rotation (no layer of this design has both): norm, weight, rotation."""
    part, w, planes, m, g, D = _attention(dtype, 4, 2, 16, 8, 30, 16, 64, 3, rot=8)
    x = rounded(torch.randn(60, D, generator=g), dtype)
    pos = torch.arange(60)
    wd = double(w)
    q = P.rotate_halves(P.rms((x.double() @ wd["m.q"].T).view(60, 4, 16), 1e-5) * wd["m.q.norm"], pos, 8, 300.0)
    k = P.rotate_halves(P.rms((x.double() @ wd["m.k"].T).view(60, 2, 16), 1e-5) * wd["m.k.norm"], pos, 8, 300.0)
    v = (x.double() @ wd["m.v"].T).view(60, 2, 8)
    s = torch.einsum("ihd,jhd->hij", q, k.repeat_interleave(2, 1)) * m["scale"]
    dist = pos[:, None] - pos[None, :]
    a = torch.softmax(s.masked_fill(~((dist >= 0) & (dist < 30)), float("-inf")), dim=-1)
    o = torch.einsum("hij,jhd->ihd", a, v.repeat_interleave(2, 1)).reshape(60, 32) * torch.sigmoid(x.double() @ wd["m.g"].T)
    cache = SimpleNamespace(planes=planes, block_table=torch.arange(4, dtype=torch.int32, device=DEV)[None], page_size=16,
                            owns=True, state={})
    y = part.forward(x.to(DEV, dtype), make_ctx([60], [0], planners=planners_of(part)), cache)
    close(y.float().cpu(), o @ wd["m.o"].T, dtype, "norm, then rotation")


@BOTH
@pytest.mark.parametrize("decode", [False, True])
@pytest.mark.parametrize("window,page,key_at", [(13, 8, 48), (16, 16, 31), (33, 32, 64), (1, 16, 40), (70, 16, 17), (40, 16, 0)])
def test_window_edges(dtype, decode, window, page, key_at):
    """One token's row is replaced by a row 25 times larger (its value grows 25-fold; the norm keeps its key's size). The
    output must move when that key is the last one inside the window and must stay bit for bit when it is one step
    outside; for a query inside a prompt's portion and for one decoded alone; keys at a page's first and last row and the
    sequence's first token."""
    part, w, planes, m, g, D = _attention(dtype, 2, 1, 16, 12, window, page, 32, 5)
    n = 160
    base = torch.randn(n, D, generator=g)
    other = 25.0 * torch.randn(D, generator=g)
    outs = {}
    for name, query_at in (("inside", key_at + window - 1), ("outside", key_at + window)):
        for planted in (False, True):
            x = base.clone()
            if planted:
                x[key_at] = other
            x = rounded(x, dtype)
            want = P.gated_window_attention(x.double(), m, double(w), "m.", 1e-5, torch.arange(n))[query_at]
            for p in planes:
                p.zero_()
            table = torch.arange(31, -1, -1, dtype=torch.int32, device=DEV)[None, : -(-n // page)].contiguous()
            cache = SimpleNamespace(planes=planes, block_table=table, page_size=page, owns=True, state={})
            pl = planners_of(part)
            if decode and query_at > 0:
                part.forward(x[:query_at].to(DEV, dtype), make_ctx([query_at], [0], planners=pl, page_size=page), cache)
                y = part.forward(x[query_at:query_at + 1].to(DEV, dtype),
                                 make_ctx([1], [query_at], planners=pl, page_size=page), cache)[0]
            else:
                y = part.forward(x[: query_at + 3].to(DEV, dtype),
                                 make_ctx([query_at + 3], [0], planners=pl, page_size=page), cache)[query_at]
            scale = want.abs().max().item()
            d = (y.float().cpu().double() - want).abs().max().item()
            assert d <= (3e-5 * max(1, scale) if dtype == torch.float32 else 0.03 * scale), (name, planted, d, scale)
            outs[(name, planted)] = y.float().cpu()
    moved = (outs[("inside", True)] - outs[("inside", False)]).abs().max().item()
    still = (outs[("outside", True)] - outs[("outside", False)]).abs().max().item()
    assert moved > 0.02 * outs[("inside", False)].abs().max().item(), moved
    assert still == 0.0, still


@BOTH
def test_a_far_key_among_hundreds(dtype):
    """A window of 700 and scores several times their usual size: every query's softmax rests on the few keys that stand
    out, which lie anywhere among the window's hundreds, at page borders and among the sequence's first tokens. Whole, and
    with the last 60 positions decoded one by one."""
    n, page = 900, 16
    part, w, planes, m, g, D = _attention(dtype, 2, 1, 16, 12, 700, page, 64, 9, scale=1.5)
    x = rounded(torch.randn(n, D, generator=torch.Generator().manual_seed(77)), dtype)
    want = P.gated_window_attention(x.double(), m, double(w), "m.", 1e-5, torch.arange(n))
    near = P.gated_window_attention(x.double(), {**m, "mask": {"size": 600}}, double(w), "m.", 1e-5, torch.arange(n))
    assert (want - near).abs().max() > 0.2 * want.abs().max(), "far keys would not show"
    table = torch.randperm(64, generator=g).to(torch.int32)[None, : -(-n // page)].contiguous().to(DEV)
    cache = SimpleNamespace(planes=planes, block_table=table, page_size=page, owns=True, state={})
    ctx = lambda k, at: make_ctx([k], [at], planners=planners_of(part), page_size=page)
    whole = part.forward(x.to(DEV, dtype), ctx(n, 0), cache).float().cpu()
    close(whole, want, dtype, "whole", bf16=0.06)
    for p in planes:
        p.zero_()
    head = n - 60
    rows = [part.forward(x[:head].to(DEV, dtype), ctx(head, 0), cache).float().cpu()]
    rows += [part.forward(x[i:i + 1].to(DEV, dtype), ctx(1, i), cache).float().cpu() for i in range(head, n)]
    close(torch.cat(rows), want, dtype, "tail decoded", bf16=0.06)


def _recurrent(kind, dtype, sizes, seed, D=56, **fade):
    """(part, weights, its mixer's config keys, generator, D, plain function of (rows, weights, positions)) of one of the
    three recurrent mixers with weights as ``shape_weights`` makes them."""
    from llm_rs_b200.parts import Runtime
    from llm_rs_b200.parts.delta_rule import ChannelDelta
    from llm_rs_b200.parts.recurrent import Retention
    from llm_rs_b200.parts.ssd import Mamba2
    g = torch.Generator().manual_seed(seed)
    if kind == "delta":
        heads, kv, dk, dv, conv, ra, rg = sizes
        part = ChannelDelta(D, heads, kv, dk, dv, conv, ra, rg, norm_eps=1e-5, prefix="mix.")
        m = {"heads": heads, "kv_heads": kv, "dim": dk, "vdim": dv, "conv": conv}
        plain = lambda x, w, pos: P.channel_delta(x, m, w, "mix.", 1e-5)
    elif kind == "retention":
        heads, dk, dv, rot, decay = sizes
        part = Retention(D, heads, dk, dv, decay, rot_dims=rot, rot_base=900.0, norm_eps=1e-5, prefix="mix.")
        m = {"heads": heads, "dim": dk, "vdim": dv, "decay": decay, "rot": {"base": 900.0, "dims": rot}}
        plain = lambda x, w, pos: P.retention(x, m, w, "mix.", 1e-5, pos)
    else:
        heads, dv, state, groups, conv, parts = sizes
        part = Mamba2(D, heads, dv, state, groups, conv, norm_parts=parts, norm_eps=1e-5, prefix="mix.")
        m = {"heads": heads, "vdim": dv, "state": state, "groups": groups, "conv": conv, "norm_groups": parts}
        plain = lambda x, w, pos: P.mamba2(x, m, w, "mix.", 1e-5)
    w = shape_weights(random_weights(part, g, 1.5), seed, torch.float32)
    for name, value in fade.items():
        w["mix." + name] = torch.full_like(w["mix." + name], value)
    w = {k: t.bfloat16().float() for k, t in w.items()}
    part.bind(on_device(part, w, dtype), Runtime(torch.device(DEV), dtype, 1 << 20))
    return part, w, g, D, plain


RECURRENT = [
    ("delta", (4, 2, 16, 8, 4, 12, 20)), ("delta", (2, 2, 8, 24, 2, 8, 8)), ("delta", (3, 1, 12, 20, 1, 5, 7)),
    ("delta", (4, 4, 32, 16, 5, 16, 16)), ("delta", (4, 2, 64, 64, 4, 32, 16)), ("delta", (2, 1, 128, 32, 3, 24, 40)),
    # (many heads and wide values: steps of two requests take the kernel of fewer lanes a column, of one that of more)
    ("delta", (20, 4, 16, 120, 2, 6, 6)), ("delta", (20, 2, 128, 120, 3, 8, 8)),
    ("delta", (1, 1, 200, 40, 4, 9, 3)), ("delta", (6, 3, 20, 17, 3, 1, 1)), ("delta", (2, 2, 7, 9, 2, 6, 6)),
    ("retention", (3, 16, 24, 8, [0.9, 0.97, 0.995])), ("retention", (2, 20, 12, 20, [0.95, 1.0])),
    ("retention", (1, 6, 10, 2, [0.98])), ("retention", (2, 64, 32, 32, [0.96, 0.0])), ("retention", (1, 128, 40, 128, [0.999])),
    ("retention", (2, 200, 16, 100, [0.99, 0.9])), ("retention", (2, 9, 7, 0, [0.9, 0.99])), ("retention", (5, 32, 33, 2, [0.9] * 5)),
    ("mamba", (4, 12, 10, 2, 2, 3)), ("mamba", (2, 20, 16, 1, 3, 5)), ("mamba", (8, 32, 64, 4, 4, 1)),
    ("mamba", (3, 7, 9, 3, 1, 7)), ("mamba", (4, 64, 128, 1, 4, 16)), ("mamba", (2, 16, 200, 2, 5, 2)),
    ("mamba", (6, 1, 4, 2, 3, 1)), ("mamba", (1, 100, 33, 1, 4, 10))]


@BOTH
@pytest.mark.parametrize("kind,sizes", RECURRENT)
def test_recurrent_mixers_against_plain(kind, sizes, dtype):
    """Each recurrent mixer alone over two requests in their own slots (which held another request's state): portions,
    single tokens, portions shorter than the convolution, steps that a request sits out; key heads or groups shared by
    several heads and by all; key sizes of every kernel variant, value widths that are no multiple of its slices; one
    to five taps; norm parts within and across heads."""
    part, w, g, D, plain = _recurrent(kind, dtype, sizes, 40 + sum(s for s in sizes if isinstance(s, int)))
    seqs = [rounded(torch.randn(n, D, generator=g), dtype) for n in (151, 42)]
    want = [plain(s.double(), double(w), torch.arange(len(s))) for s in seqs]
    got = run_in_cuts(part, None, junk_state(part), seqs, CUTS, 16, dtype, g, 32)
    for r in range(2):
        close(got[r], want[r], dtype, (kind, r), f32=1e-4, bf16=0.05)


@BOTH
@pytest.mark.parametrize("kind,sizes,fade", [
    ("delta", (2, 1, 16, 12, 4, 8, 8), {"A_log": -5.0}), ("retention", (2, 16, 12, 8, [0.999, 1.0]), {}),
    ("mamba", (2, 12, 16, 1, 3, 2), {"A_log": -6.0})])
def test_the_state_reaches_far_back(kind, sizes, fade, dtype):
    """Slow decays and a first token 60 times larger than the rest: 500 tokens later its write still moves the output (the
    plain implementation says so), and the engine's output agrees, whole, in portions and over 400 single tokens."""
    part, w, g, D, plain = _recurrent(kind, dtype, sizes, 7, **fade)
    x = torch.randn(502, D, generator=g)
    without = plain(x.double(), double(w), torch.arange(502))
    x[0] *= 60.0
    x = rounded(x, dtype)
    want = plain(x.double(), double(w), torch.arange(502))
    if kind != "delta":      # (a delta rule writes over what its keys find; unit keys hide the row's size)
        assert (want - without)[450:].abs().max() > 0.05 * without[450:].abs().max(), "the first token would not show"
    other = rounded(torch.randn(402, D, generator=g), dtype)
    want_other = plain(other.double(), double(w), torch.arange(402))
    whole = run_in_cuts(part, None, junk_state(part), [x, other], [(502, 402)], 16, dtype, g, 96)
    single = run_in_cuts(part, None, junk_state(part), [x, other], [(33, 2), (69, 0)] + [(1, 1)] * 400, 16, dtype, g, 96)
    for got, how in ((whole, "whole"), (single, "one by one")):
        close(got[0], want, dtype, (kind, how), f32=3e-4, bf16=0.06)
        close(got[1], want_other, dtype, (kind, how, "beside"), f32=3e-4, bf16=0.06)


@BOTH
def test_channels_of_a_head_decay_by_themselves(dtype):
    """Half of a head's key channels forget at once and half keep for hundreds of tokens: mixing the channels up, or one
    decay for the whole head, gives another output (shown on the plain implementation)."""
    part, w, g, D, plain = _recurrent("delta", dtype, (2, 1, 16, 12, 3, 8, 8), 11)
    bias = torch.where(torch.arange(32) % 2 == 0, torch.tensor(-6.0), torch.tensor(3.0))
    w["mix.dt_bias"] = bias
    part.dt_bias = bias.to(DEV)
    x = rounded(torch.randn(120, D, generator=g), dtype)
    want = plain(x.double(), double(w), torch.arange(120))
    for wrong in (bias.roll(1), torch.full_like(bias, -1.5)):
        assert (plain(x.double(), double({**w, "mix.dt_bias": wrong}), torch.arange(120)) - want).abs().max() > 0.2 * want.abs().max()
    got = run_in_cuts(part, None, junk_state(part), [x, x[:5]], [(70, 5), (2, 0), (1, 0), (47, 0)], 16, dtype, g, 32)
    close(got[0], want, dtype, "decay per channel", f32=1e-4, bf16=0.05)


@BOTH
def test_rotation_angles_far_into_a_sequence(dtype):
    """Retention at positions from 300,000 on: angles are made in double, so that far positions rotate as exactly as near
    ones (a float32 product of position and frequency would be off by hundredths of a turn)."""
    part, w, g, D, plain = _recurrent("retention", dtype, (2, 16, 12, 16, [0.95, 0.99]), 5)
    at = 300_000
    seqs = [rounded(torch.randn(n, D, generator=g), dtype) for n in (40, 9)]
    want = [plain(s.double(), double(w), at + torch.arange(len(s))) for s in seqs]
    got = run_in_cuts(part, None, junk_state(part), seqs, [(33, 2), (1, 6), (6, 1)], 16, dtype, g, 32, first_position=at)
    for r in range(2):
        close(got[r], want[r], dtype, r, f32=1e-4, bf16=0.05)


@pytest.mark.parametrize("fused", [True, False])
@BOTH
def test_parallel_mixer_against_plain(dtype, fused, monkeypatch):
    """The two side by side, with the two output projections as one product and as two products and a sum."""
    from llm_rs_b200.parts import PartSpec, Runtime, parallel
    monkeypatch.setattr(parallel, "FUSE_PARALLEL", fused)
    D, g = 56, torch.Generator().manual_seed(11)
    left = {"hidden_size": D, "n_heads": 4, "n_kv_heads": 2, "dim": 16, "vdim": 8, "scale": 0.3, "mask": "window",
            "mask_size": 21, "qk_norm": "head", "norm_eps": 1e-5, "gated": True, "gate_per": "channel"}
    right = {"hidden_size": D, "n_heads": 6, "vdim": 20, "state": 12, "groups": 3, "conv": 3, "norm_parts": 4, "norm_eps": 1e-5}
    part = parallel.ParallelMixer(PartSpec("scored_attention", left), PartSpec("mamba2", right), 0.6, 1.7, prefix="m.")
    w = {k: t.bfloat16().float() for k, t in shape_weights(random_weights(part, g, 1.5), 3, torch.float32).items()}
    part.bind(on_device(part, w, dtype), Runtime(torch.device(DEV), dtype, 4096))
    assert (part.fused is not None) == fused
    m = {"left": {"heads": 4, "kv_heads": 2, "dim": 16, "vdim": 8, "scale": 0.3, "mask": {"size": 21}},
         "right": {"heads": 6, "vdim": 20, "state": 12, "groups": 3, "norm_groups": 4}, "left_scale": 0.6, "right_scale": 1.7}
    seqs = [rounded(torch.randn(n, D, generator=g), dtype) for n in (151, 42)]
    want = [P.parallel_mixer(s.double(), m, double(w), "m.", 1e-5, torch.arange(len(s))) for s in seqs]
    got = run_in_cuts(part, make_pages(2, 16, 8, 16, 64, dtype), junk_state(part), seqs, CUTS, 16, dtype, g, 64)
    for r in range(2):
        close(got[r], want[r], dtype, r, f32=1e-4, bf16=0.04)


# ---- whole models -----------------------------------------------------------------------------------
def _steps(mode, reqs):
    if mode == "tail":
        return RU.tail_one_by_one(reqs, tail=70)      # longer than every window but the widest
    if mode == "portions":
        return RU.portions(reqs, sizes=(1, 1, 2, 7, 2, 13, 5, 2, 31, 3, 17, 2, 64))
    return {"whole": RU.whole, "mixed": RU.mixed}[mode](reqs)


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("mode", MODES)
@pytest.mark.parametrize("name", list(KOPATAR))
def test_replay_matches_plain(models, name, mode, dtype):
    from llm_rs_b200.engine import ModelRunner
    path, cfg, w, reqs, ref = models[name]
    steps = _steps(mode, reqs)
    runner = ModelRunner.from_model_dir(path, dtype=getattr(torch, dtype), max_tokens=RU.live_token_peak(steps),
                                        page_size=KOPATAR[name][3], max_requests=4)
    free_before = [runner.manager.free_pages(g) for g in range(len(runner.manager.groups))]
    got = RU.run_steps(runner, steps)
    assert [runner.manager.free_pages(g) for g in range(len(runner.manager.groups))] == free_before, "pages were lost"
    runner.check_kernels()
    assert len(got) == sum(len(t) for t in reqs.values())
    _assert_logits(got, ref, dtype, f"{name} {mode} {dtype}")


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("seed", [21, 22])
@pytest.mark.parametrize("name", list(KOPATAR))
def test_mixed_replay_with_other_cuts_and_pages_and_slots_used_again(models, name, seed, dtype):
    """Mixed batches with other seeds and portion sizes, two or three live requests, the requests twice over, so that
    every page and every state slot serves several requests."""
    from llm_rs_b200.engine import ModelRunner
    path, cfg, w, reqs, ref = models[name]
    rng = np.random.default_rng(seed)
    sizes = tuple(int(x) for x in rng.choice([2, 3, 7, 16, 31, 33, 64, 65, 129], size=5, replace=False))
    twice = {**reqs, **{r + "again": t for r, t in reqs.items()}}
    steps = RU.mixed(twice, seed=seed, max_live=2 + seed % 2, decode_tail=5 + seed % 7, sizes=sizes)
    runner = ModelRunner.from_model_dir(path, dtype=getattr(torch, dtype), max_tokens=RU.live_token_peak(steps),
                                        page_size=KOPATAR[name][3], max_requests=3)
    got = RU.run_steps(runner, steps)
    assert len(got) == 2 * sum(len(t) for t in reqs.values())
    _assert_logits(got, ref, dtype, f"{name} seed {seed} {dtype}")


@pytest.mark.parametrize("name", ["A", "D", "E"])
def test_residual_stream_after_every_layer_run(models, name):
    """The stream after each layer run, every pass counted (float32 engine)."""
    from llm_rs_b200.engine import ModelRunner, StepEntry
    path, cfg, w, reqs, ref = models[name]
    toks, want, seen = reqs["r3"], [], []
    P.forward(toks, cfg, w, residuals=want)
    runner = ModelRunner.from_model_dir(path, dtype=torch.float32, max_tokens=128, page_size=16, max_requests=2)
    for block in runner.model.blocks:
        def wrapped(h, pending, ctx, cache, inner=block.forward, **kw):
            h, pending = inner(h, pending, ctx, cache, **kw)
            seen.append((h if pending is None else h + pending).cpu())
            return h, pending
        block.forward = wrapped
    runner.step([StepEntry("x", toks, [len(toks) - 1])])
    assert len(seen) == len(want)
    for i, (got, ref_i) in enumerate(zip(seen, want)):
        close(got, ref_i, torch.float32, f"layer run {i}", f32=3e-5)


def test_long_decoding_beyond_the_pool(models):
    """A request of 600 tokens through model F (windows only) with pages for 192 tokens: the windows give pages back as
    they pass, in every pass over the loop, the recurrences keep their state. 60 tokens as portions, the other 540
    decoded one by one."""
    from llm_rs_b200.engine import ModelRunner
    path, cfg, w, reqs, ref = models["F"]
    toks = np.random.default_rng(5).integers(0, cfg["vocab"], 600).tolist()
    want = P.forward(toks, cfg, w).numpy()
    runner = ModelRunner.from_model_dir(path, dtype=torch.float32, max_tokens=192, page_size=32, max_requests=2)
    steps = [{"entries": [{"id": "long", "tokens": toks[a:a + 30], "want": list(range(30))}], "end": []} for a in (0, 30)]
    steps += [{"entries": [{"id": "long", "tokens": [t], "want": [0]}], "end": []} for t in toks[60:]]
    got = RU.run_steps(runner, steps)
    worst, where, n = RU.max_diff(got, {"long": want})
    assert n == 600 and worst <= TOL_F32 * max(1.0, float(np.abs(want).max())), (worst, where)


@pytest.mark.parametrize("graphs", [False, True])
@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("name", list(KOPATAR))
def test_greedy_generation_through_the_engine(models, name, dtype, graphs):
    """Prompts of unequal length through ``Engine.generate``: scheduler, prompt portions, decoding (captured in CUDA
    graphs or not: states and the convolutions' rows live on the device), the device sampler's argmax. float32 gives the
    plain implementation's tokens; bfloat16 may choose another token only where the plain logits of the two are closer
    than its rounding."""
    from llm_rs_b200.engine import Engine, EngineConfig
    from llm_rs_b200.sampling import SamplingParams
    path, cfg, w, reqs, ref = models[name]
    prompts = [reqs[r][:n] for r, n in zip(list(reqs)[1:4], (9, 33, 20))]
    engine = Engine(EngineConfig(model_path=path, block_pool_size=64, page_size=KOPATAR[name][3], dtype=dtype,
                                 max_requests=4, cuda_graphs=graphs, prefill_chunk=16, max_tokens_per_step=24))
    got = engine.generate(prompts, SamplingParams(temperature=0.0, max_new_tokens=12, ignore_eos=True))
    for prompt, new in zip(prompts, got):
        assert len(new) == 12
        toks = list(prompt) + new
        rows = P.forward(toks, cfg, w)[len(prompt) - 1: -1]
        for row, t in zip(rows, new):
            gap = float(row.max() - row[t])
            assert gap <= (1e-4 if dtype == "float32" else 0.06) * float(row.abs().max()), (name, gap)


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_trace_program_on_a_kopatar_folder(models, tmp_path, dtype):
    """bin/trace_run picks the design by config.json and replays a mixed trace."""
    path, cfg, w, reqs, ref = models["B"]
    steps = RU.want_only(RU.mixed(reqs, seed=9), {r: set(range(0, len(t), 3)) | {len(t) - 1} for r, t in reqs.items()})
    out_dir = tmp_path / "out"
    lines = [json.dumps({"step": i, **st}) for i, st in enumerate(steps)]
    root = os.path.dirname(os.path.dirname(os.path.abspath(__file__)))
    proc = subprocess.run(
        [sys.executable, os.path.join(root, "bin", "trace_run"), "--model", path, "--dtype", dtype, "--out", str(out_dir),
         "--max-tokens", str(RU.live_token_peak(steps)), "--max-requests", "4", "--page-size", "8"],
        input="\n".join(lines) + "\n", capture_output=True, text=True, timeout=600)
    assert proc.returncode == 0, proc.stderr[-2000:]
    assert proc.stdout.split("\n")[:len(steps)] == [f"done {i}" for i in range(len(steps))]
    at, got, V = {}, {}, cfg["vocab"]
    for i, st in enumerate(steps):
        n_want = sum(len(e["want"]) for e in st["entries"])
        if not n_want:
            assert not (out_dir / f"{i}.f32").exists()
        else:
            data = np.fromfile(out_dir / f"{i}.f32", dtype="<f4").reshape(-1, V)
            assert data.shape[0] == n_want
        k = 0
        for e in st["entries"]:
            base = at.get(e["id"], 0)
            for wnt in e["want"]:
                got[(e["id"], base + wnt)] = data[k]
                k += 1
            at[e["id"]] = base + len(e["tokens"])
    _assert_logits(got, ref, dtype, f"trace program {dtype}")


def test_command_line_writes_and_runs_a_kopatar_folder(tmp_path):
    """``random_model`` from a config.json of the design, then ``run_model`` with sampling switched off: the registry,
    the loader, the engine and the sampler through the command line; the tokens are the plain implementation's."""
    cfg_path = tmp_path / "cfg.json"
    cfg_path.write_text(json.dumps(KOPATAR["A"][0]))
    out = tmp_path / "model"
    root = os.path.dirname(os.path.dirname(os.path.abspath(__file__)))
    run = lambda *a: subprocess.run([sys.executable, "-m", "llm_rs_b200.cli", *a], cwd=root, capture_output=True,
                                    text=True, timeout=600)
    made = run("random_model", "--config", str(cfg_path), "--out", str(out), "--seed", "5", "--sigma", "0.15",
               "--norm-jitter", "0.2")
    assert made.returncode == 0, made.stderr[-2000:]
    prompt = [5, 17, 3, 9, 200, 41, 7, 7, 150]
    done = run("run_model", "--model-path", str(out), "--prompt-ids", ",".join(map(str, prompt)), "--dtype", "float32",
               "--max-new-tokens", "10", "--ignore-eos", "--page-size", "16", "--block-pool-size", "32")
    assert done.returncode == 0, done.stderr[-2000:]
    lines = dict(l.split(":", 1) for l in done.stdout.splitlines() if ":" in l)
    got = [int(t) for t in lines["Generated token ids"].split(",")]
    cfg, w = P.load_model_dir(str(out))
    rows = P.forward(prompt + got, cfg, w)[len(prompt) - 1: -1]
    assert len(got) == 10
    for row, tok in zip(rows, got):
        assert float(row.max() - row[tok]) <= 1e-4 * float(row.abs().max())
