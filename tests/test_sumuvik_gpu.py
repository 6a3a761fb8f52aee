"""The Sumuvik design on the GPU against the plain implementation (tests/plain_sumuvik.py, float64, no cache): each mechanism
alone (two norms of one row, the clamped gated unit in every kernel, the router with groups, window attention that keeps first
tokens, the short convolution, the gated linear recurrence), keys at the window's edge and among the first tokens made to stand
out, then whole models replayed whole, with a tail decoded token by token, in portions down to one and two tokens and in mixed
batches with so few pages and slots that they are used again; float32 and bfloat16; long decoding beyond the pool; greedy
generation through the engine's entry point and scheduler, with and without CUDA graphs; the trace program and the command
line."""
import json
import math
import os
import subprocess
import sys
from types import SimpleNamespace

import numpy as np
import pytest
import torch

import plain_sumuvik as P
import replay_util as RU
from step_util import (CUTS, DEV, close, double, junk_state, make_ctx, make_pages, on_device, planners_of, random_weights,
                       rounded, run_in_cuts)
from sumuvik_configs import SUMUVIK, shape_weights, write_sumuvik_model

pytestmark = pytest.mark.gpu

TOL_F32 = 2e-4          # float32 engine against float64: rounding only
TOL_BF16_REL = 0.05     # of the largest logit; a wrong key, window, state or expert moves logits by their own size
LENGTHS = {"A": [2, 19, 40, 77, 131, 260], "B": [1, 9, 33, 70, 128, 161], "C": [5, 31, 66, 150, 300],
           "D": [1, 2, 18, 65, 140, 230], "E": [3, 16, 47, 90, 200], "F": [1, 6, 29, 64, 133, 210]}
MODES = ["whole", "tail", "portions", "mixed"]
BOTH = pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])


@pytest.fixture(scope="module")
def models(tmp_path_factory):
    folder = tmp_path_factory.mktemp("sumuvik")
    out = {}
    for name in SUMUVIK:
        path = write_sumuvik_model(name, str(folder))
        cfg, w = P.load_model_dir(path)
        rng = np.random.default_rng(17 + ord(name))
        reqs = {f"r{i}": rng.integers(0, cfg["vocab"], n).tolist() for i, n in enumerate(LENGTHS[name])}
        ref = {r: P.forward(toks, cfg, w).numpy() for r, toks in reqs.items()}
        out[name] = (path, cfg, w, reqs, ref)
    return out


def _assert_logits(got, ref, dtype, what):
    """float32: every position within TOL_F32 (this pins the logic). bfloat16: three positions in a hundred may exceed the
    tolerance (a router's close call turns under rounding). A wrong key, window or state in a bfloat16 kernel moves every
    later position."""
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


# ---- mechanisms alone: norms, units, router ----------------------------------------------------------
@BOTH
@pytest.mark.parametrize("rows,width", [(5, 64), (1, 1), (33, 100), (3, 3001), (2, 2048), (4, 4096), (2, 5000), (2, 8192), (2, 9000)])
def test_two_norms_of_one_row(rows, width, dtype):
    """The branch outputs that were not added yet (none, one or two, in either type) go into the stream, two norms come out;
    with a list of rows only those are normed and the stream stays."""
    from llm_rs_b200 import ops
    g = torch.Generator().manual_seed(width)
    w1, w2 = (1.0 + 0.3 * torch.randn(width, generator=g) for _ in range(2))
    base = torch.randn(rows, width, generator=g)
    deltas = [torch.randn(rows, width, generator=g), rounded(torch.randn(rows, width, generator=g), torch.bfloat16)]
    for use in ((0, 0), (1, 0), (0, 1), (1, 1)):
        d = [t.to(DEV) if u else None for t, u in zip(deltas, use)]
        d[1] = d[1].bfloat16() if use[1] else None
        want = base.double() + sum((t.double() for t, u in zip(deltas, use) if u), torch.zeros(1, dtype=torch.float64))
        n1, n2 = (P.rms_norm(want, w.double(), 1e-5) for w in (w1, w2))
        h = base.to(DEV)
        y1, y2 = ops.add_two_rmsnorm(h, *d, w1.to(DEV), w2.to(DEV), 1e-5, dtype)
        close(y1.float().cpu(), n1, dtype, "first", bf16=0.01)
        close(y2.float().cpu(), n2, dtype, "second", bf16=0.01)
        close(h.cpu(), want, torch.float32, "stream", f32=1e-6)
        h, pick = base.to(DEV), torch.tensor([rows - 1, 0], dtype=torch.int32, device=DEV)
        y1, y2 = ops.add_two_rmsnorm(h, *d, w1.to(DEV), None, 1e-5, dtype, rows=pick)
        close(y1.float().cpu(), n1[pick.cpu().long()], dtype, "rows", bf16=0.01)
        assert y2 is None and torch.equal(h.cpu(), base)


@BOTH
@pytest.mark.parametrize("tokens", [1, 8, 40, 100, 300])
@pytest.mark.parametrize("D,ff,limit", [(64, 256, 0.6), (40, 20, 1.5), (128, 384, 2.0)])
def test_clamped_unit_against_plain(D, ff, limit, tokens, dtype):
    """The dense feed-forward in steps of every size: the unit in the epilogues of the tensor-core products (few tokens,
    single SMs, pairs) and as a kernel of its own; gates and ups beyond the limit on both sides."""
    from llm_rs_b200.parts import Runtime
    from llm_rs_b200.parts.mlp import SwiGLU
    g = torch.Generator().manual_seed(ff + tokens)
    part = SwiGLU(D, ff, suffix="", limit=limit, alpha=1.702, up_shift=1.0, prefix="m.")
    w = random_weights(part, g, 1.5)
    part.bind(on_device(part, w, dtype), Runtime(torch.device(DEV), dtype, 64))
    x = rounded(torch.randn(tokens, D, generator=g), dtype)
    wd = double(w)
    want = P.gated_unit(x.double(), wd, "m.", limit)
    up, gate = x.double() @ wd["m.up"].T, x.double() @ wd["m.gate"].T
    assert bool((up > limit).any()) and bool((up < -limit).any()) and bool((gate > limit).any()) and bool((gate < -limit).any())
    close(part.forward(x.to(DEV, dtype), None).float().cpu(), want, dtype, "returned", bf16=0.02)
    h = torch.randn(tokens, D, generator=g)
    hd = h.to(DEV)
    y = part.forward(x.to(DEV, dtype), None, residual=hd)
    got = hd.cpu() if y is None else hd.cpu() + y.float().cpu()
    close(got, want + h.double(), dtype, "added", bf16=0.02)


ROUTERS = [(8, 2, (4, 2), 1.7), (6, 3, (2, 1), 0.5), (12, 1, (6, 5), 1.0), (16, 4, (4, 2), 2.5), (7, 7, (1, 1), 1.0),
           (1, 1, (1, 1), 3.0), (5, 2, (5, 2), 1.0), (64, 6, (8, 3), 1.2), (200, 8, (10, 4), 2.0), (256, 8, (256, 9), 1.0),
           (33, 2, (3, 3), 1.0)]


@pytest.mark.parametrize("n,top,groups,scale", ROUTERS)
def test_router_with_groups_against_plain(n, top, groups, scale):
    """Choice by score + correction inside the best groups, weights by the scores alone; corrections that make choice scores
    negative; groups of one expert, all groups kept, one group."""
    from llm_rs_b200 import ops
    g = torch.Generator().manual_seed(n)
    logits = 2.0 * torch.randn(50, n + 3, generator=g)
    for shift in (0.0, -2.0):
        corr = 0.4 * torch.randn(n, generator=g) + shift
        e, wt = ops.moe_route_groups(logits.to(DEV), corr.to(DEV), n, top, *groups, scale)
        e, wt = e.view(50, top).cpu(), wt.view(50, top).cpu()
        for t in range(50):
            want = P.route(torch.sigmoid(logits[t, :n].double()), corr.double(), top,
                           {"count": groups[0], "keep": groups[1]}, scale)
            assert e[t].tolist() == [x for x, _ in want], t
            assert torch.allclose(wt[t].double(), torch.tensor([x for _, x in want], dtype=torch.float64), rtol=1e-5)
    e, wt = ops.moe_route_groups(torch.zeros(2, n).to(DEV), None, n, top, *groups, scale)      # equals: the lower ones
    want = P.route(torch.full((n,), 0.5, dtype=torch.float64), torch.zeros(n, dtype=torch.float64), top,
                   {"count": groups[0], "keep": groups[1]}, scale)
    assert e[:top].tolist() == [x for x, _ in want]


@BOTH
@pytest.mark.parametrize("tokens", [1, 7, 70, 260])
@pytest.mark.parametrize("D,ff,n,top,groups,shared", [
    (64, 24, 8, 2, (4, 2), (40, 1.2)), (40, 7, 6, 3, (2, 1), None), (128, 64, 16, 4, (4, 3), (128, 0.5)), (48, 16, 1, 1, (1, 1), (8, 0.3))])
def test_experts_against_plain(D, ff, n, top, groups, shared, tokens, dtype):
    """Routed experts beside a shared one whose limit differs, returned and added into a stream."""
    from llm_rs_b200.parts import Runtime
    from llm_rs_b200.parts.moe import MixtureOfExperts
    g = torch.Generator().manual_seed(D + tokens)
    extra = {} if shared is None else {"shared_size": shared[0], "shared_limit": shared[1]}
    part = MixtureOfExperts(D, ff, n, top, router="sigmoid_groups", groups=groups, route_scale=1.4, limit=0.8, alpha=1.702,
                            up_shift=1.0, prefix="mlp.", **extra)
    w = shape_weights(random_weights(part, g, 1.2), 5, torch.float32)
    w = {k: t.bfloat16().float() for k, t in w.items()}
    part.bind(on_device(part, w, dtype), Runtime(torch.device(DEV), dtype, 64))
    x = rounded(torch.randn(tokens, D, generator=g), dtype)
    f = {"router": {"experts": n, "top": top, "scale": 1.4, "groups": {"count": groups[0], "keep": groups[1]}},
         "expert": {"limit": 0.8}}
    if shared:
        f["shared"] = {"limit": shared[1]}
    want = P.experts(x.double(), f, double(w), "mlp.")
    close(part.forward(x.to(DEV, dtype), None).float().cpu(), want, dtype, "returned", bf16=0.03)
    h = torch.randn(tokens, D, generator=g).to(DEV)
    before = h.cpu().double()
    assert part.forward(x.to(DEV, dtype), None, residual=h) is None
    close(h.cpu(), want + before, dtype, "added", bf16=0.03)


# ---- mechanisms alone: attention ----------------------------------------------------------------------
def _attention(dtype, heads, kv, dk, dv, window, keep, page, n_pages, seed, scale=None, D=56, rot=None, scaling=None, sigma=1.5):
    from llm_rs_b200.parts import Runtime
    from llm_rs_b200.parts.scored_attention import ScoredAttention
    g = torch.Generator().manual_seed(seed)
    scale = 1.0 / math.sqrt(dk) if scale is None else scale
    rot = rot if rot is not None else (300.0, dk - dk % 2 if dk < 20 else dk // 4 * 2)
    part = ScoredAttention(D, heads, kv, dk, dv, scale=scale, mask="window" if window else "causal", mask_size=window,
                           keep_first=keep, qk_norm="none", gated=True, rot_dims=rot[1], rot_base=rot[0],
                           rot_pairing="neighbours", rot_scaling=scaling, qkv_bias=True, sink_score=0.0, prefix="m.")
    w = random_weights(part, g, sigma)
    part.bind(on_device(part, w, dtype), Runtime(torch.device(DEV), dtype, 4096))
    m = {"heads": heads, "kv_heads": kv, "dim": dk, "vdim": dv, "scale": scale, "rot": {"base": rot[0], "dims": rot[1], "scaling": scaling}}
    if window:
        m["mask"] = {"size": window, "keep_first": keep}
    return part, w, make_pages(kv, dk, dv, page, n_pages, dtype), m, g, D


@pytest.mark.parametrize("generic", [False, True])
@BOTH
@pytest.mark.parametrize("heads,kv,dk,dv,window,keep,page", [
    (4, 2, 16, 32, 20, 5, 16), (5, 1, 24, 8, 7, 1, 8), (2, 2, 8, 40, 1, 3, 4), (6, 6, 64, 64, 96, 40, 16), (8, 4, 64, 32, 30, 70, 32),
    (3, 3, 128, 128, 0, 0, 64), (4, 4, 128, 128, 33, 20, 16), (6, 1, 48, 32, 75, 0, 16), (7, 1, 40, 40, 151, 9, 16),
    (12, 3, 80, 48, 16, 16, 16), (3, 1, 20, 12, 2, 17, 16), (2, 1, 7, 1, 9, 2, 16), (2, 2, 128, 128, 20, 64, 64)])
def test_window_attention_that_keeps_first_tokens(dtype, heads, kv, dk, dv, window, keep, page, generic):
    """The mixer part alone: windows shorter and longer than a page, of one token and none; first tokens kept beside them that
    fill no page, a page and more, fewer and more than the window; on the tensor cores and on the kernel for any type."""
    from llm_rs_b200 import ops
    if generic and dtype == torch.float32:
        pytest.skip("float32 has one kernel")
    scaling = {"factor": 4.0, "low": 1.0, "high": 3.0, "original": 60}
    part, w, planes, m, g, D = _attention(dtype, heads, kv, dk, dv, window, keep, page, 128, dk + heads, scaling=scaling)
    seqs = [rounded(torch.randn(n, D, generator=g), dtype) for n in (151, 42)]
    want = [P.attention(s.double(), m, double(w), "m.") for s in seqs]
    ops.scored_generic_only(generic)
    try:
        got = run_in_cuts(part, planes, {}, seqs, CUTS, page, dtype, g, 128)
    finally:
        ops.scored_generic_only(False)
    for r in range(2):
        close(got[r], want[r], dtype, r)


@pytest.mark.parametrize("heads,kv,window,keep,page", [(4, 2, 200, 4, 16), (2, 1, 96, 130, 16), (4, 1, 300, 64, 64), (2, 2, 64, 1, 32)])
def test_long_portions_on_the_tensor_memory_kernel(heads, kv, window, keep, page):
    """Heads of 128 channels and portions of hundreds of tokens: the tcgen05 kernel with kept tokens, gates and the sink,
    continued from the pages, against the plain implementation and the mma.sync kernel; pages that the window has passed
    and that hold no kept token are marked as given back."""
    from llm_rs_b200 import ops
    from llm_rs_b200.parts import scored_attention
    n, dtype = 900, torch.bfloat16
    part, w, planes, m, g, D = _attention(dtype, heads, kv, 128, 128, window, keep, page, 1024 // page, 3)
    x = rounded(torch.randn(n, D, generator=g), dtype)
    want = P.attention(x.double(), m, double(w), "m.")
    table = torch.randperm(1024 // page, generator=g).to(torch.int32)[: -(-n // page)]
    outs = {}
    for tc in (True, False):
        for p in planes:
            p.zero_()
        old, scored_attention._ATTN_TC = scored_attention._ATTN_TC, tc
        try:
            rows, at = [], 0
            for k in (500, 257, 143):
                mine = table.clone()
                for j in range(len(mine)):
                    if (j + 1) * page - 1 <= at - window and j * page >= keep:
                        mine[j] = -1
                cache = SimpleNamespace(planes=planes, block_table=mine[None].to(DEV), page_size=page, owns=True, state={})
                ctx = make_ctx([k], [at], planners=planners_of(part), page_size=page)
                rows.append(part.forward(x[at:at + k].to(DEV, dtype), ctx, cache).float().cpu())
                at += k
        finally:
            scored_attention._ATTN_TC = old
        outs[tc] = torch.cat(rows)
        close(outs[tc], want, dtype, tc)
    ops.check_attention_error()
    assert not torch.equal(outs[True], outs[False]), "both runs took one kernel"


@BOTH
@pytest.mark.parametrize("decode", [False, True])
@pytest.mark.parametrize("window,keep,page,key_at", [
    (13, 3, 8, 48), (16, 0, 16, 31), (33, 40, 32, 64), (1, 5, 16, 40), (70, 16, 16, 17), (40, 1, 16, 1), (9, 16, 16, 16), (20, 7, 16, 7)])
def test_window_edges(dtype, decode, window, keep, page, key_at):
    """One token's row is replaced by a row 25 times larger, just outside the kept ones. The output must move when that key is
    the last one inside the window and must stay bit for bit when it is one step outside; for a query inside a prompt's
    portion and for one decoded alone."""
    _edges(dtype, decode, window, keep, page, key_at, {"inside": (key_at + window - 1, True), "outside": (key_at + window, False)})


@BOTH
@pytest.mark.parametrize("decode", [False, True])
@pytest.mark.parametrize("window,keep,page", [(13, 3, 8), (16, 16, 16), (9, 33, 32), (1, 1, 16), (20, 17, 16)])
def test_first_token_edges(dtype, decode, window, keep, page):
    """The last kept token still moves a query far behind its window; the token after it does not."""
    _edges(dtype, decode, window, keep, page, keep - 1, {"kept": (140, True)})
    _edges(dtype, decode, window, keep, page, keep, {"not kept": (140, False)})


def _edges(dtype, decode, window, keep, page, key_at, queries):
    part, w, planes, m, g, D = _attention(dtype, 2, 1, 16, 12, window, keep, page, 32, 5, scale=0.02)
    n = 160
    base = torch.randn(n, D, generator=g)
    other = 25.0 * torch.randn(D, generator=g)
    for name, (query_at, moves) in queries.items():
        outs = []
        for planted in (False, True):
            x = base.clone()
            if planted:
                x[key_at] = other
            x = rounded(x, dtype)
            want = P.attention(x.double(), m, double(w), "m.")[query_at]
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
            outs.append(y.float().cpu())
        d = (outs[1] - outs[0]).abs().max().item()
        assert d > 0.02 * outs[0].abs().max().item() if moves else d == 0.0, (name, d)


@BOTH
def test_a_far_key_among_hundreds(dtype):
    """A window of 700 beside 20 kept tokens and scores several times their usual size: every query's softmax rests on the few
    keys that stand out, which lie anywhere among the hundreds, at page borders and among the first tokens. Whole, and with
    the last 60 positions decoded one by one."""
    n, page = 900, 16
    part, w, planes, m, g, D = _attention(dtype, 2, 1, 16, 12, 700, 20, page, 64, 9, scale=0.6)
    x = rounded(torch.randn(n, D, generator=torch.Generator().manual_seed(77)), dtype)
    want = P.attention(x.double(), m, double(w), "m.")
    for mask in ({"size": 600, "keep_first": 20}, {"size": 700, "keep_first": 0}):
        near = P.attention(x.double(), {**m, "mask": mask}, double(w), "m.")
        assert (want - near).abs().max() > 0.1 * want.abs().max(), "far keys would not show"
    table = torch.randperm(64, generator=g).to(torch.int32)[None, : -(-n // page)].contiguous().to(DEV)
    cache = SimpleNamespace(planes=planes, block_table=table, page_size=page, owns=True, state={})
    ctx = lambda k, at: make_ctx([k], [at], planners=planners_of(part), page_size=page)
    whole = part.forward(x.to(DEV, dtype), ctx(n, 0), cache).float().cpu()
    close(whole, want, dtype, "whole", bf16=0.06, f32=1e-4)
    for p in planes:
        p.zero_()
    head = n - 60
    rows = [part.forward(x[:head].to(DEV, dtype), ctx(head, 0), cache).float().cpu()]
    rows += [part.forward(x[i:i + 1].to(DEV, dtype), ctx(1, i), cache).float().cpu() for i in range(head, n)]
    close(torch.cat(rows), want, dtype, "tail decoded", bf16=0.06, f32=1e-4)


@BOTH
@pytest.mark.parametrize("decode", [False, True])
def test_scores_far_below_the_sink(dtype, decode):
    """One added to the denominator: with scores of some minus thirty the head's output all but vanishes, with scores of some
    plus thirty it is the plain softmax's."""
    for sign in (-1.0, 1.0):
        part, w, planes, m, g, D = _attention(dtype, 2, 1, 8, 8, 30, 4, 16, 16, 13, scale=1.0, rot=(100.0, 0))
        for name in ("m.q", "m.k"):
            w[name] = 0.01 * w[name]
        w["m.q.b"] = torch.full((16,), 2.0)
        w["m.k.b"] = torch.full((8,), 2.0 * sign)
        w = {k: t.bfloat16().float() for k, t in w.items()}
        from llm_rs_b200.parts import Runtime
        part.bind(on_device(part, w, dtype), Runtime(torch.device(DEV), dtype, 4096))
        x = rounded(torch.randn(60, D, generator=g), dtype)
        want = P.attention(x.double(), m, double(w), "m.")
        cache = SimpleNamespace(planes=planes, block_table=torch.arange(4, dtype=torch.int32, device=DEV)[None], page_size=16,
                                owns=True, state={})
        ctx = lambda k, at: make_ctx([k], [at], planners=planners_of(part))
        if decode:
            part.forward(x[:59].to(DEV, dtype), ctx(59, 0), cache)
            y, want = part.forward(x[59:].to(DEV, dtype), ctx(1, 59), cache), want[59:]
        else:
            y = part.forward(x.to(DEV, dtype), ctx(60, 0), cache)
        close(y.float().cpu(), want, dtype, sign)
        assert want.abs().max() < 1e-8 if sign < 0 else want.abs().max() > 0.05


@BOTH
def test_rotation_angles_far_into_a_sequence(dtype):
    """Positions from 300,000 on: angles are made in double, so that far positions rotate as exactly as near ones."""
    part, w, planes, m, g, D = _attention(dtype, 2, 1, 16, 12, 12, 0, 16, 64, 21, rot=(1e4, 16),
                                          scaling={"factor": 2.0, "low": 1.0, "high": 4.0, "original": 1000})
    at, n = 300_000, 30
    x = rounded(torch.randn(n, D, generator=g), dtype)
    wd = double(w)
    pos = at + torch.arange(n)
    turn = lambda z: P.rotate_pairs(z, pos, 16, 1e4, m["rot"]["scaling"])
    q = turn((x.double() @ wd["m.q"].T + wd["m.q.b"]).view(n, 2, 16))
    k = turn((x.double() @ wd["m.k"].T + wd["m.k.b"]).view(n, 1, 16)).repeat_interleave(2, 1)
    v = (x.double() @ wd["m.v"].T + wd["m.v.b"]).view(n, 1, 12).repeat_interleave(2, 1)
    a = P.softmax_plus_one(torch.einsum("ihd,jhd->hij", q, k) * m["scale"], P.visible(n, 12, 0)[None])
    o = torch.einsum("hij,jhd->ihd", a, v) * torch.sigmoid(x.double() @ wd["m.g"].T)[:, :, None]
    want = (o.reshape(n, 24) @ wd["m.o"].T)[12:]      # earlier queries see rows that no step has written
    table = torch.full((1, (at + n) // 16 + 1), -1, dtype=torch.int32, device=DEV)
    table[0, (at - 12) // 16:] = torch.arange(table.size(1) - (at - 12) // 16, dtype=torch.int32, device=DEV)
    cache = SimpleNamespace(planes=planes, block_table=table, page_size=16, owns=True, state={})
    rows, i = [], 0
    for k_new in (17, 1, 2, 10):
        ctx = make_ctx([k_new], [at + i], planners=planners_of(part))
        rows.append(part.forward(x[i:i + k_new].to(DEV, dtype), ctx, cache).float().cpu())
        i += k_new
    close(torch.cat(rows)[12:], want, dtype, "far")


# ---- mechanisms alone: the recurrence -----------------------------------------------------------------
def _recurrent(dtype, width, blocks, conv, seed, D=56, **fixed):
    from llm_rs_b200.parts import Runtime
    from llm_rs_b200.parts.rglru import GatedLinearRecurrence
    g = torch.Generator().manual_seed(seed)
    names = {"r": "ra", "r_bias": "ra.b", "i": "ri", "i_bias": "ri.b"}
    part = GatedLinearRecurrence(D, width, blocks, conv, names=names, prefix="mix.")
    w = shape_weights(random_weights(part, g, 1.5), seed, torch.float32)
    for name, value in fixed.items():
        key = "mix." + name.replace("_", ".")
        w[key] = torch.full_like(w[key], value)
    w = {k: t.bfloat16().float() for k, t in w.items()}
    part.bind(on_device(part, w, dtype), Runtime(torch.device(DEV), dtype, 1 << 20))
    return part, w, g, D, lambda x: P.rglru(x.double(), {}, double(w), "mix.")


RECURRENT = [(96, 4, 4), (48, 2, 3), (33, 3, 1), (60, 1, 2), (24, 24, 2), (64, 1, 5), (256, 2, 4), (320, 5, 4), (128, 8, 6),
             (1024, 4, 4), (300, 1, 4), (45, 5, 4), (16, 1, 3), (7, 1, 4), (600, 1, 3), (1001, 1, 2)]


@BOTH
@pytest.mark.parametrize("width,blocks,conv", RECURRENT)
def test_recurrence_against_plain(width, blocks, conv, dtype):
    """The mixer alone over two requests in their own slots (which held another request's state): portions, single tokens,
    portions shorter than the convolution, steps that a request sits out; diagonal blocks of one channel to a thousand,
    of even and odd sizes; one to six taps."""
    part, w, g, D, plain = _recurrent(dtype, width, blocks, conv, width + blocks)
    seqs = [rounded(torch.randn(n, D, generator=g), dtype) for n in (151, 42)]
    got = run_in_cuts(part, None, junk_state(part), seqs, CUTS, 16, dtype, g, 32)
    for r in range(2):
        close(got[r], plain(seqs[r]), dtype, r, f32=5e-5, bf16=0.04)


@BOTH
@pytest.mark.parametrize("n_first", [1, 3, 63, 64, 65, 127, 255, 256, 257, 511, 512, 513, 1030])
def test_portions_around_the_scan_s_turns(n_first, dtype):
    """A first portion that ends at, just before and just after the ends of the scan's runs and turns, continued by portions
    of other lengths beside a second request; slow decays, so that a state that is lost or counted twice shows."""
    part, w, g, D, plain = _recurrent(dtype, 40, 2, 4, 3, lam=-6.0)
    n = n_first + 90
    seqs = [rounded(torch.randn(k, D, generator=g), dtype) for k in (n, 700)]
    cuts = [(n_first, 2), (1, 600), (1, 1), (64, 1), (2, 0), (22, 96)]
    got = run_in_cuts(part, None, junk_state(part), seqs, cuts, 16, dtype, g, 160)
    for r in range(2):
        close(got[r], plain(seqs[r]), dtype, r, f32=1e-4, bf16=0.04)


@BOTH
def test_the_state_reaches_far_back(dtype):
    """Slow decays and a first token 60 times larger than the rest: 450 tokens later it still moves the output (the plain
    implementation says so), and the engine's output agrees, whole, in portions and over 400 single tokens."""
    part, w, g, D, plain = _recurrent(dtype, 48, 4, 3, 7, lam=-7.0, ra_b=-1.0)
    x = torch.randn(502, D, generator=g)
    without = plain(x)
    x[0] *= 60.0
    x = rounded(x, dtype)
    want = plain(x)
    assert (want - without)[450:].abs().max() > 0.05 * without[450:].abs().max(), "the first token would not show"
    other = rounded(torch.randn(402, D, generator=g), dtype)
    for cuts, how in (([(502, 402)], "whole"), ([(33, 2), (69, 0)] + [(1, 1)] * 400, "one by one")):
        got = run_in_cuts(part, None, junk_state(part), [x, other], cuts, 16, dtype, g, 96)
        close(got[0], want, dtype, how, f32=3e-4, bf16=0.06)
        close(got[1], plain(other), dtype, (how, "beside"), f32=3e-4, bf16=0.06)


@BOTH
@pytest.mark.parametrize("lam", [-30.0, -12.0, 5.0, 40.0])
def test_decays_near_one_and_zero(lam, dtype):
    """A channel that all but keeps everything (1 - a^2 of 1e-12 must not come out as zero) and one that forgets at once."""
    part, w, g, D, plain = _recurrent(dtype, 32, 2, 2, 5, lam=lam)
    seqs = [rounded(torch.randn(n, D, generator=g), dtype) for n in (151, 42)]
    got = run_in_cuts(part, None, junk_state(part), seqs, CUTS, 16, dtype, g, 32)
    for r in range(2):
        want = plain(seqs[r])
        size = want.abs().max()      # of the output by itself: it may be tiny
        close(got[r] / size, want / size, dtype, r, f32=1e-4, bf16=0.04)


@BOTH
@pytest.mark.parametrize("requests", [1, 3, 8, 9, 40, 100])
def test_steps_of_many_requests(requests, dtype):
    """One token each of up to a hundred requests in scattered slots, three steps in a row."""
    part, w, g, D, plain = _recurrent(dtype, 96, 3, 4, 9)
    slots = torch.randperm(128, generator=g)[:requests].tolist()
    seqs = torch.randn(requests, 3, D, generator=g)
    seqs = rounded(seqs, dtype)
    state = junk_state(part, 128)
    for t in state.values():
        t[slots] = 0.0
    kept = {n: t.clone() for n, t in state.items()}
    cache = SimpleNamespace(state=state)
    rows = [part.forward(seqs[:, i].to(DEV, dtype), make_ctx([1] * requests, [i] * requests, slots=slots), cache).float().cpu()
            for i in range(3)]
    got = torch.stack(rows, dim=1)
    want = torch.stack([plain(seqs[r]) for r in range(requests)])
    close(got.flatten(0, 1), want.flatten(0, 1), dtype, "steps", f32=5e-5, bf16=0.04)
    others = [s for s in range(128) if s not in slots]
    assert all(torch.equal(state[n][others], kept[n][others]) for n in state), "another slot was touched"


# ---- whole models -----------------------------------------------------------------------------------
def _steps(mode, reqs):
    if mode == "tail":
        return RU.tail_one_by_one(reqs, tail=70)      # longer than every window but the widest
    if mode == "portions":
        return RU.portions(reqs, sizes=(1, 1, 2, 7, 2, 13, 5, 2, 31, 3, 17, 2, 64))
    return {"whole": RU.whole, "mixed": RU.mixed}[mode](reqs)


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("mode", MODES)
@pytest.mark.parametrize("name", list(SUMUVIK))
def test_replay_matches_plain(models, name, mode, dtype):
    from llm_rs_b200.engine import ModelRunner
    path, cfg, w, reqs, ref = models[name]
    steps = _steps(mode, reqs)
    runner = ModelRunner.from_model_dir(path, dtype=getattr(torch, dtype), max_tokens=RU.live_token_peak(steps),
                                        page_size=SUMUVIK[name][3], max_requests=4)
    free_before = [runner.manager.free_pages(g) for g in range(len(runner.manager.groups))]
    got = RU.run_steps(runner, steps)
    assert [runner.manager.free_pages(g) for g in range(len(runner.manager.groups))] == free_before, "pages were lost"
    runner.check_kernels()
    assert len(got) == sum(len(t) for t in reqs.values())
    _assert_logits(got, ref, dtype, f"{name} {mode} {dtype}")


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("seed", [21, 22])
@pytest.mark.parametrize("name", list(SUMUVIK))
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
                                        page_size=SUMUVIK[name][3], max_requests=3)
    got = RU.run_steps(runner, steps)
    assert len(got) == 2 * sum(len(t) for t in reqs.values())
    _assert_logits(got, ref, dtype, f"{name} seed {seed} {dtype}")


@pytest.mark.parametrize("name", list(SUMUVIK))
def test_residual_stream_after_every_layer(models, name):
    """The stream after each layer (float32 engine)."""
    from llm_rs_b200.engine import ModelRunner, StepEntry
    path, cfg, w, reqs, ref = models[name]
    toks, want, seen = reqs["r3"], [], []
    P.forward(toks, cfg, w, residuals=want)
    runner = ModelRunner.from_model_dir(path, dtype=torch.float32, max_tokens=192, page_size=16, max_requests=2)
    for block in runner.model.blocks:
        def wrapped(h, pending, ctx, cache, inner=block.forward, **kw):
            h, pending = inner(h, pending, ctx, cache, **kw)
            seen.append((h + sum(d for d in pending or () if d is not None)).cpu())
            return h, pending
        block.forward = wrapped
    runner.step([StepEntry("x", toks, [len(toks) - 1])])
    assert len(seen) == len(want)
    for i, (got, ref_i) in enumerate(zip(seen, want)):
        close(got, ref_i, torch.float32, f"layer {i}", f32=3e-5)


def test_long_decoding_beyond_the_pool(models):
    """A request of 600 tokens through model F (windows only) with pages for 192 tokens: the windows give pages back as they
    pass, the pages of the kept tokens stay. 60 tokens as portions, the other 540 decoded one by one."""
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
    held = [runner.manager.groups[g].n_pages - runner.manager.free_pages(g) for g in range(len(runner.manager.groups))]
    kept = {34: 2, 50: 2, 0: 0}      # pages of 32 that the kept tokens fill
    for g, n_held in enumerate(held):
        need = runner.manager.groups[g].need
        assert kept[need.keep_first] < n_held <= kept[need.keep_first] + -(-need.window // 32) + 1


@pytest.mark.parametrize("graphs", [False, True])
@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("name", list(SUMUVIK))
def test_greedy_generation_through_the_engine(models, name, dtype, graphs):
    """Prompts of unequal length through ``Engine.generate``: scheduler, prompt portions, decoding (captured in CUDA
    graphs or not: states and the convolutions' rows live on the device), the device sampler's argmax. float32 gives the
    plain implementation's tokens; bfloat16 may choose another token only where the plain logits of the two are closer
    than its rounding."""
    from llm_rs_b200.engine import Engine, EngineConfig
    from llm_rs_b200.sampling import SamplingParams
    path, cfg, w, reqs, ref = models[name]
    prompts = [reqs[r][:n] for r, n in zip(list(reqs)[1:4], (9, 33, 20))]
    engine = Engine(EngineConfig(model_path=path, block_pool_size=64, page_size=SUMUVIK[name][3], dtype=dtype,
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
def test_trace_program_on_a_sumuvik_folder(models, tmp_path, dtype):
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


def test_command_line_writes_and_runs_a_sumuvik_folder(tmp_path):
    """``random_model`` from a config.json of the design, then ``run_model`` with sampling switched off: the registry,
    the loader, the engine and the sampler through the command line; the tokens are the plain implementation's."""
    cfg_path = tmp_path / "cfg.json"
    cfg_path.write_text(json.dumps(SUMUVIK["A"][0]))
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
