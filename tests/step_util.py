"""Runs a mixer part by itself on the GPU: the index arrays of a step, scattered pages, portions beside single tokens."""
import math
from types import SimpleNamespace

import numpy as np
import torch

DEV = "cuda:0"


class Ctx(SimpleNamespace):
    """The index arrays of a step, as the step function gives them to the parts, with a mixer's plan and workspace."""

    def plan(self, key):
        return self.plans[key]

    def scratch(self, name, n_floats):
        return torch.zeros((max(n_floats, 1),), dtype=torch.float32, device=DEV)


def make_ctx(n_new, cached, slots=None, planners=(), page_size=16):
    from llm_rs_b200.parts.base import StepInfo
    i32 = lambda v: torch.tensor(v, dtype=torch.int32, device=DEV)
    a32 = lambda v: np.asarray(v, np.int32)
    q_start = np.concatenate([[0], np.cumsum(n_new)[:-1]]).astype(int).tolist()
    token_req = [r for r, n in enumerate(n_new) for _ in range(n)]
    positions = [c + i for c, n in zip(cached, n_new) for i in range(n)]
    slots = list(slots if slots is not None else range(len(n_new)))
    ctx = Ctx(n_tokens=sum(n_new), n_requests=len(n_new), q_start=i32(q_start), n_new=i32(n_new), cached_len=i32(cached),
              slot_ids=i32(slots), token_req=i32(token_req), positions=i32(positions), plans={}, shared={})
    for key, planner in planners:
        plan = planner.plan(StepInfo(sum(n_new), len(n_new), a32(q_start), a32(n_new), a32(cached), a32(slots),
                                     [], [], page_size, False))
        ctx.plans[key] = SimpleNamespace(
            arrays={k: torch.from_numpy(np.ascontiguousarray(v)).to(DEV) for k, v in plan.arrays.items()},
            values=dict(plan.values))
    return ctx


def planners_of(part):
    return part.planners() if hasattr(part, "planners") else ([(part.plan_key(), part)] if part.plan_key() else [])


def rounded(x, dtype):
    return x.bfloat16().float() if dtype == torch.bfloat16 else x


def double(w):
    return {k: v.double() for k, v in w.items()}


def random_weights(part, g, sigma=1.0):
    """Random tensors for a part's ``weight_specs``: matrices ~ sigma / sqrt(columns), vectors ~ sigma, rounded to
    bfloat16 so that both precisions and the plain implementation see the same numbers."""
    w = {}
    for s in part.weight_specs():
        t = sigma * torch.randn(s.shape, generator=g)
        if s.role == "conv":
            t = 0.6 * torch.randn(s.shape, generator=g)
        elif len(s.shape) == 2:
            t = t / math.sqrt(s.shape[-1])
        if s.role == "norm":
            t = 1.0 + 0.3 * torch.randn(s.shape, generator=g)
        w[s.name] = t.bfloat16().float()
    return w


def on_device(part, w, dtype):
    """The weights as the loader hands them over: matrices in ``dtype``, everything else float32."""
    matrix = {s.name for s in part.weight_specs() if s.role == "matrix"}
    return {k: v.to(DEV, dtype if k in matrix else torch.float32) for k, v in w.items()}


def close(got, want, dtype, what, f32=3e-5, bf16=0.03):
    """float32: every element against the largest of the wanted ones. bfloat16: every row but one in fifty."""
    scale = want.abs().max().item()
    d = (got.double() - want).abs().reshape(want.shape[0], -1).amax(dim=1)
    if dtype == torch.float32:
        assert d.max().item() <= f32 * max(1.0, scale), (what, d.max().item(), scale, int(d.argmax()))
        return
    over = int((d > bf16 * scale).sum())
    assert over <= max(1, d.numel() // 50), (what, over, d.max().item(), scale)


def make_pages(kv_heads, dk, dv, page, n_pages, dtype):
    pages = torch.zeros(n_pages, kv_heads, page * (dk + dv), dtype=dtype, device=DEV)
    return [pages[:, :, : page * dk].unflatten(2, (page, dk)), pages[:, :, page * dk:].unflatten(2, (page, dv))]


def junk_state(part, slots=5):
    """State tensors full of what earlier requests left; the slots in use are cleared as the cache manager does."""
    need = part.state_need()
    return {} if need is None else {n: torch.randn(slots, *shape, device=DEV) for n, shape in need.tensors.items()}


CUTS = [(97, 30), (2, 1), (1, 1), (30, 2), (1, 1), (19, 6), (0, 1), (1, 0)]       # 151 and 42 tokens


def run_in_cuts(part, planes, state, seqs, cuts, page, dtype, g, n_pages, first_position=0):
    """Two requests over scattered pages and their own slots (3 and 2): a prompt portion each, then portions and single
    tokens in the same steps, steps that one request sits out."""
    lens = [s.shape[0] for s in seqs]
    assert all(sum(c[r] for c in cuts) == n for r, n in enumerate(lens))
    perm = torch.randperm(n_pages, generator=g).tolist()
    width = -(-max(lens) // page)
    table = torch.tensor([perm[:width], perm[width:2 * width]], dtype=torch.int32, device=DEV)
    for t in state.values():
        t[2:4].zero_()
    cache = SimpleNamespace(planes=planes, block_table=table, page_size=page, owns=True, state=state)
    at, got = [0, 0], [[], []]
    for cut in cuts:
        live = [r for r in range(2) if cut[r]]
        ctx = make_ctx([cut[r] for r in live], [first_position + at[r] for r in live], slots=[3 - r for r in live],
                       planners=planners_of(part), page_size=page)
        cache.block_table = table[live].contiguous()
        x = torch.cat([seqs[r][at[r]: at[r] + cut[r]] for r in live]).to(DEV, dtype)
        y = part.forward(x, ctx, cache).float().cpu()
        o = 0
        for r in live:
            got[r].append(y[o:o + cut[r]])
            o += cut[r]
            at[r] += cut[r]
    return [torch.cat(rows) for rows in got]
