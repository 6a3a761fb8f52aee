"""The Sumuvik design without a GPU: its configuration (every key, optional keys absent, refusals), the model a configuration
is turned into (part kinds, pages and state per entry, tensor names), pages of a window that keeps first tokens, rescaled
frequencies, and the plain implementation's own properties (tests/plain_sumuvik.py is the oracle of the GPU tests, so what it
computes is pinned here by hand-made cases)."""
import copy
import math

import pytest
import torch

import plain_sumuvik as P
from llm_rs_b200.cache import CacheManager, GroupSpec
from llm_rs_b200.config import ConfigError, SumuvikConfig, load_config, resolve_architecture
from llm_rs_b200.parts import CacheNeed, DecoderModel
from llm_rs_b200.parts.position import wavelength_scaled_frequencies
from sumuvik_configs import SUMUVIK, write_sumuvik_model

F64 = torch.float64


# ---- configuration ------------------------------------------------------------------------------------
@pytest.mark.parametrize("name", list(SUMUVIK))
def test_config_round_trip(name, tmp_path):
    raw = SUMUVIK[name][0]
    cfg = SumuvikConfig.from_dict(raw)
    assert SumuvikConfig.from_dict(cfg.to_dict()) == cfg
    assert resolve_architecture(raw).config_cls is SumuvikConfig
    assert load_config(write_sumuvik_model(name, str(tmp_path)))[1] == cfg


def test_optional_keys():
    raw = {"architecture": "Sumuvik", "vocab": 9, "width": 8, "norm": {"eps": 1e-6}, "layers": [
        {"type": "attention", "mixer": {"heads": 2, "dim": 4, "scale": 0.5, "mask": None, "rot": None}},
        {"type": "attention", "mixer": {"heads": 2, "dim": 4, "scale": 1, "mask": {"size": 3},
                                        "rot": {"dims": 2, "base": 10, "scaling": None}},
         "mlp": {"kind": "moe", "expert": {"ff": 3, "limit": 1}, "router": {"experts": 4, "top": 2}, "shared": None}}]}
    cfg = SumuvikConfig.from_dict(raw)
    a, b = (l.mixer for l in cfg.layers)
    assert cfg.embedding_scale == 1.0 and cfg.layers[0].mlp is None
    assert (a.kv_heads, a.vdim, a.window, a.keep_first, a.rot_dims, a.scaling) == (2, 4, 0, 0, 0, None)
    assert (b.window, b.keep_first, b.rot_base, b.scaling) == (3, 0, 10.0, None)
    m = cfg.layers[1].mlp
    assert (m.scale, m.groups, m.keep, m.shared) == (1.0, 1, 1, None)
    model = DecoderModel(resolve_architecture(raw).build_spec(cfg))
    names = {s.name for s in model.weight_specs() if s.load}
    assert "l0.norm2" not in names and "l1.norm2" in names and "l1.mlp.shared.up" not in names
    assert model.cache_needs()[0][0].kind == "full" and model.cache_needs()[1][0].kind == "window"


@pytest.mark.parametrize("change,message", [
    (lambda r: r.pop("vocab"), "vocab"),
    (lambda r: r.pop("norm"), "norm.eps"),
    (lambda r: r.update(layers=[]), "layers"),
    (lambda r: r["layers"][0].update(type="conv"), "type"),
    (lambda r: r["layers"][0].pop("mixer"), "mixer"),
    (lambda r: r["layers"][0]["mixer"].update(blocks=5), "blocks"),
    (lambda r: r["layers"][0]["mixer"].pop("conv"), "conv"),
    (lambda r: r["layers"][1]["mixer"].update(kv_heads=3), "multiple"),
    (lambda r: r["layers"][1]["mixer"].pop("scale"), "scale"),
    (lambda r: r["layers"][1]["mixer"].update(mask=7), "mask"),
    (lambda r: r["layers"][1]["mixer"]["mask"].update(size=0), "size"),
    (lambda r: r["layers"][1]["mixer"]["mask"].update(keep_first=-1), "keep_first"),
    (lambda r: r["layers"][1]["mixer"]["rot"].update(dims=7), "rot.dims"),
    (lambda r: r["layers"][1]["mixer"]["rot"].pop("base"), "base"),
    (lambda r: r["layers"][1]["mixer"]["rot"]["scaling"].pop("low"), "low"),
    (lambda r: r["layers"][1]["mixer"]["rot"]["scaling"].update(high=0.5), "high"),
    (lambda r: r["layers"][0]["mlp"].pop("limit"), "limit"),
    (lambda r: r["layers"][0]["mlp"].update(limit=-1.0), "limit"),
    (lambda r: r["layers"][0]["mlp"].update(kind="swiglu"), "dense"),
    (lambda r: r["layers"][1]["mlp"].pop("expert"), "expert"),
    (lambda r: r["layers"][1]["mlp"]["router"].update(groups={"count": 3, "keep": 1}), "groups"),
    (lambda r: r["layers"][1]["mlp"]["router"].update(top=5), "top"),
    (lambda r: r["layers"][1]["mlp"]["shared"].pop("limit"), "limit"),
])
def test_config_refusals(change, message):
    raw = copy.deepcopy(SUMUVIK["A"][0])
    change(raw)
    with pytest.raises(ConfigError, match=message):
        SumuvikConfig.from_dict(raw)


# ---- the model a configuration becomes -------------------------------------------------------------------
def test_spec_of_a_configuration():
    raw = SUMUVIK["A"][0]
    spec = resolve_architecture(raw).build_spec(SumuvikConfig.from_dict(raw))
    assert [l.mixer.kind for l in spec.layers] == ["rglru", "scored_attention", "rglru", "scored_attention"]
    assert [l.feed_forward and l.feed_forward.kind for l in spec.layers] == ["swiglu", "moe", "moe", None]
    assert all(l.block.kind == "parallel" for l in spec.layers) and spec.embedding.params["scale"] == 3.5
    m = spec.layers[1].mixer.params
    assert (m["mask"], m["mask_size"], m["keep_first"], m["sink_score"], m["qkv_bias"], m["rot_pairing"]) == \
        ("window", 20, 5, 0.0, True, "neighbours")
    f = spec.layers[1].feed_forward.params
    assert (f["router"], f["groups"], f["route_scale"], f["limit"], f["shared_limit"], f["alpha"], f["up_shift"]) == \
        ("sigmoid_groups", (4, 2), 1.7, 0.8, 1.2, 1.702, 1.0)
    needs = DecoderModel(spec).cache_needs()
    assert needs[0] == (None, needs[0][1]) and needs[0][1].tensors == {"rglru.state": (96,), "rglru.conv": (3, 96)}
    assert (needs[1][0].window, needs[1][0].keep_first, needs[1][0].planes) == (20, 5, (16, 8)) and needs[1][1] is None
    names = {s.name: s.shape for s in DecoderModel(spec).weight_specs()}
    assert names["l0.mix.ra"] == (4, 24, 24) and names["l0.mix.ri.b"] == (4, 24) and names["l0.mix.conv"] == (96, 4)
    assert names["l1.mix.q.b"] == (64,) and names["l1.mix.v.b"] == (16,) and names["l1.mix.g"] == (4, 64)
    assert names["l1.mlp.e7.down"] == (64, 24) and names["l1.mlp.correction"] == (8,) and names["l1.mlp.shared.gate"] == (40, 64)
    assert names["head"] == (211, 64) and "l1.mix.sink" not in names
    # A layer without a feed-forward reads no second norm, and takes a folder that stores one.
    assert [(s.optional, s.load) for s in DecoderModel(spec).weight_specs() if s.name == "l3.norm2"] == [(True, False)]


@pytest.mark.parametrize("bad", [
    {"keep_first": 2, "mask": "chunk", "mask_size": 4}, {"keep_first": -1}, {"rot_pairing": "thirds"},
    {"sink": True, "sink_score": 0.0}, {"qkv_bias": True, "v_norm": "head_unit"}])
def test_attention_options_that_do_not_go_together(bad):
    from llm_rs_b200.parts.scored_attention import ScoredAttention
    with pytest.raises(ValueError):
        ScoredAttention(**{"hidden_size": 8, "n_heads": 2, "n_kv_heads": 1, "dim": 4, "vdim": 4, "scale": 1.0,
                           "mask": "window", "mask_size": 4, **bad})


@pytest.mark.parametrize("bad", [
    {"groups": (3, 1)}, {"groups": (4, 5)}, {"groups": (4, 1), "top": 3}, {"router": "linear", "groups": (2, 1)},
    {"router": "linear", "route_scale": 2.0}])
def test_router_options_that_do_not_go_together(bad):
    from llm_rs_b200.parts.moe import MixtureOfExperts
    with pytest.raises(ValueError):
        MixtureOfExperts(**{"hidden_size": 8, "expert_size": 4, "n_experts": 8, "top": 2, "router": "sigmoid_groups", **bad})


# ---- pages of a window that keeps first tokens -----------------------------------------------------------
def _manager(window, keep, page, pages, slots=3):
    return CacheManager([GroupSpec(CacheNeed("window", 1, 4, window, keep_first=keep), [0], pages)], page, slots)


@pytest.mark.parametrize("window,keep,page", [(5, 0, 4), (5, 1, 4), (5, 4, 4), (5, 5, 4), (9, 30, 8), (40, 3, 8), (1, 17, 16)])
@pytest.mark.parametrize("cuts", [[1] * 90, [90], [2, 33, 1, 1, 20, 33], [64, 26]])
def test_exactly_the_pages_that_are_read_stay(window, keep, page, cuts):
    """After every step a page is held exactly when it holds one of the first ``keep`` tokens or a key that the next query
    sees, and during a step every page that one of its queries sees is there."""
    m = _manager(window, keep, page, 64)
    m.admit("a")
    at = 0
    for n in cuts:
        m.reserve("a", n)
        table = m.table("a", 0)
        seen = {j // page for i in range(at, at + n) for j in range(i + 1) if i - j < window or j < keep}
        assert all(table[p] >= 0 for p in seen)
        m.commit("a", n)
        at += n
        table = m.table("a", 0)
        for p in range(len(table)):
            needed = p * page < keep or at - ((p + 1) * page - 1) < window      # its last key may still be seen
            assert (table[p] >= 0) == needed, (at, p)
        m.check_invariants()
    m.release("a")
    assert m.free_pages(0) == 64


def test_a_request_that_starts_late_still_gets_its_first_pages():
    """What a request that is not live would take when it starts at a cached length: the window's pages and those that hold
    the kept tokens."""
    m = _manager(4, 6, 4, 32)
    assert m.pages_needed(None, 2, cached_len=40) == [2 + 2]      # pages of keys 37 .. 41, and of tokens 0 .. 5
    assert m.pages_needed(None, 3) == [1]


# ---- frequencies ------------------------------------------------------------------------------------------
@pytest.mark.parametrize("dims,base,scaling", [
    (8, 500.0, None), (24, 1e5, (6.0, 1.0, 3.0, 256)), (128, 5e5, (32.0, 1.0, 4.0, 8192)), (6, 100.0, (3.0, 1.0, 1.0, 9)),
    (20, 1e4, (2.0, 2.0, 6.0, 200)), (0, 10.0, None)])
def test_rescaled_frequencies(dims, base, scaling):
    sc = dict(zip(("factor", "low", "high", "original"), scaling)) if scaling else None
    got = wavelength_scaled_frequencies(dims, base, sc)
    assert torch.allclose(got, P.frequencies(dims, base, sc), rtol=1e-13, atol=0)


def test_rescaled_frequencies_by_hand():
    f = P.frequencies(16, 1e4, {"factor": 8.0, "low": 1.0, "high": 4.0, "original": 256})
    plain = P.frequencies(16, 1e4)
    turns = 256 * plain / (2 * math.pi)
    assert bool((f[turns > 4] == plain[turns > 4]).all()) and bool((turns > 4).any())
    assert torch.allclose(f[turns < 1], plain[turns < 1] / 8) and bool((turns < 1).any())
    mid = (turns >= 1) & (turns <= 4)
    s = (turns[mid] - 1) / 3
    assert bool(mid.any()) and torch.allclose(f[mid], (1 - s) * plain[mid] / 8 + s * plain[mid])


# ---- the plain implementation's own properties ---------------------------------------------------------------
def _rand(seed):
    g = torch.Generator().manual_seed(seed)
    return lambda *s: torch.randn(*s, generator=g, dtype=F64)


def test_what_a_query_sees():
    seen = P.visible(20, 4, 3)
    for i in range(20):
        assert [j for j in range(20) if seen[i, j]] == [j for j in range(i + 1) if i - j < 4 or j < 3]
    assert torch.equal(P.visible(9, 0, 3), torch.ones(9, 9).tril().bool())


def test_one_is_added_to_the_denominator():
    s = torch.tensor([[0.5, -1.0, 200.0]], dtype=F64)
    seen = torch.tensor([[True, True, False]])
    want = torch.tensor([math.exp(0.5), math.exp(-1.0)], dtype=F64) / (1 + math.exp(0.5) + math.exp(-1.0))
    assert torch.allclose(P.softmax_plus_one(s, seen)[0, :2], want) and float(P.softmax_plus_one(s, seen)[0, 2]) == 0.0
    assert float(P.softmax_plus_one(torch.full((1, 3), -400.0, dtype=F64), seen.fill_(True)).sum()) < 1e-100


def test_rotation_turns_neighbours():
    x = torch.tensor([[[1.0, 0.0, 0.0, 2.0, 7.0]]], dtype=F64)
    y = P.rotate_pairs(x, torch.tensor([3]), 4, 100.0)[0, 0]
    a, b = 3.0, 3.0 / 10.0
    want = [math.cos(a), math.sin(a), -2 * math.sin(b), 2 * math.cos(b), 7.0]
    assert torch.allclose(y, torch.tensor(want, dtype=F64))


def test_recurrence_is_a_decayed_sum():
    r = _rand(1)
    T, W = 7, 5
    u, rg, ig, lam = r(T, W), torch.sigmoid(r(T, W)), torch.sigmoid(r(T, W)), r(W)
    S = P.linear_recurrence(u, rg, ig, lam)
    for t in range(T):
        want = torch.zeros(W, dtype=F64)
        for s in range(t + 1):
            fade = torch.ones(W, dtype=F64)
            for k in range(s + 1, t + 1):
                fade = fade * torch.exp(-8 * rg[k] * torch.log1p(torch.exp(lam)))
            a = torch.exp(-8 * rg[s] * torch.log1p(torch.exp(lam)))
            want += fade * torch.sqrt(1 - a * a) * ig[s] * u[s]
        assert torch.allclose(S[t], want, atol=1e-12)


def test_the_convolution_reads_zeros_before_the_start():
    """Not the projection's bias: a token before the start does not exist."""
    x = torch.tensor([[1.0], [10.0], [100.0]], dtype=F64)
    y = P.short_conv(x, torch.tensor([[5.0, 3.0, 2.0]], dtype=F64), torch.tensor([0.5], dtype=F64))
    assert y[:, 0].tolist() == [2.5, 23.5, 235.5]


def test_routing_by_hand():
    s = torch.tensor([0.9, 0.1, 0.5, 0.5, 0.2, 0.6], dtype=F64)
    none = torch.zeros(6, dtype=F64)
    assert P.route(s, none, 2, None, 2.0) == [(0, 2 * 0.9 / 1.5), (5, 2 * 0.6 / 1.5)]
    # Groups of two are worth 1.0, 1.0 and 0.8: with the best one only the lower of two equals is kept.
    assert [e for e, _ in P.route(s, none, 2, {"count": 3, "keep": 1}, 1.0)] == [0, 1]
    assert [e for e, _ in P.route(s, none, 2, {"count": 3, "keep": 2}, 1.0)] == [0, 2]
    # Choice scores below zero are still chosen inside a kept group, and the weights do not know the correction.
    low = torch.tensor([-3.0, -3.0, -5.0, -5.0, -5.0, -5.0], dtype=F64)
    got = P.route(s, low, 2, {"count": 3, "keep": 1}, 1.0)
    assert [e for e, _ in got] == [0, 1] and abs(got[0][1] - 0.9) < 1e-12 and abs(got[1][1] - 0.1) < 1e-12


def test_every_mechanism_moves_the_logits(tmp_path):
    """Leaving out any mechanism changes what the model computes by a visible share: a GPU test against it would notice."""
    cfg, w = P.load_model_dir(write_sumuvik_model("A", str(tmp_path)))
    toks = torch.randint(0, cfg["vocab"], (60,), generator=torch.Generator().manual_seed(4)).tolist()
    base = P.forward(toks, cfg, w)

    def moved(change=None, **tensors):
        c = copy.deepcopy(cfg)
        if change:
            change(c)
        return float((P.forward(toks, c, {**w, **tensors}) - base).abs().max() / base.abs().max())
    for name in ("l1.mix.q.b", "l1.mix.k.b", "l1.mix.v.b", "l1.mix.g", "l0.mix.y.b", "l0.mix.x.b", "l0.mix.conv.b",
                 "l0.mix.ra", "l0.mix.ri", "l0.mix.ra.b", "l0.mix.ri.b", "l0.mix.lam", "l1.mlp.correction"):
        assert moved(**{name: 0 * w[name]}) > 0.01, name
    A = lambda c: c["layers"][1]
    for what, change in {
            "kept": lambda c: A(c)["mixer"]["mask"].update(keep_first=0), "kept one less": lambda c: A(c)["mixer"]["mask"].update(keep_first=4),
            "window": lambda c: A(c)["mixer"]["mask"].update(size=19), "scaling": lambda c: A(c)["mixer"]["rot"].pop("scaling"),
            "groups": lambda c: A(c)["mlp"]["router"].pop("groups"), "scale": lambda c: A(c)["mlp"]["router"].update(scale=1.0),
            "shared": lambda c: A(c)["mlp"].pop("shared"), "limit": lambda c: A(c)["mlp"]["expert"].update(limit=9.0),
            "shared limit": lambda c: A(c)["mlp"]["shared"].update(limit=9.0), "dense limit": lambda c: c["layers"][0]["mlp"].update(limit=9.0),
            "embedding": lambda c: c["embedding"].update(scale=1.0)}.items():
        assert moved(change) > 0.004, what
