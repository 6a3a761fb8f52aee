"""The Kopatar design without a GPU: its configuration (every key, optional keys absent, refusals, ranks from the tensors'
shapes), the model a configuration is turned into (part kinds, run order of a loop, pages and state per entry, tensor
names), and the plain implementation's own properties (tests/plain_kopatar.py is the oracle of the GPU tests, so what it
computes is pinned here by hand-made cases)."""
import copy
import math

import pytest
import torch

import plain_kopatar as P
from kopatar_configs import KOPATAR, write_kopatar_model
from llm_rs_b200.config import ConfigError, KopatarConfig, load_config, resolve_architecture
from llm_rs_b200.parts import DecoderModel

F64 = torch.float64


# ---- configuration ------------------------------------------------------------------------------------
@pytest.mark.parametrize("name", list(KOPATAR))
def test_config_round_trip(name):
    raw = KOPATAR[name][0]
    cfg = KopatarConfig.from_dict(raw)
    assert KopatarConfig.from_dict(cfg.to_dict()) == cfg
    assert resolve_architecture(raw).config_cls is KopatarConfig


def test_optional_keys():
    raw = {"architecture": "Kopatar", "vocab": 9, "width": 8, "norm": {"eps": 1e-6}, "loop": None, "layers": [
        {"type": "retention", "mixer": {"heads": 1, "dim": 4, "decay": [1]}, "mlp": None},
        {"type": "parallel", "mixer": {"left": {"heads": 2, "dim": 4, "scale": 0.5},
                                       "right": {"heads": 2, "vdim": 3, "state": 4, "conv": 2}}}]}
    cfg = KopatarConfig.from_dict(raw)
    assert cfg.loop is None and cfg.layers[0].mixer.rot_dims == 0 and cfg.layers[0].mixer.vdim == 4
    m = cfg.layers[1].mixer
    assert (m.left.kv_heads, m.left.vdim, m.left.window, m.left_scale, m.right_scale) == (2, 4, 0, 1.0, 1.0)
    assert (m.right.groups, m.right.norm_groups) == (1, 1) and cfg.layers[1].mlp is None
    model = DecoderModel(resolve_architecture(raw).build_spec(cfg))
    names = {s.name for s in model.weight_specs()}
    assert "l0.norm2" not in names and "l0.norm1" in names and "loop.step" not in names
    assert model.cache_needs()[1][0].kind == "full"


@pytest.mark.parametrize("change,message", [
    (lambda r: r.pop("vocab"), "vocab"),
    (lambda r: r.update(layers=[]), "layers"),
    (lambda r: r["layers"][0].update(type="conv"), "type"),
    (lambda r: r["layers"][0]["mixer"].update(kv_heads=3), "multiple"),
    (lambda r: r["layers"][0]["mixer"].pop("decay_rank"), "decay_rank"),
    (lambda r: r["layers"][0]["mixer"].pop("conv"), "conv"),
    (lambda r: r["layers"][1]["mixer"].update(decay=[0.5]), "decay"),
    (lambda r: r["layers"][1]["mixer"].update(decay=[0.5, 0.5, 1.5]), "decay"),
    (lambda r: r["layers"][1]["mixer"].update(rot={"base": 10.0, "dims": 7}), "rot.dims"),
    (lambda r: r["layers"][2]["mixer"].pop("left"), "left"),
    (lambda r: r["layers"][2]["mixer"]["left"].pop("scale"), "scale"),
    (lambda r: r["layers"][2]["mixer"]["right"].update(groups=3), "groups"),
    (lambda r: r["layers"][2]["mixer"]["right"].update(norm_groups=7), "norm_groups"),
    (lambda r: r["layers"][2]["mixer"].update(left_scale="one"), "left_scale"),
    (lambda r: r["layers"][0].update(mlp={"kind": "moe", "ff": 3}), "dense"),
    (lambda r: r["loop"].update(stop=9), "loop"),
    (lambda r: r["loop"].update(start=3), "loop"),
    (lambda r: r["loop"].update(times=0), "times"),
])
def test_config_refusals(change, message):
    raw = copy.deepcopy(KOPATAR["A"][0])
    change(raw)
    with pytest.raises(ConfigError, match=message):
        KopatarConfig.from_dict(raw)


def test_tensor_shapes_give_the_ranks(tmp_path):
    entry, cfg = load_config(write_kopatar_model("D", str(tmp_path)))
    assert (cfg.layers[0].mixer.decay_rank, cfg.layers[0].mixer.gate_rank) == (5, 7)
    assert cfg == KopatarConfig.from_dict(KOPATAR["D"][0])


# ---- the model a configuration becomes -------------------------------------------------------------------
def test_spec_of_a_configuration():
    raw = KOPATAR["A"][0]
    spec = resolve_architecture(raw).build_spec(KopatarConfig.from_dict(raw))
    assert [l.mixer.kind for l in spec.layers] == ["channel_delta", "retention", "parallel", "channel_delta"]
    assert all(l.block.kind == "prenorm" for l in spec.layers)
    assert spec.layers[3].feed_forward is None and spec.layers[3].feed_forward_norm is None
    assert spec.layers[0].feed_forward.params["activation"] == "xielu"
    left, right = (spec.layers[2].mixer.params[k] for k in ("left", "right"))
    assert (left.kind, right.kind) == ("scored_attention", "mamba2")
    assert (left.params["qk_norm"], left.params["gate_per"], left.params["mask"], left.params["mask_size"]) == \
        ("head", "channel", "window", 20)
    assert spec.layers[1].mixer.params["k_scale"] == 16 ** -0.5 and spec.layers[0].mixer.params["q_scale"] == 16 ** -0.5
    assert [(s.layer, s.reenter, s.pass_index) for s in spec.run_order] == [
        (0, False, 0), (1, True, 0), (2, False, 0), (1, True, 1), (2, False, 1), (3, False, 0)]
    assert [(s.layer, s.pass_index if s.reenter else None) for s in spec.run_order] == P.layer_order(raw)
    model = DecoderModel(spec)
    needs = model.cache_needs()
    assert [n[0] is not None for n in needs] == [False, False, True, False, True, False]
    assert needs[2][0].window == 20 and needs[2][0].planes == (16, 8)
    assert needs[0][1].tensors == {"gated_delta.state": (4, 16, 8), "gated_delta.conv": (3, 96)}
    assert needs[1][1].tensors == {"recurrent.state": (3, 16, 24)}
    assert needs[2][1].tensors == {"ssd.state": (4, 10, 12), "ssd.conv": (1, 88)}
    names = {s.name: s.shape for s in model.weight_specs()}
    assert names["l0.mix.a1"] == (12, 64) and names["l0.mix.a2"] == (64, 12) and names["l0.mix.dt_bias"] == (64,)
    assert names["l0.mix.g1"] == (20, 64) and names["l0.mix.g2"] == (32, 20) and names["l0.mix.v.conv"] == (32, 4)
    assert names["l2.mix.left.q.norm"] == (16,) and names["l2.mix.left.g"] == (32, 64)
    assert names["l2.mix.right.in"] == (48 + 88 + 4, 64) and names["l2.mix.right.conv.b"] == (88,)
    assert names["loop.step"] == (2, 64) and names["l0.mlp.act"] == (2,) and "l3.norm2" not in names
    assert "l1.mix.norm" not in names and all(s.name != "head" or not s.load for s in model.weight_specs())


@pytest.mark.parametrize("name", list(KOPATAR))
def test_run_order_is_the_plain_one(name):
    raw = KOPATAR[name][0]
    spec = resolve_architecture(raw).build_spec(KopatarConfig.from_dict(raw))
    assert [(s.layer, s.pass_index if s.reenter else None) for s in spec.run_order] == P.layer_order(raw)
    assert (spec.reentry is None) == ("loop" not in raw)


def test_joined_rows_start_on_multiples_of_eight():
    from llm_rs_b200.parts.linear import joined_rows
    ws = [torch.full((n, 3), float(n)) for n in (5, 8, 1)]
    w, starts = joined_rows(ws)
    assert starts == [0, 8, 16] and w.shape == (24, 3)
    for t, s in zip(ws, starts):
        assert torch.equal(w[s:s + t.size(0)], t)
    assert w[5:8].abs().sum() == 0 and w[17:].abs().sum() == 0


# ---- the plain implementation's own properties ---------------------------------------------------------------
def _rand(g):
    return lambda *s: torch.randn(*s, generator=g, dtype=F64)


def test_xielu_by_hand():
    act = torch.tensor([0.4, -0.7], dtype=F64)
    up, down = math.log1p(math.exp(0.4)), 0.5 + math.log1p(math.exp(-0.7))
    for z in (-3.0, -1e-3, 0.0, 1e-3, 2.5):
        want = up * z * z + z / 2 if z > 0 else down * (math.exp(z) - 1 - z) + z / 2
        assert abs(float(P.xielu(torch.tensor([z], dtype=F64), act)[0]) - want) < 1e-12


def test_a_token_outside_the_window_has_no_influence():
    g = torch.Generator().manual_seed(0)
    r, D = _rand(g), 12
    m = {"heads": 2, "kv_heads": 1, "dim": 8, "vdim": 6, "scale": 0.3, "mask": {"size": 5}}
    w = {"m.q": r(16, D), "m.k": r(8, D), "m.v": r(6, D), "m.g": r(12, D), "m.o": r(D, 12),
         "m.q.norm": 1 + 0.2 * r(8), "m.k.norm": 1 + 0.2 * r(8)}
    x = r(20, D)
    y = P.gated_window_attention(x, m, w, "m.", 1e-6, torch.arange(20))
    x2 = x.clone()
    x2[7] += 3.0
    y2 = P.gated_window_attention(x2, m, w, "m.", 1e-6, torch.arange(20))
    assert torch.equal(y[12:], y2[12:]) and not torch.allclose(y[11], y2[11]) and torch.equal(y[:7], y2[:7])


def test_retention_is_a_decayed_sum_of_scores():
    """o_t = sum_s decay^(t - s) (q_t . k_s) v_s with rotated q and k."""
    g = torch.Generator().manual_seed(1)
    r, D, T = _rand(g), 10, 9
    m = {"heads": 2, "dim": 6, "vdim": 4, "decay": [0.9, 0.5], "rot": {"base": 50.0, "dims": 4}}
    w = {"m.q": r(12, D), "m.k": r(12, D), "m.v": r(8, D), "m.g": r(8, D), "m.o": r(D, 8)}
    x, pos = r(T, D), torch.arange(T)
    q = P.rotate_halves((x @ w["m.q"].T).view(T, 2, 6), pos, 4, 50.0)
    k = P.rotate_halves((x @ w["m.k"].T).view(T, 2, 6), pos, 4, 50.0) * 6 ** -0.5
    v = (x @ w["m.v"].T).view(T, 2, 4)
    o = torch.zeros(T, 2, 4, dtype=F64)
    for h in range(2):
        for t in range(T):
            for s in range(t + 1):
                o[t, h] += m["decay"][h] ** (t - s) * (q[t, h] @ k[s, h]) * v[s, h]
    want = (P.rms(o, 1e-6).reshape(T, 8) * P.silu(x @ w["m.g"].T)) @ w["m.o"].T
    assert torch.allclose(P.retention(x, m, w, "m.", 1e-6, pos), want, atol=1e-10)


def test_channel_decay_of_equal_channels_is_a_scalar_decay():
    """With no low-rank part and equal biases every channel decays alike: the rule of one decay per head; a decay of zero
    (a large bias) leaves the token's own write alone."""
    g = torch.Generator().manual_seed(2)
    r, D, T = _rand(g), 10, 7
    m = {"heads": 2, "kv_heads": 1, "dim": 4, "vdim": 3}
    w = {"m.q": r(4, D), "m.k": r(4, D), "m.v": r(6, D), "m.b": r(2, D), "m.a1": r(3, D), "m.a2": 0 * r(8, 3),
         "m.A_log": r(2), "m.dt_bias": torch.full((8,), 60.0, dtype=F64), "m.g1": r(2, D), "m.g2": r(6, 2), "m.norm": 1 + r(3),
         "m.o": r(D, 6), "m.q.conv": r(4, 2), "m.k.conv": r(4, 2), "m.v.conv": r(6, 2)}
    w["m.A_log"] = torch.tensor([1.0, 1.0], dtype=F64)
    x = r(T, D)
    y = P.channel_delta(x, m, w, "m.", 1e-6)
    conv = lambda n, wd: P.silu(P.short_conv(x @ w["m." + n].T, w["m." + n + ".conv"])).view(T, -1, wd)
    q, k, v = P.unit(conv("q", 4)) * 0.5, P.unit(conv("k", 4)), conv("v", 3)
    own = torch.sigmoid(x @ w["m.b"].T)[:, :, None] * v * (q * k).sum(-1, keepdim=True)
    gate = torch.sigmoid((x @ w["m.g1"].T) @ w["m.g2"].T)
    want = ((P.rms(own, 1e-6) * w["m.norm"]).reshape(T, 6) * gate) @ w["m.o"].T
    assert torch.allclose(y, want, atol=1e-9)


def test_mamba2_is_a_decayed_sum():
    """y_t = D x_t + sum_s (product of the decays after s) dt_s (C_t . B_s) x_s, gate before the norm in parts."""
    g = torch.Generator().manual_seed(3)
    r, D, T = _rand(g), 8, 6
    m = {"heads": 2, "vdim": 3, "state": 4, "groups": 1, "norm_groups": 3, "conv": 2}
    w = {"m.in": r(6 + 6 + 8 + 2, D), "m.conv": r(14, 2), "m.conv.b": r(14), "m.dt_bias": r(2), "m.A_log": r(2), "m.D": r(2),
         "m.norm": 1 + 0.1 * r(6), "m.o": r(D, 6)}
    x = r(T, D)
    p = x @ w["m.in"].T
    z, xbc, dt = p[:, :6], P.silu(P.short_conv(p[:, 6:20], w["m.conv"], w["m.conv.b"])), P.softplus(p[:, 20:] + w["m.dt_bias"])
    X, B, C = xbc[:, :6].view(T, 2, 3), xbc[:, 6:10], xbc[:, 10:14]
    y = torch.zeros(T, 2, 3, dtype=F64)
    for h in range(2):
        for t in range(T):
            y[t, h] = w["m.D"][h] * X[t, h]
            for s in range(t + 1):
                fade = torch.exp(-torch.exp(w["m.A_log"][h]) * dt[s + 1:t + 1, h].sum())
                y[t, h] += fade * dt[s, h] * (C[t] @ B[s]) * X[s, h]
    y = (y.reshape(T, 6) * P.silu(z)).view(T, 3, 2)
    y = y / torch.sqrt((y * y).mean(-1, keepdim=True) + 1e-6)
    assert torch.allclose(P.mamba2(x, m, w, "m.", 1e-6), (y.reshape(T, 6) * w["m.norm"]) @ w["m.o"].T, atol=1e-10)


def test_every_mechanism_moves_the_logits(tmp_path):
    """Leaving out the loop's vector, its embedding, a pass, one side of the parallel mixer or a convolution's bias changes
    what model A computes by a visible share: a GPU test against it would notice."""
    cfg, w = P.load_model_dir(write_kopatar_model("A", str(tmp_path)))
    toks = torch.randint(0, cfg["vocab"], (40,), generator=torch.Generator().manual_seed(4)).tolist()
    base = P.forward(toks, cfg, w)

    def moved(c=cfg, **changed):
        return float((P.forward(toks, c, {**w, **changed}) - base).abs().max() / base.abs().max())
    assert moved(**{"loop.step": w["loop.step"].flip(0)}) > 0.02
    once = copy.deepcopy(cfg)
    once["loop"]["times"] = 1
    assert moved(once) > 0.05
    for side in ("left_scale", "right_scale"):
        c = copy.deepcopy(cfg)
        c["layers"][2]["mixer"][side] = 0.0
        assert moved(c) > 0.02, side
    assert moved(**{"l2.mix.right.conv.b": 0 * w["l2.mix.right.conv.b"]}) > 0.01
    assert moved(**{"l0.mix.a2": 0 * w["l0.mix.a2"]}) > 0.01
    assert moved(**{"l2.mix.left.g": 0 * w["l2.mix.left.g"]}) > 0.01
