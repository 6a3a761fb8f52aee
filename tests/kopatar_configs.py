"""Small Kopatar configurations for the tests: they differ in every size and option (layer order, loops over the middle,
the whole and a single layer, one pass, none; grouped and single key heads, key and value widths that differ, ranks that
are multiples of nothing, windows shorter and longer than a page and of one token, partial and full rotation, decays of 0
and 1, groups of one and several heads, norm groups that cut across heads, convolutions of one to five taps, layers without
a feed-forward)."""
import os

import torch


def _delta(heads, kv_heads, dim, vdim, conv, decay_rank, gate_rank):
    return {"type": "channel_delta", "mixer": {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "conv": conv,
                                               "decay_rank": decay_rank, "gate_rank": gate_rank}}


def _retention(heads, dim, vdim, decay, base, rot):
    return {"type": "retention", "mixer": {"heads": heads, "dim": dim, "vdim": vdim, "decay": decay,
                                           "rot": {"base": base, "dims": rot}}}


def _parallel(left, right, left_scale, right_scale):
    heads, kv_heads, dim, vdim, scale, window = left
    r_heads, r_vdim, state, groups, conv, norm_groups = right
    return {"type": "parallel", "mixer": {
        "left": {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "scale": scale, "mask": {"size": window}},
        "right": {"heads": r_heads, "vdim": r_vdim, "state": state, "groups": groups, "conv": conv,
                  "norm_groups": norm_groups},
        "left_scale": left_scale, "right_scale": right_scale}}


def _layers(*pairs):
    return [{**mixer, "mlp": None if ff is None else {"kind": "dense", "ff": ff}} for mixer, ff in pairs]


# The middle two layers run twice, one layer before and one (without a feed-forward) after them; grouped key heads; a
# partial rotation; a window of 20 over pages of 16; norm groups that cut across the heads.
KOPATAR_A = {
    "architecture": "Kopatar", "vocab": 211, "width": 64, "norm": {"eps": 1e-5},
    "loop": {"start": 1, "stop": 3, "times": 2},
    "layers": _layers(
        (_delta(4, 2, 16, 8, 4, 12, 20), 80),
        (_retention(3, 16, 24, [0.9, 0.97, 0.995], 500.0, 8), 48),
        (_parallel((4, 2, 16, 8, 0.3, 20), (4, 12, 10, 2, 2, 3), 0.6, 1.2), 64),
        (_delta(2, 2, 8, 24, 2, 8, 8), None))}

# No loop; the parallel mixer first, a window of 7 over pages of 8; one group for all heads; a full rotation; an odd width.
KOPATAR_B = {
    "architecture": "Kopatar", "vocab": 157, "width": 72, "norm": {"eps": 1e-6},
    "layers": _layers(
        (_parallel((3, 3, 8, 24, 0.35, 7), (2, 20, 16, 1, 3, 5), 0.9, 0.8), 50),
        (_retention(2, 20, 12, [0.95, 0.99], 1e4, 20), None),
        (_delta(6, 3, 24, 12, 3, 10, 6), 36),
        (_parallel((6, 2, 12, 12, 0.28, 64), (6, 8, 12, 3, 4, 2), 1.0, 1.0), 44))}

# Sizes at which the bfloat16 kernels take the tensor cores; every layer runs three times; windows of 48 and 130; keys of
# 128 channels in the delta rule, states of 64 and 128 rows.
KOPATAR_C = {
    "architecture": "Kopatar", "vocab": 640, "width": 256, "norm": {"eps": 1e-6},
    "loop": {"start": 0, "stop": 4, "times": 3},
    "layers": _layers(
        (_parallel((8, 2, 64, 32, 0.11, 48), (8, 32, 64, 4, 4, 1), 0.75, 1.1), 256),
        (_delta(4, 2, 128, 64, 4, 16, 32), 128),
        (_retention(4, 64, 128, [0.96, 0.98, 0.99, 0.999], 1e6, 32), 192),
        (_parallel((4, 4, 128, 128, 0.09, 130), (4, 64, 128, 2, 3, 4), 1.1, 0.7), 320))}

# Sizes that are multiples of nothing (width 100, a vocabulary of 61), convolutions of ONE tap (no rows to carry), a window
# of ONE token, a loop of one pass over the first layer, three value heads over one key head, heads of seven channels.
KOPATAR_D = {
    "architecture": "Kopatar", "vocab": 61, "width": 100, "norm": {"eps": 1e-6},
    "loop": {"start": 0, "stop": 1, "times": 1},
    "layers": _layers(
        (_delta(3, 1, 12, 20, 1, 5, 7), 36),
        (_parallel((5, 1, 40, 6, 0.2, 1), (3, 7, 9, 3, 1, 7), 1.0, 0.5), 28),
        (_retention(1, 6, 10, [0.98], 300.0, 2), 33))}

# Recurrent layers only (no pages at all); the last layer runs four times; decays of 0 (a head that sees its own token
# only) and 1 (one that never forgets).
KOPATAR_E = {
    "architecture": "Kopatar", "vocab": 130, "width": 48, "norm": {"eps": 1e-5},
    "loop": {"start": 2, "stop": 3, "times": 4},
    "layers": _layers(
        (_retention(4, 8, 16, [0.0, 0.5, 0.999, 1.0], 77.0, 4), 64),
        (_delta(2, 1, 32, 16, 5, 16, 4), 40),
        (_retention(2, 16, 8, [0.9, 0.99], 1e5, 16), 32))}

# Parallel mixers only, windows of 33 and 9 over pages of 32: every page comes back as the windows pass.
KOPATAR_F = {
    "architecture": "Kopatar", "vocab": 97, "width": 40, "norm": {"eps": 1e-6},
    "loop": {"start": 0, "stop": 2, "times": 2},
    "layers": _layers(
        (_parallel((2, 2, 16, 16, 0.25, 33), (4, 10, 8, 1, 5, 4), 0.8, 0.8), 40),
        (_parallel((4, 2, 8, 12, 0.35, 9), (2, 16, 20, 2, 3, 1), 0.5, 1.5), None))}

# name -> (config.json, seed, sigma of matrices, page size)
KOPATAR = {"A": (KOPATAR_A, 3, 0.13, 16), "B": (KOPATAR_B, 4, 0.13, 8), "C": (KOPATAR_C, 5, 0.055, 16),
           "D": (KOPATAR_D, 6, 0.11, 16), "E": (KOPATAR_E, 7, 0.15, 16), "F": (KOPATAR_F, 8, 0.17, 32)}


def shape_weights(tensors, seed, dtype):
    """Random weights reworked in place so that the mechanisms show and stay well conditioned: keys that lean towards their
    own token's query in the two recurrences whose output is divided by its size (the first token's output is otherwise
    a number near zero divided by itself), decays that forget within tens to hundreds of tokens and differ from channel to
    channel, loop vectors and embeddings of the stream's size."""
    g = torch.Generator().manual_seed(1000 + seed)
    for key in sorted(tensors):
        t = tensors[key]
        if key == "embed" or key == "loop.step":
            tensors[key] = (torch.randn(t.shape, generator=g) * (1.0 if key == "embed" else 0.5)).to(dtype)
        elif key.endswith(".A_log"):
            tensors[key] = (0.5 * torch.randn(t.shape, generator=g) - 1.5).to(dtype)
        elif key.endswith(".dt_bias"):
            tensors[key] = (torch.randn(t.shape, generator=g) - 1.5).to(dtype)
        elif key.endswith(".a2"):
            tensors[key] = (4.0 * t.float()).to(dtype)
        elif key.endswith(".conv.b"):
            tensors[key] = (0.3 * torch.randn(t.shape, generator=g)).to(dtype)
        elif key.endswith("mix.k") or key.endswith("mix.k.conv"):
            q = tensors[key.replace("mix.k", "mix.q")].float()
            tensors[key] = (0.8 * q + 0.6 * t.float()).to(dtype)
    return tensors


def write_kopatar_model(name: str, folder: str, dtype=torch.bfloat16) -> str:
    """Write a small Kopatar folder with random weights (see ``shape_weights``); returns its path."""
    import json

    from llm_rs_b200.config import KopatarConfig, resolve_architecture
    from llm_rs_b200.parts import DecoderModel
    from llm_rs_b200.weights.random_init import random_tensors
    from llm_rs_b200.weights.safetensors_io import save_file
    raw, seed, sigma, _ = KOPATAR[name]
    cfg = KopatarConfig.from_dict(raw)
    path = os.path.join(folder, f"kopatar_{name}")
    model = DecoderModel(resolve_architecture(raw).build_spec(cfg))
    tensors = shape_weights(random_tensors(model.weight_specs(), seed, sigma, 0.3, dtype, "cpu"), seed, dtype)
    os.makedirs(path, exist_ok=True)
    # The ranks of the low-rank projections are left to the tensors' shapes, as in a checkpoint.
    made = cfg.to_dict()
    for layer in made["layers"]:
        layer["mixer"].pop("decay_rank", None)
        layer["mixer"].pop("gate_rank", None)
    with open(os.path.join(path, "config.json"), "w") as f:
        json.dump(made, f, indent=2)
    save_file(tensors, os.path.join(path, "model.safetensors"))
    return path
