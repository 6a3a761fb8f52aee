"""Small Sumuvik configurations for the tests: they differ in every size and option (layer order, grouped and single key
heads, key and value widths that differ, windows shorter and longer than a page and of one token, first tokens kept beside
them: none, one, part of a page, more than the window; partial, full and no rotation with and without rescaled frequencies,
convolutions of one to five taps, diagonal blocks of odd and even sizes, dense and routed feed-forwards with and without
groups of experts and a shared expert, layers without a feed-forward, small and large limits)."""
import json
import os

import torch


def _attention(heads, kv_heads, dim, vdim, scale, window=0, keep=0, rot=None, scaling=None):
    m = {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "scale": scale}
    if window:
        m["mask"] = {"size": window, "keep_first": keep}
    if rot:
        m["rot"] = {"base": rot[0], "dims": rot[1]}
        if scaling:
            m["rot"]["scaling"] = dict(zip(("factor", "low", "high", "original"), scaling))
    return {"type": "attention", "mixer": m}


def _rglru(width, blocks, conv):
    return {"type": "rglru", "mixer": {"width": width, "blocks": blocks, "conv": conv}}


def _dense(ff, limit):
    return {"kind": "dense", "ff": ff, "limit": limit}


def _moe(ff, limit, experts, top, scale=1.0, groups=None, shared=None):
    router = {"experts": experts, "top": top, "scale": scale}
    if groups:
        router["groups"] = {"count": groups[0], "keep": groups[1]}
    f = {"kind": "moe", "expert": {"ff": ff, "limit": limit}, "router": router}
    if shared:
        f["shared"] = {"ff": shared[0], "limit": shared[1]}
    return f


def _layers(*pairs):
    return [{**mixer, "mlp": f} for mixer, f in pairs]


# Both mixers with both feed-forwards and none; a window of 20 over pages of 16 with five kept tokens.
SUMUVIK_A = {
    "architecture": "Sumuvik", "vocab": 211, "width": 64, "norm": {"eps": 1e-5}, "embedding": {"scale": 3.5},
    "layers": _layers(
        (_rglru(96, 4, 4), _dense(80, 1.5)),
        (_attention(4, 2, 16, 8, 0.3, 20, 5, (500.0, 8), (4.0, 1.0, 3.0, 40)), _moe(24, 0.8, 8, 2, 1.7, (4, 2), (40, 1.2))),
        (_rglru(48, 2, 3), _moe(16, 2.0, 6, 3, 0.6, (2, 1))),
        (_attention(6, 3, 8, 24, 0.35, 33, 1, (1e4, 8)), None))}

# Attention over every key, without rotation; one kept token beside a window of 7 over pages of 8; an odd width.
SUMUVIK_B = {
    "architecture": "Sumuvik", "vocab": 157, "width": 72, "norm": {"eps": 1e-6}, "embedding": {"scale": 0.7},
    "layers": _layers(
        (_attention(3, 3, 8, 24, 0.35, 7, 1, (300.0, 2)), _moe(20, 1.0, 5, 2, 2.5, None, (12, 0.5))),
        (_attention(6, 2, 12, 12, 0.28), _dense(36, 0.6)),
        (_rglru(60, 1, 2), None),
        (_attention(4, 1, 20, 16, 0.2, 64, 40, (1e4, 20), (8.0, 1.5, 2.5, 64)), _dense(44, 3.0)))}

# Sizes at which the bfloat16 kernels take the tensor cores; windows of 48 and 130, 16 and 37 kept tokens.
SUMUVIK_C = {
    "architecture": "Sumuvik", "vocab": 640, "width": 256, "norm": {"eps": 1e-6}, "embedding": {"scale": 2.0},
    "layers": _layers(
        (_attention(8, 2, 64, 32, 0.11, 48, 16, (1e6, 32), (2.0, 1.0, 4.0, 100)), _dense(256, 1.0)),
        (_rglru(320, 5, 4), _moe(128, 1.0, 16, 4, 1.2, (4, 2), (128, 1.0))),
        (_attention(4, 4, 128, 128, 0.09, 130, 37, (1e6, 128)), _moe(64, 1.4, 9, 2, 1.0, (3, 2))),
        (_rglru(256, 2, 4), _dense(384, 2.0)))}

# Sizes that are multiples of nothing, a convolution of ONE tap, a window of ONE token beside three kept ones, diagonal blocks
# of eleven channels, five query heads over one key head, the best group of two only.
SUMUVIK_D = {
    "architecture": "Sumuvik", "vocab": 61, "width": 100, "norm": {"eps": 1e-6}, "embedding": {"scale": 1.0},
    "layers": _layers(
        (_rglru(33, 3, 1), _moe(7, 0.9, 6, 2, 0.5, (2, 1), (9, 0.7))),
        (_attention(5, 1, 40, 6, 0.2, 1, 3, (100.0, 6), (3.0, 1.0, 1.0, 9)), _dense(28, 1.1)),
        (_attention(2, 2, 5, 7, 0.5, 11, 2), _moe(33, 1.3, 7, 7, 1.0)))}

# Recurrent layers only (no pages at all); one block over all channels, as many blocks as channels; one expert.
SUMUVIK_E = {
    "architecture": "Sumuvik", "vocab": 130, "width": 48, "norm": {"eps": 1e-5}, "embedding": {"scale": 6.0},
    "layers": _layers(
        (_rglru(64, 1, 5), _dense(64, 0.5)),
        (_rglru(24, 24, 2), _moe(16, 1.0, 1, 1, 3.0)),
        (_rglru(128, 8, 4), _moe(24, 5.0, 12, 1, 1.0, (6, 5), (8, 0.3))))}

# Attention through windows only, over pages of 32: kept tokens that fill a page and a bit, more of them than the window is
# long, and none.
SUMUVIK_F = {
    "architecture": "Sumuvik", "vocab": 97, "width": 40, "norm": {"eps": 1e-6}, "embedding": {"scale": 1.3},
    "layers": _layers(
        (_attention(2, 2, 16, 16, 0.3, 33, 34, (50.0, 16)), _dense(40, 1.0)),
        (_attention(4, 2, 8, 12, 0.4, 9, 50, (1e3, 4), (2.0, 2.0, 6.0, 200)), _moe(12, 1.0, 4, 2, 1.5, (2, 2))),
        (_attention(4, 2, 8, 12, 0.4, 17, 0, (1e3, 4)), None))}

# name -> (config.json, seed, sigma of matrices, page size)
SUMUVIK = {"A": (SUMUVIK_A, 3, 0.14, 16), "B": (SUMUVIK_B, 4, 0.14, 8), "C": (SUMUVIK_C, 5, 0.06, 16),
           "D": (SUMUVIK_D, 6, 0.12, 16), "E": (SUMUVIK_E, 7, 0.15, 16), "F": (SUMUVIK_F, 8, 0.17, 32)}


def shape_weights(tensors, seed, dtype):
    """Random weights reworked in place so that the mechanisms show: decays that forget within some to hundreds of tokens and
    differ from channel to channel, biases of the size of what they are added to, router logits that lie apart with
    corrections that change the choice, embeddings of the stream's size."""
    g = torch.Generator().manual_seed(1000 + seed)
    for key in sorted(tensors):
        t = tensors[key].float()
        noise = torch.randn(t.shape, generator=g)
        if key == "embed":
            tensors[key] = noise.to(dtype)
        elif key.endswith(".lam"):
            tensors[key] = (1.5 * noise - 3.5).to(dtype)
        elif key.endswith(".correction"):
            tensors[key] = (0.4 * noise - 0.3).to(dtype)
        elif key.endswith(".router"):
            tensors[key] = (3.0 * t).to(dtype)
        elif key.endswith((".q.b", ".k.b", ".v.b", ".x.b", ".y.b", ".conv.b", ".ra.b", ".ri.b")):
            tensors[key] = (0.5 * noise).to(dtype)
        elif key.endswith((".ra", ".ri")):
            tensors[key] = (noise / t.shape[-1] ** 0.5).to(dtype)
        elif key.endswith(("mix.g", ".gate", ".up")):
            tensors[key] = (1.5 * t).to(dtype)
    return tensors


def write_sumuvik_model(name: str, folder: str, dtype=torch.bfloat16) -> str:
    """Write a small Sumuvik folder with random weights (see ``shape_weights``); returns its path."""
    from llm_rs_b200.config import SumuvikConfig, resolve_architecture
    from llm_rs_b200.parts import DecoderModel
    from llm_rs_b200.weights.random_init import random_tensors
    from llm_rs_b200.weights.safetensors_io import save_file
    raw, seed, sigma, _ = SUMUVIK[name]
    cfg = SumuvikConfig.from_dict(raw)
    path = os.path.join(folder, f"sumuvik_{name}")
    model = DecoderModel(resolve_architecture(raw).build_spec(cfg))
    tensors = shape_weights(random_tensors(model.weight_specs(), seed, sigma, 0.3, dtype, "cpu"), seed, dtype)
    os.makedirs(path, exist_ok=True)
    with open(os.path.join(path, "config.json"), "w") as f:
        json.dump(cfg.to_dict(), f, indent=2)
    save_file(tensors, os.path.join(path, "model.safetensors"))
    return path
