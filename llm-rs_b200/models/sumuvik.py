"""The Sumuvik design as a ``ModelSpec``.

Every layer is a ``parallel`` block (mixer and feed-forward read the same stream, each through a norm of its own) around one
of two mixers: ``scored_attention`` (grouped heads with projection biases, neighbouring channels rotated by rescaled
frequencies, a sliding window beside the sequence's first tokens, one added to the softmax's denominator, a gate per head) or
``rglru`` (a gated linear recurrence per channel behind a short convolution, beside a GELU branch). The feed-forward is the
clamped gated unit, dense or as routed experts beside a shared one, or absent. The embedding is scaled, the head is its own.

The constants the design fixes are given to the parts here: the unit's 1.702 and the 1 added to up, the recurrence's 8, the
sink's score of 0.
"""
from __future__ import annotations

from ..config import ArchitectureEntry, register_architecture
from ..config.sumuvik import DenseMLP, MoEMLP, RecurrentMixer, SumuvikConfig, WindowMixer
from ..parts import LayerSpec, ModelSpec, PartSpec, RunStep

EMBEDDING, FINAL_NORM, HEAD = "embed", "final.norm", "head"
MIXER_SCOPE, FEED_FORWARD_SCOPE = "mix.", "mlp."
UNIT = {"alpha": 1.702, "up_shift": 1.0}
DECAY_SCALE = 8.0
SINK_SCORE = 0.0
RECURRENT_NAMES = {"r": "ra", "r_bias": "ra.b", "i": "ri", "i_bias": "ri.b"}
# No key of the configuration bounds a sequence; a layer that keeps every key bounds it by the pool.
MAX_POSITIONS = 1 << 30


def _mixer(m, D: int) -> PartSpec:
    if isinstance(m, RecurrentMixer):
        return PartSpec("rglru", {"hidden_size": D, "width": m.width, "blocks": m.blocks, "conv": m.conv,
                                  "decay_scale": DECAY_SCALE, "names": RECURRENT_NAMES})
    assert isinstance(m, WindowMixer)
    return PartSpec("scored_attention", {
        "hidden_size": D, "n_heads": m.heads, "n_kv_heads": m.kv_heads, "dim": m.dim, "vdim": m.vdim, "scale": m.scale,
        "mask": "window" if m.window else "causal", "mask_size": m.window, "keep_first": m.keep_first, "qk_norm": "none",
        "rot_dims": m.rot_dims, "rot_base": m.rot_base, "rot_pairing": "neighbours",
        "rot_scaling": None if m.scaling is None else m.scaling.to_dict(), "sink_score": SINK_SCORE, "qkv_bias": True,
        "gated": True})


def _feed_forward(f, D: int):
    if f is None:
        return None
    if isinstance(f, DenseMLP):
        return PartSpec("swiglu", {"hidden_size": D, "intermediate_size": f.unit.ff, "limit": f.unit.limit, "suffix": "",
                                   **UNIT})
    assert isinstance(f, MoEMLP)
    shared = {} if f.shared is None else {"shared_size": f.shared.ff, "shared_limit": f.shared.limit}
    return PartSpec("moe", {"hidden_size": D, "expert_size": f.expert.ff, "limit": f.expert.limit, "n_experts": f.experts,
                            "top": f.top, "router": "sigmoid_groups", "groups": (f.groups, f.keep), "route_scale": f.scale,
                            **UNIT, **shared})


def build_spec(cfg: SumuvikConfig) -> ModelSpec:
    D = cfg.width
    norm = lambda name: PartSpec("rmsnorm", {"dim": D, "eps": cfg.norm_eps, "name": name})
    layers = []
    for i, layer in enumerate(cfg.layers):
        ffn = _feed_forward(layer.mlp, D)
        layers.append(LayerSpec(
            prefix=f"l{i}.", block=PartSpec("parallel"), mixer=_mixer(layer.mixer, D), feed_forward=ffn,
            mixer_norm=norm("norm1"), feed_forward_norm=norm("norm2"),
            mixer_scope=MIXER_SCOPE, feed_forward_scope=FEED_FORWARD_SCOPE))
    return ModelSpec(
        hidden_size=D, vocab_size=cfg.vocab, layers=tuple(layers), run_order=tuple(RunStep(i) for i in range(len(layers))),
        embedding=PartSpec("pair_embedding", {"vocab_size": cfg.vocab, "hidden_size": D, "scale": cfg.embedding_scale,
                                              "name": EMBEDDING}),
        final_norm=norm(FINAL_NORM),
        lm_head=PartSpec("linear_head", {"vocab_size": cfg.vocab, "hidden_size": D, "name": HEAD}),
        max_positions=MAX_POSITIONS, eos_token_ids=())


register_architecture(ArchitectureEntry(
    name=SumuvikConfig.architecture, model_type=SumuvikConfig.model_type,
    config_cls=SumuvikConfig, build_spec=build_spec), replace=True)
