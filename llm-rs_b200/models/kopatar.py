"""The Kopatar design as a ``ModelSpec``.

Every layer is a ``prenorm`` block around one of three mixers: ``channel_delta`` (a gated delta rule with a decay per key
channel behind short convolutions), ``retention`` (a fixed decay per head over rotated queries and keys) or ``parallel``
(softmax attention with normed heads, a sliding window and a gate on every channel, beside a Mamba-2 recurrence; a
weighted sum of the two). The feed-forward is dense with the xIELU activation, or absent. The head is the embedding table.
A stretch of layers may run several times with the same weights: every pass has run-order entries (so pages and state) of
its own, and ahead of it the stream takes the embedding output (not in the first pass) and a vector of that pass
(``embedding_add``).

The constants the design fixes are given to the parts here: the 1e-6 under the root of the delta rule's unit vectors,
its query scale and retention's key scale dim^-1/2, which norms and gates each mixer has.
"""
from __future__ import annotations

from ..config import ArchitectureEntry, register_architecture
from ..config.kopatar import ChannelDeltaMixer, KopatarConfig, RetentionMixer
from ..parts import LayerSpec, ModelSpec, PartSpec, RunStep

EMBEDDING, FINAL_NORM, LOOP_STEP = "embed", "final.norm", "loop.step"
MIXER_SCOPE, FEED_FORWARD_SCOPE = "mix.", "mlp."
UNIT_KEY_EPS = 1e-6
# No key of the configuration bounds a sequence; a layer that keeps every key bounds it by the pool.
MAX_POSITIONS = 1 << 30


def run_order(cfg: KopatarConfig):
    """The layers in the order they run; the first entry of every pass over the looped stretch re-enters."""
    n = len(cfg.layers)
    if cfg.loop is None:
        return tuple(RunStep(i) for i in range(n))
    a, b = cfg.loop.start, cfg.loop.stop
    order = [RunStep(i) for i in range(a)]
    for t in range(cfg.loop.times):
        order += [RunStep(i, reenter=(i == a), pass_index=t) for i in range(a, b)]
    return tuple(order + [RunStep(i) for i in range(b, n)])


def _mixer(m, D: int, eps: float) -> PartSpec:
    if isinstance(m, ChannelDeltaMixer):
        return PartSpec("channel_delta", {
            "hidden_size": D, "n_heads": m.heads, "n_kv_heads": m.kv_heads, "dim": m.dim, "vdim": m.vdim, "conv": m.conv,
            "decay_rank": m.decay_rank, "gate_rank": m.gate_rank, "norm_eps": eps, "key_eps": UNIT_KEY_EPS,
            "q_scale": m.dim ** -0.5})
    if isinstance(m, RetentionMixer):
        return PartSpec("retention", {
            "hidden_size": D, "n_heads": m.heads, "dim": m.dim, "vdim": m.vdim, "decay": m.decay, "rot_dims": m.rot_dims,
            "rot_base": m.rot_base, "k_scale": m.dim ** -0.5, "norm_eps": eps})
    l, r = m.left, m.right
    left = PartSpec("scored_attention", {
        "hidden_size": D, "n_heads": l.heads, "n_kv_heads": l.kv_heads, "dim": l.dim, "vdim": l.vdim, "scale": l.scale,
        "mask": "window" if l.window else "causal", "mask_size": l.window, "qk_norm": "head", "norm_eps": eps,
        "gated": True, "gate_per": "channel"})
    right = PartSpec("mamba2", {
        "hidden_size": D, "n_heads": r.heads, "vdim": r.vdim, "state": r.state, "groups": r.groups, "conv": r.conv,
        "norm_parts": r.norm_groups, "norm_eps": eps})
    return PartSpec("parallel", {"left": left, "right": right, "left_scale": m.left_scale, "right_scale": m.right_scale})


def build_spec(cfg: KopatarConfig) -> ModelSpec:
    D, eps = cfg.width, cfg.norm_eps
    norm = lambda name: PartSpec("rmsnorm", {"dim": D, "eps": eps, "name": name})
    layers = []
    for i, layer in enumerate(cfg.layers):
        ffn = None
        if layer.mlp is not None:
            ffn = PartSpec("dense", {"hidden_size": D, "intermediate_size": layer.mlp.ff, "activation": "xielu"})
        layers.append(LayerSpec(
            prefix=f"l{i}.", block=PartSpec("prenorm"), mixer=_mixer(layer.mixer, D, eps), feed_forward=ffn,
            mixer_norm=norm("norm1"), feed_forward_norm=norm("norm2") if ffn is not None else None,
            mixer_scope=MIXER_SCOPE, feed_forward_scope=FEED_FORWARD_SCOPE))
    return ModelSpec(
        hidden_size=D, vocab_size=cfg.vocab, layers=tuple(layers), run_order=run_order(cfg),
        embedding=PartSpec("token_embedding", {"vocab_size": cfg.vocab, "hidden_size": D, "name": EMBEDDING}),
        final_norm=norm(FINAL_NORM),
        lm_head=PartSpec("linear_head", {"vocab_size": cfg.vocab, "hidden_size": D, "name": "head", "tied_to": EMBEDDING}),
        reentry=None if cfg.loop is None else PartSpec("embedding_add", {"hidden_size": D, "times": cfg.loop.times,
                                                                         "name": LOOP_STEP}),
        max_positions=MAX_POSITIONS, eos_token_ids=())


register_architecture(ArchitectureEntry(
    name=KopatarConfig.architecture, model_type=KopatarConfig.model_type,
    config_cls=KopatarConfig, build_spec=build_spec), replace=True)
