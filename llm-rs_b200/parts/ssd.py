"""State-space duality (Mamba-2): a recurrent mixer whose keys and queries are shared by groups of heads."""
from __future__ import annotations

import torch

from .. import ops
from .base import Mixer, Runtime
from .linear import Linear, joined_rows
from .registry import register
from .spec import StateNeed, WeightSpec


@register("mixer", "mamba2")
class Mamba2(Mixer):
    """``n_heads`` heads of ``vdim`` channels (inner = n_heads * vdim) over states of ``state`` rows; ``groups`` groups of
    heads share their B and C (head h reads group h // (n_heads / groups)). One projection of the input is laid out
    z [inner] | x [inner] | B [groups * state] | C [groups * state] | dt [n_heads]; x, B and C pass a short causal convolution
    over time per channel (``conv`` taps, the last one the current token's, with a bias, zeros before the start) and SiLU;
    ``dt = softplus(dt + dt_bias)``, not clamped. Per head

        S_t = exp(-exp(A_log) dt) S_(t-1) + dt B_t x_t^T,     y_t = S_t^T C_t + D x_t

    and the concatenated y is multiplied by silu(z), THEN divided by its root mean square in ``norm_parts`` equal parts
    (``norm_eps``), multiplied by a weight of size inner and projected.

    Step size, decay, state, gate and norm are float32. Per-request state: S and the last ``conv`` - 1 rows that entered the
    convolution; no pages. ``heads(...)`` gives the normed rows before the output projection, optionally scaled and
    written into a view, for a mixer that runs this one beside another.

    ``names`` maps the roles in, conv, conv_bias, dt_bias, A_log, D, norm, o to tensor names."""
    ROLES = ("in", "conv", "conv_bias", "dt_bias", "A_log", "D", "norm", "o")
    STATE, CONV_STATE = "ssd.state", "ssd.conv"
    fuses_residual = True

    def __init__(self, hidden_size: int, n_heads: int, vdim: int, state: int, groups: int, conv: int, norm_parts: int = 1,
                 norm_eps: float = 1e-6, names=None, prefix: str = ""):
        if n_heads % groups:
            raise ValueError(f"{n_heads} heads are no multiple of {groups} groups")
        if (n_heads * vdim) % norm_parts:
            raise ValueError(f"{n_heads * vdim} channels do not fall into {norm_parts} equal parts")
        if state > 256:
            raise ValueError(f"states of {state} rows: the recurrence kernel takes at most 256")
        if conv < 1:
            raise ValueError(f"a convolution of {conv} taps")
        self.hidden_size, self.n_heads, self.vdim, self.state, self.groups = hidden_size, n_heads, vdim, state, groups
        self.conv, self.norm_parts, self.norm_eps, self.prefix = int(conv), int(norm_parts), float(norm_eps), prefix
        self.names = {role: role for role in self.ROLES}
        self.names["conv_bias"] = "conv.b"
        self.names.update(names or {})
        if set(self.names) != set(self.ROLES):
            raise ValueError(f"names may rename {self.ROLES}, got {sorted(set(self.names) - set(self.ROLES))}")
        self.inner = n_heads * vdim
        self.channels = self.inner + 2 * groups * state      # what passes the convolution

    def _name(self, role: str) -> str:
        return self.prefix + self.names[role]

    def weight_specs(self):
        H, nm, C, nh = self.hidden_size, self._name, self.channels, self.n_heads
        return [WeightSpec(nm("in"), (self.inner + C + nh, H)), WeightSpec(nm("conv"), (C, self.conv), role="conv"),
                WeightSpec(nm("conv_bias"), (C,), role="bias"), WeightSpec(nm("dt_bias"), (nh,), role="bias"),
                WeightSpec(nm("A_log"), (nh,), role="bias"), WeightSpec(nm("D"), (nh,), role="norm"),
                WeightSpec(nm("norm"), (self.inner,), role="norm"), WeightSpec(nm("o"), (H, self.inner))]

    def bind(self, tensors, runtime: Runtime):
        nm = self._name
        self.act_dtype = runtime.act_dtype
        w, starts = joined_rows(list(torch.split(tensors[nm("in")], [self.inner, self.channels, self.n_heads], dim=0)))
        self.at_xbc, self.at_dt = starts[1:]
        self.in_proj = Linear(w, None, runtime.act_dtype)
        self.o_proj = Linear(tensors[nm("o")], None, runtime.act_dtype)
        f32 = lambda role: tensors[nm(role)].to(torch.float32).contiguous()
        self.taps, self.conv_bias, self.dt_bias = f32("conv"), f32("conv_bias"), f32("dt_bias")
        self.a_log, self.skip, self.norm_w = f32("A_log"), f32("D"), f32("norm")

    def chain(self):
        return [self.in_proj, self.o_proj]

    def state_need(self):
        return StateNeed({self.STATE: (self.n_heads, self.state, self.vdim),
                          self.CONV_STATE: (self.conv - 1, self.channels)})

    def takes_prenormed(self, n_tokens: int) -> bool:
        return self.in_proj.takes_prenormed(n_tokens)

    def emits_prenormed(self, n_tokens: int) -> bool:
        return self.o_proj.emits_prenormed(n_tokens)

    def heads(self, x, ctx, cache, out=None, out_scale: float = 1.0):
        proj = self.in_proj.forward(x)
        return ops.ssd(proj[:, self.at_xbc: self.at_xbc + self.channels], proj[:, : self.inner],
                       proj[:, self.at_dt: self.at_dt + self.n_heads], self.taps, self.conv_bias, self.dt_bias, self.a_log,
                       self.skip, self.norm_w, cache.state[self.STATE], cache.state[self.CONV_STATE], ctx, self.n_heads,
                       self.vdim, self.groups, self.state, self.norm_parts, self.norm_eps, out=out, out_scale=out_scale)

    def forward(self, x, ctx, cache, out_dtype=None, residual=None, next_norm=None):
        return self.o_proj.forward_branch(self.heads(x, ctx, cache), residual, next_norm, out_dtype)
