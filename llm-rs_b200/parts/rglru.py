"""A gated linear recurrence per channel beside a gated branch: Griffin's recurrent block with a real-gated linear recurrent
unit (De et al., "Griffin: Mixing Gated Linear Recurrences with Local Attention for Efficient Language Models")."""
from __future__ import annotations

import torch

from .. import ops
from .base import Mixer, Runtime
from .linear import Linear, joined_rows
from .registry import register
from .spec import StateNeed, WeightSpec


@register("mixer", "rglru")
class GatedLinearRecurrence(Mixer):
    """Two branches of ``width`` channels: ``y = gelu_tanh(W_y x + b_y)`` and ``u = conv(W_x x + b_x)``, a causal convolution
    over time per channel (``conv`` taps, the last one the current token's, with a bias, zeros before the start, no
    activation). ``u`` falls into ``blocks`` equal parts; in each, ``r = sigmoid(R_b u_b + r_b)`` and
    ``i = sigmoid(I_b u_b + i_b)`` with square matrices. Per channel, with ``log a = -decay_scale * r * softplus(lam)``,

        S_t = a_t S_(t-1) + sqrt(1 - a_t^2) i_t u_t       (S starts at zero)

    and the output is ``W_o (S * y)``.

    The gates' products accumulate in float32 and leave float32; gates, decay, state and the GELU are float32; u and the
    two projections have the activation type. Per-request state: S and the last ``conv`` - 1 inputs of the convolution; no
    pages. The two projections are one product, their biases are added where its halves are read. A step of single tokens
    takes one kernel for gates, recurrence and output (``ops.rglru_step``), any other step a product with the gates as
    its epilogue and a scan over the tokens.

    ``names`` maps the roles y, y_bias, x, x_bias, conv, conv_bias, r, r_bias, i, i_bias, lam, o to tensor names."""
    ROLES = ("y", "y_bias", "x", "x_bias", "conv", "conv_bias", "r", "r_bias", "i", "i_bias", "lam", "o")
    STATE, CONV_STATE = "rglru.state", "rglru.conv"
    fuses_residual = True

    def __init__(self, hidden_size: int, width: int, blocks: int, conv: int, decay_scale: float = 8.0, names=None,
                 prefix: str = ""):
        if width % blocks:
            raise ValueError(f"{width} channels do not fall into {blocks} equal blocks")
        if width // blocks > 1024:
            raise ValueError(f"blocks of {width // blocks} channels: the step kernel takes at most 1024")
        if conv < 1:
            raise ValueError(f"a convolution of {conv} taps")
        self.hidden_size, self.width, self.blocks, self.conv = hidden_size, width, blocks, int(conv)
        self.decay_scale, self.prefix = float(decay_scale), prefix
        self.names = {role: role for role in self.ROLES}
        self.names.update({"y_bias": "y.b", "x_bias": "x.b", "conv_bias": "conv.b", "r_bias": "r.b", "i_bias": "i.b"})
        self.names.update(names or {})
        if set(self.names) != set(self.ROLES):
            raise ValueError(f"names may rename {self.ROLES}, got {sorted(set(self.names) - set(self.ROLES))}")

    def _name(self, role: str) -> str:
        return self.prefix + self.names[role]

    def weight_specs(self):
        H, W, B, nm = self.hidden_size, self.width, self.blocks, self._name
        n = W // B
        return [WeightSpec(nm("y"), (W, H)), WeightSpec(nm("y_bias"), (W,), role="bias"),
                WeightSpec(nm("x"), (W, H)), WeightSpec(nm("x_bias"), (W,), role="bias"),
                WeightSpec(nm("conv"), (W, self.conv), role="conv"), WeightSpec(nm("conv_bias"), (W,), role="bias"),
                WeightSpec(nm("r"), (B, n, n)), WeightSpec(nm("r_bias"), (B, n), role="bias"),
                WeightSpec(nm("i"), (B, n, n)), WeightSpec(nm("i_bias"), (B, n), role="bias"),
                WeightSpec(nm("lam"), (W,), role="bias"), WeightSpec(nm("o"), (H, W))]

    def bind(self, tensors, runtime: Runtime):
        nm = self._name
        w, (_, self.at_x) = joined_rows([tensors[nm("y")], tensors[nm("x")]])
        self.in_proj = Linear(w, None, runtime.act_dtype)
        self.o_proj = Linear(tensors[nm("o")], None, runtime.act_dtype)
        f32 = lambda role: tensors[nm(role)].to(torch.float32).reshape(-1).contiguous()
        self.y_bias, self.x_bias, self.conv_bias = f32("y_bias"), f32("x_bias"), f32("conv_bias")
        self.r_bias, self.i_bias = f32("r_bias"), f32("i_bias")
        self.taps = tensors[nm("conv")].to(torch.float32).t().contiguous()        # [taps, width]
        r, i = tensors[nm("r")], tensors[nm("i")]
        same = torch.bfloat16 if r.dtype == i.dtype == runtime.act_dtype == torch.bfloat16 else torch.float32
        self.w_r, self.w_i = r.to(same).contiguous(), i.to(same).contiguous()
        self.w_step = ops.rglru_step_weights(self.w_r, self.w_i)
        # log a = rate * r; made once, in double.
        lam = tensors[nm("lam")].double()
        self.rate = (-self.decay_scale * torch.nn.functional.softplus(lam)).to(torch.float32).contiguous()

    def chain(self):
        return [self.in_proj, self.o_proj]

    def state_need(self):
        return StateNeed({self.STATE: (self.width,), self.CONV_STATE: (self.conv - 1, self.width)})

    def takes_prenormed(self, n_tokens: int) -> bool:
        return self.in_proj.takes_prenormed(n_tokens)

    def emits_prenormed(self, n_tokens: int) -> bool:
        return self.o_proj.emits_prenormed(n_tokens)

    def heads(self, x, ctx, cache):
        """S * y before the output projection, [tokens, width]."""
        W = self.width
        proj = self.in_proj.forward(x)
        y, xs = proj[:, :W], proj[:, self.at_x: self.at_x + W]
        single = ctx.n_tokens == ctx.n_requests
        u = ops.short_conv(xs, self.taps, self.conv_bias, self.x_bias, cache.state[self.CONV_STATE], ctx, single)
        gates = (self.r_bias, self.i_bias, self.rate)
        if single:
            return ops.rglru_step(u, self.w_step, *gates, y, self.y_bias, cache.state[self.STATE], ctx)
        return ops.rglru_scan(ops.rglru_gates(u, self.w_r, self.w_i, *gates), y, self.y_bias, cache.state[self.STATE], ctx)

    def forward(self, x, ctx, cache, out_dtype=None, residual=None, next_norm=None):
        return self.o_proj.forward_branch(self.heads(x, ctx, cache), residual, next_norm, out_dtype)
