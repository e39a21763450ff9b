"""A recurrent block around a real-gated linear recurrent unit (Griffin)."""
from __future__ import annotations

import torch

from ..kernels import ops
from .base import ParamDecl, Part, StateSpec, mixer_state, padded_rows
from .registry import register_part


class GatedLRU(Part):
    """Two branches of ``width`` channels: y = gelu_tanh(W_y h + y_bias) and u = conv(W_x h + x_bias) + conv_bias, a causal
    convolution of ``conv_taps`` taps per channel.  u in ``blocks`` equal parts u_b, with square matrices R_b and I_b:

        r = sigmoid(R_b u_b + r_bias),  i = sigmoid(I_b u_b + i_bias),  log a = -8 r softplus(lam)
        S <- a S + sqrt(1 - a^2) i u    (from zeros),        output W_o (S y)

    ``yx_proj``: the rows of W_y, then those of W_x; ``gates`` [2 * blocks, size, size]: every R_b, then every I_b.  S and
    the convolution's last inputs are the request's state, in float32."""
    category = "mixer"

    def __init__(self, spec, env):
        super().__init__(spec, env)
        self.hidden = int(spec["hidden_size"])
        self.width = int(spec["width"])
        self.blocks = int(spec["blocks"])
        self.taps = int(spec["conv_taps"])
        if self.width % self.blocks:
            raise ValueError("blocks must divide the width")
        if not 1 <= self.taps <= 8:
            raise ValueError(f"{self.taps} taps are refused: the convolution kernels take 1 to 8")
        self.size = self.width // self.blocks

    def param_decls(self):
        w = self.width
        decls = {"yx_proj": ParamDecl((2 * w, self.hidden)), "gates": ParamDecl((2 * self.blocks, self.size, self.size)),
                 "conv": ParamDecl((w, self.taps)), "o_proj": ParamDecl((self.hidden, w))}
        for name in ("y_bias", "x_bias", "conv_bias", "lam"):
            decls[name] = ParamDecl((w,), "vector")
        for name in ("r_bias", "i_bias"):
            decls[name] = ParamDecl((self.blocks, self.size), "vector")
        return decls

    def bind(self, name, tensor):
        super().bind(name, tensor)
        if name == "yx_proj":
            self.params[name] = padded_rows(tensor)
        elif name == "gates":
            # per block, its R rows and then its I rows: both products of a part are one
            n, s = self.blocks, self.size
            self.params[name] = tensor.view(2, n, s, s).transpose(0, 1).reshape(n, 2 * s, s).contiguous()
        elif name not in ("o_proj",):
            self.params[name] = tensor.to(torch.float32).contiguous()

    def cache_spec(self):
        return None

    def state_spec(self):
        return None

    def state_specs(self):
        specs = {"state": StateSpec((self.width,), torch.float32)}
        if self.taps > 1:
            specs["conv"] = StateSpec((self.taps - 1, self.width), torch.float32)
        return specs

    def in_proj_name(self) -> str:
        return "yx_proj"

    def forward(self, x, ctx, cache):
        return self.forward_packed(ops.linear(x, self.params["yx_proj"]), 0, ctx, cache)

    def forward_packed(self, packed, column, ctx, cache):
        """From the packed projection on: y in ``packed`` from ``column`` on, W_x h behind it."""
        p = self.params
        u = ops.causal_taps(packed, p["conv"], mixer_state(cache, "conv"), ctx, packed.dtype, channels=self.width,
                            column=column + self.width, bias=p["x_bias"], out_bias=p["conv_bias"])
        s = ops.gated_lru(u, packed, column, p["gates"], p["r_bias"], p["i_bias"], p["lam"], p["y_bias"],
                          mixer_state(cache, "state"), ctx)
        return ops.linear(s, p["o_proj"])


register_part("mixer", "gated_lru", GatedLRU)
