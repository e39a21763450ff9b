"""Linear attention whose state decays per key channel or per head, with or without the delta rule."""
from __future__ import annotations

from typing import Optional

import torch

from ..kernels import ops
from .base import ParamDecl, Part, StateSpec, mixer_state, padded_rows
from .registry import register_part


class ChannelDecayAttention(Part):
    """q, k (``num_kv_heads`` heads of ``head_dim``) and v (``num_heads`` of ``v_head_dim``) from one packed projection;
    head h uses q and k of head floor(h / (num_heads / num_kv_heads)).  Per head, S [head_dim, v_head_dim] in float32 in
    the request's slot (zeros at a sequence's start), g a decay per key channel acting on S's rows (or one a head, the same
    for every row):

        S <- diag(g) S + k v^T;                                               o = S^T q
        S <- diag(g) S;   u = beta (v - S^T k);   S <- S + k u^T;             o = S^T q       (``delta``)

    Each of these is a parameter of the part:
      * ``conv_taps`` T: q, k, v pass a causal convolution per channel (``conv`` [channels, T]; the last T - 1 inputs are
        state too) (None: no convolution);  ``qkv_silu``: and then silu;
      * ``qk_unit_eps``: q and k become unit vectors per head, x / sqrt(sum x^2 + eps) (None: not);  ``q_scale``;
      * ``decay`` "logistic": g = sigmoid(z)^(1 / ``tau``); "softplus": g = exp(-exp(a_log_h) softplus(z)); both with
        z = a2 (a1 h) + decay_bias [heads * head_dim], a1's ``decay_rank`` rows being part of the packed projection;
        ``decay_per`` "head" instead of "channel": one g a head, z = one packed row a head + decay_bias [heads], no a2;
      * ``delta``: beta = sigmoid of one packed row a head;
      * ``gate`` "silu": packed rows, one a column; "low_rank_sigmoid": sigmoid(g2 (g1 h)), g1's ``gate_rank`` rows packed.
    Each head's o is RMS-normed (``eps``, weight ``norm`` [v_head_dim] shared by the heads), times the gate, then the output
    projection.  Packed rows: q, k, v, gate (silu), a1 (or the heads' decay rows), g1 (low rank), beta.  No biases elsewhere.  Everything behind the
    packed projection and the convolution is float."""
    category = "mixer"

    def __init__(self, spec, env):
        super().__init__(spec, env)
        self.hidden = int(spec["hidden_size"])
        self.nh = int(spec["num_heads"])
        self.nkv = int(spec.get("num_kv_heads") or self.nh)
        self.d = int(spec["head_dim"])
        self.dv = int(spec["v_head_dim"])
        self.eps = float(spec["eps"])
        self.taps = int(spec.get("conv_taps") or 0)
        self.qkv_silu = bool(spec.get("qkv_silu", False))
        self.unit_eps = spec.get("qk_unit_eps")
        self.q_scale = float(spec.get("q_scale", 1.0))
        self.decay = str(spec["decay"])
        self.tau = float(spec.get("tau", 1.0))
        self.delta = bool(spec.get("delta", False))
        self.gate = str(spec["gate"])
        self.decay_per = str(spec.get("decay_per", "channel"))
        self.decay_rank = int(spec.get("decay_rank") or 0)
        self.gate_rank = int(spec.get("gate_rank") or 0)
        if self.nh % self.nkv:
            raise ValueError("num_heads must be a multiple of num_kv_heads")
        if not 1 <= self.d <= 512:
            raise ValueError(f"head_dim {self.d} is refused: the kernels keep up to 512 rows of a state")
        if not 0 <= self.taps <= 8:
            raise ValueError(f"{self.taps} taps are refused: the convolution kernels take up to 8")
        if self.decay not in ("logistic", "softplus") or self.gate not in ("silu", "low_rank_sigmoid"):
            raise ValueError(f"decay {self.decay!r} or gate {self.gate!r} is refused")
        if self.decay_per not in ("channel", "head"):
            raise ValueError(f"decay_per {self.decay_per!r} is refused: channel or head")
        self.per_head = self.decay_per == "head"
        if (self.decay_rank < 1 and not self.per_head) or (self.gate == "low_rank_sigmoid" and self.gate_rank < 1):
            raise ValueError("the low-rank projections need ranks")
        self.channels = 2 * self.nkv * self.d + self.nh * self.dv
        self.gate_column = self.channels
        self.a_column = self.channels + (self.nh * self.dv if self.gate == "silu" else 0)
        at = self.a_column + (self.nh if self.per_head else self.decay_rank)
        if self.gate == "low_rank_sigmoid":
            self.gate_column = at
            at += self.gate_rank
        self.beta_column = at if self.delta else None
        self.rows = at + (self.nh if self.delta else 0)
        self._form: Optional[ops.LinearStateForm] = None

    def param_decls(self):
        decls = {"in_proj": ParamDecl((self.rows, self.hidden)),
                 "decay_bias": ParamDecl((self.nh if self.per_head else self.nh * self.d,), "vector"),
                 "norm": ParamDecl((self.dv,), "vector"), "o_proj": ParamDecl((self.hidden, self.nh * self.dv))}
        if not self.per_head:
            decls["a2"] = ParamDecl((self.nh * self.d, self.decay_rank))
        if self.taps >= 1:
            decls["conv"] = ParamDecl((self.channels, self.taps))
        if self.decay == "softplus":
            decls["a_log"] = ParamDecl((self.nh,), "vector")
        if self.gate == "low_rank_sigmoid":
            decls["g2"] = ParamDecl((self.nh * self.dv, self.gate_rank))
        return decls

    def bind(self, name, tensor):
        super().bind(name, tensor)
        if name == "in_proj":
            self.params[name] = padded_rows(tensor)
        elif name in ("conv", "decay_bias", "norm", "a_log"):
            self.params[name] = tensor.to(torch.float32).contiguous()
        self._form = None

    def cache_spec(self):
        return None

    def state_spec(self):
        return None

    def state_specs(self):
        specs = {"state": StateSpec((self.nh, self.d, self.dv), torch.float32)}
        if self.taps > 1:
            specs["conv"] = StateSpec((self.taps - 1, self.channels), torch.float32)
        return specs

    def form(self) -> ops.LinearStateForm:
        if self._form is None:
            p = self.params
            self._form = ops.LinearStateForm(
                self.nh, self.nkv, self.d, self.dv, q_scale=self.q_scale, decay=self.decay, tau=self.tau,
                decay_bias=p["decay_bias"], a_log=p.get("a_log"), beta_column=self.beta_column, silu=self.qkv_silu,
                unit_eps=self.unit_eps, decay_column=self.a_column if self.per_head else None)
        return self._form

    def in_proj_name(self) -> str:
        return "in_proj"

    def forward(self, x, ctx, cache):
        return self.forward_packed(ops.linear(x, self.params["in_proj"]), 0, ctx, cache)

    def forward_packed(self, packed, column, ctx, cache):
        """From the packed projection on, its columns beginning at ``column`` of ``packed``."""
        p = self.params
        form, conv, conv_state = self.form(), p.get("conv"), mixer_state(cache, "conv")
        state, low_rank = mixer_state(cache, "state"), self.gate == "low_rank_sigmoid"
        # a decode step: everything between the two projections in one kernel
        gated = ops.state_decode(form, packed, conv, conv_state, state, ctx, p.get("a2"), self.a_column, p["norm"], self.eps,
                                 self.gate_column, p["g2"] if low_rank else None, column=column)
        if gated is None:
            z = None if self.per_head else ops.linear_columns(packed, column + self.a_column, p["a2"], out_dtype=torch.float32)
            o = ops.state_recurrence(form, packed, z, conv, conv_state, state, ctx, column=column)
            gate = ops.linear_columns(packed, column + self.gate_column, p["g2"]) if low_rank else packed
            gated = ops.head_unit_norm_gate(o, gate, 0 if low_rank else column + self.gate_column, self.nh, self.dv, self.eps,
                                            weight=p["norm"], gate="sigmoid" if low_rank else "silu")
        return ops.linear(gated, p["o_proj"])


register_part("mixer", "channel_decay_attention", ChannelDecayAttention)
