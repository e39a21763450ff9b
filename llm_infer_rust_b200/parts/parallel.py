"""Two mixers side by side on one input."""
from __future__ import annotations

import torch

from ..kernels import ops
from .base import ParamDecl, Part, padded_rows, sub_cache
from .registry import build_part, register_part


class ParallelMixers(Part):
    """(R(left(h); left_out) + R(right(h); right_out)) / 2, R the RMS norm over the model's width (``eps``) with a branch's
    own weights.  ``left`` and ``right`` are part specifications; at most one of them keeps keys and values in pages, both
    may keep state.  Branches that can start from a packed projection (``in_proj_name`` and ``forward_packed``) share ONE
    product for their projections; from there on, in a step of few tokens, they run side
    by side (``ops.side_by_side``).  The mean is handed on unformed (``ops.NormedPair``): the norm that adds the mixer's
    output into the stream takes it in its own kernel."""
    category = "mixer"

    def __init__(self, spec, env):
        super().__init__(spec, env)
        self.hidden = int(spec["hidden_size"])
        self.eps = float(spec["eps"])
        self.left = build_part("mixer", spec["left"], env)
        self.right = build_part("mixer", spec["right"], env)
        paged = [m for m in (self.left, self.right) if m.cache_spec() is not None]
        if len(paged) > 1:
            raise ValueError("two mixers side by side may keep one set of pages between them")
        if any(m.state_spec() is not None for m in (self.left, self.right)):
            raise ValueError("mixers side by side name their states (state_specs)")
        self.paged = paged[0] if paged else None
        self.joint = None              # (packed weights of both branches, first row of the right one)

    def children(self):
        return {"left": self.left, "right": self.right}

    def param_decls(self):
        return {"left_out": ParamDecl((self.hidden,), "vector"), "right_out": ParamDecl((self.hidden,), "vector")}

    def bind(self, name, tensor):
        super().bind(name, tensor)
        self.params[name] = tensor.to(torch.float32).contiguous()

    def cache_spec(self):
        return self.paged.cache_spec() if self.paged is not None else None

    def state_spec(self):
        return None

    def state_specs(self):
        specs = {}
        for name, mixer in self.children().items():
            own = getattr(mixer, "state_specs", None)
            for key, value in (own() if own is not None else {}).items():
                specs[f"{name}.{key}"] = value
        return specs

    def _joint_projection(self):
        if self.joint is None:
            names = [m.in_proj_name() for m in (self.left, self.right)]
            first = padded_rows(self.left.params[names[0]])
            weight = padded_rows(torch.cat([first, self.right.params[names[1]]]))
            self.joint = (weight, first.shape[0])
            # the branches' own matrices become views: nothing is kept twice
            for mixer, name, at in ((self.left, names[0], 0), (self.right, names[1], first.shape[0])):
                mixer.params[name] = weight[at:at + mixer.params[name].shape[0]]
        return self.joint

    def forward(self, x, ctx, cache):
        left, right = (sub_cache(cache, name) for name in ("left", "right"))
        if all(hasattr(m, "forward_packed") for m in (self.left, self.right)):
            weight, column = self._joint_projection()
            packed = ops.linear(x, weight)
            a, b = ops.side_by_side(x.shape[0], x.device, lambda: self.left.forward_packed(packed, 0, ctx, left),
                                    lambda: self.right.forward_packed(packed, column, ctx, right))
        else:
            a, b = ops.side_by_side(x.shape[0], x.device, lambda: self.left.forward(x, ctx, left),
                                    lambda: self.right.forward(x, ctx, right))
        return ops.NormedPair(a, b, self.params["left_out"], self.params["right_out"], self.eps)


register_part("mixer", "parallel_mixers", ParallelMixers)
