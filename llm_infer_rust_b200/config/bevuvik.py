"""Typed configuration of Bevuvik, read from its own config.json keys.

    architecture    "Bevuvik"
    vocab, width    sizes of the token table (the output head is a matrix of its own) and of the residual stream
    norm.eps        eps of the model's norms (inside the root)
    residual_mult   what every layer's sum is multiplied by before it joins the stream
    loop            start, stop, times: the layers start .. stop-1 run ``times`` times in a row (absent or null: every
                    layer runs once)
    layers[i]       type, mixer (sizes and constants, below), mlp: null or {"kind": "dense", "ff": F, "limit": L}

    attention       heads, kv_heads, dim (of one of a head's two query / key vectors), vdim, scale, diff,
                    rot {base, dims, scaling {factor, original, fast, slow} (absent: none)} (absent: no rotation),
                    mask {size} (absent: every earlier key)
    parallel        left: heads, kv_heads, dim, vdim, scale, softcap (absent: none), rot {base, dims};
                    right: heads, kv_heads, dim, vdim, conv (taps)

Nothing here is a default for a size: a key that the design needs and the file lacks is an error.
"""
from __future__ import annotations

from dataclasses import dataclass
from typing import Any, Dict, Optional, Tuple, Union

from .kefetar import MAX_POSITIONS, _int, _number
from .sigudra import QK_UNIT_EPS, _grouped, _object, _state_dim, _taps
from .spec import ConfigError, LayerSpec, ModelSpec, PartSpec, RunEntry

PASS_INPUT = "loop"         # the stream input that a pass through the looped layers begins with


@dataclass(frozen=True)
class YarnScaling:
    factor: float
    original: float
    fast: float
    slow: float


@dataclass(frozen=True)
class BevuvikRotation:
    base: float
    dims: int
    scaling: Optional[YarnScaling] = None


@dataclass(frozen=True)
class DifferentialMixer:
    heads: int
    kv_heads: int
    dim: int
    vdim: int
    scale: float
    diff: float
    rot: Optional[BevuvikRotation]
    window: Optional[int]


@dataclass(frozen=True)
class CappedDeltaPair:
    """Soft-capped attention (left) beside a gated delta rule (right)."""
    heads: int
    kv_heads: int
    dim: int
    vdim: int
    scale: float
    softcap: Optional[float]
    rot: Optional[BevuvikRotation]
    right_heads: int
    right_kv_heads: int
    right_dim: int
    right_vdim: int
    conv: int


@dataclass(frozen=True)
class BevuvikFF:
    ff: int
    limit: float


@dataclass(frozen=True)
class BevuvikLayer:
    mixer: Union[DifferentialMixer, CappedDeltaPair]
    ff: Optional[BevuvikFF]


@dataclass(frozen=True)
class Loop:
    start: int
    stop: int
    times: int


def _rotation(m: dict, dim: int, where: str) -> Optional[BevuvikRotation]:
    if m.get("rot") is None:
        return None
    rot, w = _object(m, "rot", where), where + "rot."
    dims = _int(rot, "dims", w, 2)
    if dims % 2 or dims > dim:
        raise ConfigError(f"invalid {w}dims: {dims} (even and at most dim = {dim})")
    scaling = None
    if rot.get("scaling") is not None:
        s, sw = _object(rot, "scaling", w), w + "scaling."
        scaling = YarnScaling(*(_number(s, key, sw) for key in ("factor", "original", "fast", "slow")))
        if _number(rot, "base", w) <= 1.0:
            raise ConfigError(f"{w}base must be above 1 where frequencies are scaled")
    return BevuvikRotation(_number(rot, "base", w), dims, scaling)


def _value_dim(m: dict, where: str) -> int:
    vdim = _int(m, "vdim", where)
    if vdim % 2 or vdim > 512:
        raise ConfigError(f"{where}vdim must be even and at most 512")
    return vdim


@dataclass(frozen=True)
class BevuvikConfig:
    vocab: int
    width: int
    eps: float
    residual_mult: float
    layers: Tuple[BevuvikLayer, ...]
    loop: Optional[Loop]

    architecture = "Bevuvik"
    model_type = None

    @staticmethod
    def _feed_forward(mlp: Any, where: str) -> Optional[BevuvikFF]:
        if mlp is None:
            return None
        if not isinstance(mlp, dict):
            raise ConfigError(f"{where}mlp must be null or an object")
        if mlp.get("kind") != "dense":
            raise ConfigError(f"unsupported {where}mlp.kind: {mlp.get('kind')!r} (dense is known)")
        return BevuvikFF(_int(mlp, "ff", where + "mlp."), _number(mlp, "limit", where + "mlp."))

    @staticmethod
    def _mixer(kind: Any, m: dict, where: str) -> Union[DifferentialMixer, CappedDeltaPair]:
        w = where + "mixer."
        if kind == "attention":
            heads, kv_heads = _grouped(m, w)
            dim = _int(m, "dim", w)
            if dim > 256:
                raise ConfigError(f"{w}dim must be at most 256 (a key is two vectors side by side)")
            window = _int(_object(m, "mask", w), "size", w + "mask.") if m.get("mask") is not None else None
            return DifferentialMixer(heads, kv_heads, dim, _value_dim(m, w), _number(m, "scale", w),
                                     _number(m, "diff", w, positive=False), _rotation(m, dim, w), window)
        if kind == "parallel":
            left, right = _object(m, "left", w), _object(m, "right", w)
            lw, rw = w + "left.", w + "right."
            heads, kv_heads = _grouped(left, lw)
            dim = _int(left, "dim", lw)
            if dim % 2 or dim > 512:
                raise ConfigError(f"{lw}dim must be even and at most 512")
            cap = _number(left, "softcap", lw) if left.get("softcap") is not None else None
            right_heads, right_kv = _grouped(right, rw)
            return CappedDeltaPair(heads, kv_heads, dim, _value_dim(left, lw), _number(left, "scale", lw), cap,
                                   _rotation(left, dim, lw), right_heads, right_kv, _state_dim(right, rw),
                                   _int(right, "vdim", rw), _taps(right, rw))
        raise ConfigError(f"unsupported {where}type: {kind!r} (attention and parallel are known)")

    @staticmethod
    def parse(raw: Any) -> "BevuvikConfig":
        if not isinstance(raw, dict):
            raise ConfigError("config must be an object")
        vocab, width = _int(raw, "vocab", ""), _int(raw, "width", "")
        eps = _number(_object(raw, "norm", ""), "eps", "norm.")
        entries = raw.get("layers")
        if not isinstance(entries, list) or not entries:
            raise ConfigError("layers must be a non-empty list")
        layers = []
        for i, entry in enumerate(entries):
            where = f"layers[{i}]."
            if not isinstance(entry, dict):
                raise ConfigError(f"layers[{i}] must be an object")
            layers.append(BevuvikLayer(BevuvikConfig._mixer(entry.get("type"), _object(entry, "mixer", where), where),
                                       BevuvikConfig._feed_forward(entry.get("mlp"), where)))
        loop = None
        if raw.get("loop") is not None:
            r = _object(raw, "loop", "")
            loop = Loop(_int(r, "start", "loop.", 0), _int(r, "stop", "loop."), _int(r, "times", "loop."))
            if not loop.start < loop.stop <= len(layers):
                raise ConfigError(f"loop.start and loop.stop must name layers of the {len(layers)}")
        return BevuvikConfig(vocab, width, eps, _number(raw, "residual_mult", "", positive=False), tuple(layers), loop)

    # ------------------------------------------------------------------ parts
    def run_list(self) -> Tuple[RunEntry, ...]:
        n = len(self.layers)
        if self.loop is None:
            return tuple(RunEntry(i) for i in range(n))
        at = self.loop
        one_pass = [RunEntry(i, input=PASS_INPUT if i == at.start else None) for i in range(at.start, at.stop)]
        return tuple([RunEntry(i) for i in range(at.start)] + one_pass * at.times
                     + [RunEntry(i) for i in range(at.stop, n)])

    def model_spec(self) -> ModelSpec:
        norm = PartSpec("owed_rms_norm", {"width": self.width, "eps": self.eps})
        encodings: Dict[str, PartSpec] = {}
        names: Dict[tuple, str] = {}

        def rotated(rot: Optional[BevuvikRotation], pairing: str) -> dict:
            if rot is None:
                return {}
            key = (rot, pairing)
            if key not in names:
                names[key] = f"rot{len(names)}"
                params = {"rotary_dim": rot.dims, "theta": rot.base, "pairing": pairing}
                if rot.scaling is not None:
                    params["yarn"] = {"factor": rot.scaling.factor, "original": rot.scaling.original,
                                      "fast": rot.scaling.fast, "slow": rot.scaling.slow}
                encodings[names[key]] = PartSpec("rotary_frequencies", params)
            return {"rot_dims": rot.dims, "position_encoding": names[key]}

        def mixer(m) -> PartSpec:
            if isinstance(m, DifferentialMixer):
                return PartSpec("differential_attention", {
                    "hidden_size": self.width, "num_heads": m.heads, "num_kv_heads": m.kv_heads, "head_dim": m.dim,
                    "v_head_dim": m.vdim, "diff": m.diff, "eps": self.eps, "bias": True, "out_bias": True,
                    "softmax_scale": m.scale, "window": m.window, **rotated(m.rot, "interleaved")})
            return PartSpec("parallel_mixers", {
                "hidden_size": self.width, "eps": self.eps,
                "left": PartSpec("grouped_attention", {
                    "hidden_size": self.width, "num_heads": m.heads, "num_kv_heads": m.kv_heads, "head_dim": m.dim,
                    "v_head_dim": m.vdim, "softmax_scale": m.scale, "softcap": m.softcap, **rotated(m.rot, "half_split")}),
                "right": PartSpec("channel_decay_attention", {
                    "hidden_size": self.width, "num_heads": m.right_heads, "num_kv_heads": m.right_kv_heads,
                    "head_dim": m.right_dim, "v_head_dim": m.right_vdim, "eps": self.eps, "conv_taps": m.conv,
                    "qkv_silu": True, "qk_unit_eps": QK_UNIT_EPS, "q_scale": m.right_dim ** -0.5, "decay": "softplus",
                    "decay_per": "head", "delta": True, "gate": "silu"})})

        layers = []
        for l in self.layers:
            parts = {"input_norm": norm, "mixer": mixer(l.mixer)}
            if l.ff is not None:
                parts["feed_forward"] = PartSpec("gated_act", {
                    "hidden_size": self.width, "intermediate_size": l.ff.ff, "activation": "clamped_swish",
                    "limit": l.ff.limit})
            layers.append(LayerSpec(PartSpec("parallel_sublayers", {"residual_mult": self.residual_mult}), parts))
        inputs = {PASS_INPUT: PartSpec("concat_input", {"width": self.width})} if self.loop is not None else {}
        spec = ModelSpec(
            architecture=self.architecture, vocab_size=self.vocab, hidden_size=self.width, max_positions=MAX_POSITIONS,
            embedding=PartSpec("token_embedding", {"vocab_size": self.vocab, "hidden_size": self.width,
                                                   "out_dtype": "float32"}),
            layers=tuple(layers), run_list=self.run_list(), final_norm=norm,
            lm_head=PartSpec("linear_head", {"vocab_size": self.vocab, "hidden_size": self.width, "tied": False}),
            position_encodings=encodings, stream_inputs=inputs)
        spec.validate()
        return spec
