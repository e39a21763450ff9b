"""Typed configuration of Sigudra, read from its own config.json keys.

    architecture    "Sigudra"
    vocab, width    sizes of the token table (the output head is a matrix of its own) and of the residual stream
    norm.eps        eps of the model's norms (inside the root)
    embedding       bigram {buckets, mul_prev, mul_cur}: a second table by the token and the one before it (absent: none)
    layers[i]       type, mixer (sizes and constants, below), mlp: null, {"kind": "dense", "ff": F} or
                    {"kind": "moe", "expert": {"ff"}, "router": {"experts", "top"}}

    channel_delta   heads, kv_heads, dim, vdim, conv (taps)
    gla             heads, dim, vdim, tau
    parallel        left: heads, kv_heads, dim, vdim, scale, mask {size} (absent: every earlier key);
                    right: width, blocks, conv (taps)

The low-rank projections behind decays and gates have ranks that the file leaves to the tensors' shapes; ``decay_rank``
(channel_delta, gla) and ``gate_rank`` (channel_delta) name them where there is no checkpoint to ask (random weights).
Nothing here is a default for a size: a key that the design needs and the file lacks is an error.
"""
from __future__ import annotations

from dataclasses import dataclass
from typing import Any, Mapping, Optional, Tuple, Union

from .kefetar import MAX_POSITIONS, _int, _number
from .spec import ConfigError, LayerSpec, ModelSpec, PartSpec, RunEntry

QK_UNIT_EPS = 1e-6          # channel_delta: q and k as unit vectors, x / sqrt(sum x^2 + this)


@dataclass(frozen=True)
class SigudraFF:
    kind: str                  # "dense" | "moe"
    ff: int                    # of the layer, or of one expert
    experts: int = 0
    top: int = 0


@dataclass(frozen=True)
class ChannelDelta:
    heads: int
    kv_heads: int
    dim: int
    vdim: int
    conv: int
    decay_rank: int            # 0: not known without the checkpoint
    gate_rank: int


@dataclass(frozen=True)
class GatedLinear:
    heads: int
    dim: int
    vdim: int
    tau: float
    decay_rank: int


@dataclass(frozen=True)
class ParallelPair:
    heads: int
    kv_heads: int
    dim: int
    vdim: int
    scale: float
    window: Optional[int]
    right_width: int
    blocks: int
    conv: int


@dataclass(frozen=True)
class SigudraLayer:
    mixer: Union[ChannelDelta, GatedLinear, ParallelPair]
    ff: Optional[SigudraFF]


@dataclass(frozen=True)
class Bigram:
    buckets: int
    mul_prev: int
    mul_cur: int


def _object(raw: Any, key: str, where: str) -> dict:
    value = raw.get(key)
    if not isinstance(value, dict):
        raise ConfigError(f"{where}{key} must be an object")
    return value


def _rank(m: dict, key: str, where: str) -> int:
    return _int(m, key, where) if m.get(key) is not None else 0


def _taps(m: dict, where: str) -> int:
    taps = _int(m, "conv", where)
    if taps > 8:
        raise ConfigError(f"{where}conv: a convolution of more than 8 taps is refused")
    return taps


def _state_dim(m: dict, where: str) -> int:
    dim = _int(m, "dim", where)
    if dim > 512:
        raise ConfigError(f"{where}dim must be at most 512")
    return dim


def _grouped(m: dict, where: str) -> Tuple[int, int]:
    heads, kv_heads = _int(m, "heads", where), _int(m, "kv_heads", where)
    if heads % kv_heads:
        raise ConfigError(f"{where}heads must be a multiple of kv_heads")
    return heads, kv_heads


@dataclass(frozen=True)
class SigudraConfig:
    vocab: int
    width: int
    eps: float
    bigram: Optional[Bigram]
    layers: Tuple[SigudraLayer, ...]

    architecture = "Sigudra"
    model_type = None

    @staticmethod
    def _feed_forward(mlp: Any, where: str) -> Optional[SigudraFF]:
        if mlp is None:
            return None
        if not isinstance(mlp, dict):
            raise ConfigError(f"{where}mlp must be null or an object")
        w = where + "mlp."
        if mlp.get("kind") == "dense":
            return SigudraFF("dense", _int(mlp, "ff", w))
        if mlp.get("kind") == "moe":
            expert, router = _object(mlp, "expert", w), _object(mlp, "router", w)
            experts, top = _int(router, "experts", w + "router."), _int(router, "top", w + "router.")
            if top > experts:
                raise ConfigError(f"{w}router.top must be at most the {experts} experts")
            return SigudraFF("moe", _int(expert, "ff", w + "expert."), experts, top)
        raise ConfigError(f"unsupported {w}kind: {mlp.get('kind')!r} (dense and moe are known)")

    @staticmethod
    def _mixer(kind: Any, m: dict, where: str) -> Union[ChannelDelta, GatedLinear, ParallelPair]:
        w = where + "mixer."
        if kind == "channel_delta":
            heads, kv_heads = _grouped(m, w)
            return ChannelDelta(heads, kv_heads, _state_dim(m, w), _int(m, "vdim", w), _taps(m, w),
                                _rank(m, "decay_rank", w), _rank(m, "gate_rank", w))
        if kind == "gla":
            return GatedLinear(_int(m, "heads", w), _state_dim(m, w), _int(m, "vdim", w), _number(m, "tau", w),
                               _rank(m, "decay_rank", w))
        if kind == "parallel":
            left, right = _object(m, "left", w), _object(m, "right", w)
            lw, rw = w + "left.", w + "right."
            heads, kv_heads = _grouped(left, lw)
            dim, vdim = _int(left, "dim", lw), _int(left, "vdim", lw)
            if dim % 2 or vdim % 2 or dim > 512 or vdim > 512:
                raise ConfigError(f"{lw}dim and vdim must be even and at most 512")
            window = _int(_object(left, "mask", lw), "size", lw + "mask.") if left.get("mask") is not None else None
            width, blocks = _int(right, "width", rw), _int(right, "blocks", rw)
            if width % blocks:
                raise ConfigError(f"{rw}blocks must divide the width {width}")
            return ParallelPair(heads, kv_heads, dim, vdim, _number(left, "scale", lw), window, width, blocks,
                                _taps(right, rw))
        raise ConfigError(f"unsupported {where}type: {kind!r} (channel_delta, gla and parallel are known)")

    @staticmethod
    def parse(raw: Any) -> "SigudraConfig":
        if not isinstance(raw, dict):
            raise ConfigError("config must be an object")
        vocab, width = _int(raw, "vocab", ""), _int(raw, "width", "")
        eps = _number(_object(raw, "norm", ""), "eps", "norm.")
        bigram = None
        if raw.get("embedding") is not None:
            if _object(raw, "embedding", "").get("bigram") is not None:
                b, w = _object(raw["embedding"], "bigram", "embedding."), "embedding.bigram."
                bigram = Bigram(_int(b, "buckets", w), _int(b, "mul_prev", w, 0), _int(b, "mul_cur", w, 0))
                if max(b["mul_prev"], b["mul_cur"]) >= 1 << 31:
                    raise ConfigError(f"{w}mul_prev and mul_cur must be below 2^31")
        entries = raw.get("layers")
        if not isinstance(entries, list) or not entries:
            raise ConfigError("layers must be a non-empty list")
        layers = []
        for i, entry in enumerate(entries):
            where = f"layers[{i}]."
            if not isinstance(entry, dict):
                raise ConfigError(f"layers[{i}] must be an object")
            layers.append(SigudraLayer(SigudraConfig._mixer(entry.get("type"), _object(entry, "mixer", where), where),
                                       SigudraConfig._feed_forward(entry.get("mlp"), where)))
        return SigudraConfig(vocab, width, eps, bigram, tuple(layers))

    @staticmethod
    def with_ranks(raw: Any, shapes: Mapping[str, tuple]) -> Any:
        """``raw`` with the ranks of the low-rank projections, read from the first factors' shapes [rank, width]."""
        if not isinstance(raw, dict) or not isinstance(raw.get("layers"), list):
            return raw                                     # (parse says what is wrong)
        layers = []
        for i, entry in enumerate(raw["layers"]):
            if isinstance(entry, dict) and isinstance(entry.get("mixer"), dict) and \
                    entry.get("type") in ("channel_delta", "gla"):
                mixer = dict(entry["mixer"])
                for key, tensor in (("decay_rank", "a1"), ("gate_rank", "g1")):
                    shape = shapes.get(f"l{i}.mix.{tensor}")
                    if mixer.get(key) is None and shape is not None and len(shape) == 2:
                        mixer[key] = int(shape[0])
                entry = dict(entry, mixer=mixer)
            layers.append(entry)
        return dict(raw, layers=layers)

    def need_ranks(self) -> None:
        for i, l in enumerate(self.layers):
            m = l.mixer
            if isinstance(m, (ChannelDelta, GatedLinear)) and (not m.decay_rank or (isinstance(m, ChannelDelta) and not m.gate_rank)):
                raise ConfigError(f"layers[{i}].mixer: the rank of a low-rank projection is neither in the checkpoint "
                                  f"(l{i}.mix.a1, l{i}.mix.g1) nor in the configuration (decay_rank, gate_rank)")

    # ------------------------------------------------------------------ parts
    def _mixer_spec(self, m) -> PartSpec:
        if isinstance(m, ChannelDelta):
            return PartSpec("channel_decay_attention", {
                "hidden_size": self.width, "num_heads": m.heads, "num_kv_heads": m.kv_heads, "head_dim": m.dim,
                "v_head_dim": m.vdim, "eps": self.eps, "conv_taps": m.conv, "qkv_silu": True, "qk_unit_eps": QK_UNIT_EPS,
                "q_scale": m.dim ** -0.5, "decay": "softplus", "decay_rank": m.decay_rank, "delta": True,
                "gate": "low_rank_sigmoid", "gate_rank": m.gate_rank})
        if isinstance(m, GatedLinear):
            return PartSpec("channel_decay_attention", {
                "hidden_size": self.width, "num_heads": m.heads, "head_dim": m.dim, "v_head_dim": m.vdim, "eps": self.eps,
                "q_scale": m.dim ** -0.5, "decay": "logistic", "tau": m.tau, "decay_rank": m.decay_rank, "gate": "silu"})
        return PartSpec("parallel_mixers", {
            "hidden_size": self.width, "eps": self.eps,
            "left": PartSpec("grouped_attention", {
                "hidden_size": self.width, "num_heads": m.heads, "num_kv_heads": m.kv_heads, "head_dim": m.dim,
                "v_head_dim": m.vdim, "qk_norm_eps": self.eps, "qk_norm_scope": "projection", "softmax_scale": m.scale,
                "window": m.window, "gate": "head"}),
            "right": PartSpec("gated_lru", {"hidden_size": self.width, "width": m.right_width, "blocks": m.blocks,
                                            "conv_taps": m.conv})})

    def model_spec(self) -> ModelSpec:
        self.need_ranks()
        norm = PartSpec("output_layer_norm", {"width": self.width, "eps": self.eps})
        layers = []
        for l in self.layers:
            parts = {"mixer": self._mixer_spec(l.mixer), "mixer_norm": norm}
            if l.ff is not None:
                parts["ff_norm"] = norm
                if l.ff.kind == "dense":
                    parts["feed_forward"] = PartSpec("gated_act", {"hidden_size": self.width, "intermediate_size": l.ff.ff,
                                                                   "activation": "gelu_tanh"})
                else:
                    parts["feed_forward"] = PartSpec("routed_experts", {
                        "hidden_size": self.width, "intermediate_size": l.ff.ff, "experts": l.ff.experts,
                        "top": l.ff.top, "scores": "sigmoid", "renormalize": False, "activation": "swiglu",
                        "weights_on": "input"})
            layers.append(LayerSpec(PartSpec("post_norm_stream"), parts))
        embedding = {"vocab_size": self.vocab, "hidden_size": self.width, "out_dtype": "float32"}
        if self.bigram is not None:
            embedding.update(buckets=self.bigram.buckets, mul_prev=self.bigram.mul_prev, mul_cur=self.bigram.mul_cur)
        spec = ModelSpec(
            architecture=self.architecture, vocab_size=self.vocab, hidden_size=self.width, max_positions=MAX_POSITIONS,
            embedding=PartSpec("pair_embedding" if self.bigram is not None else "token_embedding", embedding),
            layers=tuple(layers), run_list=tuple(RunEntry(i) for i in range(len(layers))), final_norm=norm,
            lm_head=PartSpec("linear_head", {"vocab_size": self.vocab, "hidden_size": self.width, "tied": False}))
        spec.validate()
        return spec
