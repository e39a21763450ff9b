"""Sigudra as a registry entry: configuration, parts and checkpoint names.

Checkpoint names: ``embed``, ``bigram`` [buckets + 1, width], ``final.norm``, ``head``; per layer i ``l<i>.norm1`` and, with
a feed-forward, ``l<i>.norm2``; the mixer's tensors ``l<i>.mix.*`` and the feed-forward's ``l<i>.mlp.*``:

    channel_delta     q, k, v with q.conv, k.conv, v.conv; b, A_log; a1, a2, dt_bias (decay); g1, g2 (gate); norm; o
    gla               q, k, v, g; a1, a2, a2.b (decay); norm; o
    parallel          left.{q,k,v,g,o}, left.q.norm, left.k.norm, left.out; right.{y,x,o}, right.y.b, right.x.b, right.conv,
                      right.conv.b, right.ra, right.ra.b, right.ri, right.ri.b, right.lam, right.out
    dense             gate, up, down
    moe               router; e<j>.gate, e<j>.up, e<j>.down for every expert j

Linear weights are [out, in].  The rows of the projections that read a mixer's input are packed into one matrix, in the
order that the parts name.
"""
from __future__ import annotations

from typing import List

from ..config.registry import Architecture, register_architecture
from ..config.sigudra import ChannelDelta, GatedLinear, SigudraConfig
from ..weights.plan import SourceTensor, WeightBinding


def _channel_delta(m: ChannelDelta, w: int, src: str, dst: str) -> List[WeightBinding]:
    qk, v, keys = m.kv_heads * m.dim, m.heads * m.vdim, m.heads * m.dim
    return [
        WeightBinding(dst + "in_proj", (
            SourceTensor(src + "q", (qk, w)), SourceTensor(src + "k", (qk, w)), SourceTensor(src + "v", (v, w)),
            SourceTensor(src + "a1", (m.decay_rank, w)), SourceTensor(src + "g1", (m.gate_rank, w)),
            SourceTensor(src + "b", (m.heads, w)))),
        WeightBinding(dst + "conv", (SourceTensor(src + "q.conv", (qk, m.conv)), SourceTensor(src + "k.conv", (qk, m.conv)),
                                     SourceTensor(src + "v.conv", (v, m.conv)))),
        WeightBinding(dst + "a2", (SourceTensor(src + "a2", (keys, m.decay_rank)),)),
        WeightBinding(dst + "decay_bias", (SourceTensor(src + "dt_bias", (keys,)),)),
        WeightBinding(dst + "a_log", (SourceTensor(src + "A_log", (m.heads,)),)),
        WeightBinding(dst + "g2", (SourceTensor(src + "g2", (v, m.gate_rank)),)),
        WeightBinding(dst + "norm", (SourceTensor(src + "norm", (m.vdim,), "norm"),)),
        WeightBinding(dst + "o_proj", (SourceTensor(src + "o", (w, v)),))]


def _gated_linear(m: GatedLinear, w: int, src: str, dst: str) -> List[WeightBinding]:
    keys, v = m.heads * m.dim, m.heads * m.vdim
    return [
        WeightBinding(dst + "in_proj", (
            SourceTensor(src + "q", (keys, w)), SourceTensor(src + "k", (keys, w)), SourceTensor(src + "v", (v, w)),
            SourceTensor(src + "g", (v, w)), SourceTensor(src + "a1", (m.decay_rank, w)))),
        WeightBinding(dst + "a2", (SourceTensor(src + "a2", (keys, m.decay_rank)),)),
        WeightBinding(dst + "decay_bias", (SourceTensor(src + "a2.b", (keys,)),)),
        WeightBinding(dst + "norm", (SourceTensor(src + "norm", (m.vdim,), "norm"),)),
        WeightBinding(dst + "o_proj", (SourceTensor(src + "o", (w, v)),))]


def _parallel(m, w: int, src: str, dst: str) -> List[WeightBinding]:
    q, k, v, r = m.heads * m.dim, m.kv_heads * m.dim, m.kv_heads * m.vdim, m.right_width
    size = r // m.blocks
    ls, ld, rs, rd = src + "left.", dst + "left.", src + "right.", dst + "right."
    return [
        WeightBinding(ld + "qkv_proj", (
            SourceTensor(ls + "q", (q, w)), SourceTensor(ls + "k", (k, w)), SourceTensor(ls + "v", (v, w)),
            SourceTensor(ls + "g", (m.heads, w)))),
        WeightBinding(ld + "q_norm", (SourceTensor(ls + "q.norm", (q,), "norm"),)),
        WeightBinding(ld + "k_norm", (SourceTensor(ls + "k.norm", (k,), "norm"),)),
        WeightBinding(ld + "o_proj", (SourceTensor(ls + "o", (w, m.heads * m.vdim)),)),
        WeightBinding(rd + "yx_proj", (SourceTensor(rs + "y", (r, w)), SourceTensor(rs + "x", (r, w)))),
        WeightBinding(rd + "y_bias", (SourceTensor(rs + "y.b", (r,)),)),
        WeightBinding(rd + "x_bias", (SourceTensor(rs + "x.b", (r,)),)),
        WeightBinding(rd + "conv", (SourceTensor(rs + "conv", (r, m.conv)),)),
        WeightBinding(rd + "conv_bias", (SourceTensor(rs + "conv.b", (r,)),)),
        WeightBinding(rd + "gates", (SourceTensor(rs + "ra", (m.blocks, size, size)),
                                     SourceTensor(rs + "ri", (m.blocks, size, size)))),
        WeightBinding(rd + "r_bias", (SourceTensor(rs + "ra.b", (m.blocks, size)),)),
        WeightBinding(rd + "i_bias", (SourceTensor(rs + "ri.b", (m.blocks, size)),)),
        WeightBinding(rd + "lam", (SourceTensor(rs + "lam", (r,)),)),
        WeightBinding(rd + "o_proj", (SourceTensor(rs + "o", (w, r)),)),
        WeightBinding(dst + "left_out", (SourceTensor(ls + "out", (w,), "norm"),)),
        WeightBinding(dst + "right_out", (SourceTensor(rs + "out", (w,), "norm"),))]


def sigudra_weight_plan(c: SigudraConfig) -> List[WeightBinding]:
    c.need_ranks()
    w = c.width
    plan = [WeightBinding("embedding.weight", (SourceTensor("embed", (c.vocab, w)),))]
    if c.bigram is not None:
        plan.append(WeightBinding("embedding.pairs", (SourceTensor("bigram", (c.bigram.buckets + 1, w)),)))
    for i, l in enumerate(c.layers):
        src, dst = f"l{i}.", f"layers.{i}."
        mixer = _channel_delta if isinstance(l.mixer, ChannelDelta) else \
            _gated_linear if isinstance(l.mixer, GatedLinear) else _parallel
        plan += mixer(l.mixer, w, src + "mix.", dst + "mixer.")
        plan.append(WeightBinding(dst + "mixer_norm.weight", (SourceTensor(src + "norm1", (w,), "norm"),)))
        if l.ff is None:
            continue
        plan.append(WeightBinding(dst + "ff_norm.weight", (SourceTensor(src + "norm2", (w,), "norm"),)))
        f, ff = src + "mlp.", l.ff.ff
        if l.ff.kind == "dense":
            plan += [WeightBinding(dst + "feed_forward.gate_up_proj", (SourceTensor(f + "gate", (ff, w)),
                                                                       SourceTensor(f + "up", (ff, w)))),
                     WeightBinding(dst + "feed_forward.down_proj", (SourceTensor(f + "down", (w, ff)),))]
            continue
        gate_up, down = [], []
        for e in range(l.ff.experts):
            gate_up += [SourceTensor(f"{f}e{e}.gate", (ff, w)), SourceTensor(f"{f}e{e}.up", (ff, w))]
            down.append(SourceTensor(f"{f}e{e}.down", (w, ff)))
        plan += [WeightBinding(dst + "feed_forward.router", (SourceTensor(f + "router", (l.ff.experts, w)),)),
                 WeightBinding(dst + "feed_forward.gate_up_proj", tuple(gate_up)),
                 WeightBinding(dst + "feed_forward.down_proj", tuple(down))]
    plan.append(WeightBinding("final_norm.weight", (SourceTensor("final.norm", (w,), "norm"),)))
    plan.append(WeightBinding("lm_head.weight", (SourceTensor("head", (c.vocab, w)),)))
    return plan


SIGUDRA = Architecture(name=SigudraConfig.architecture, model_type=SigudraConfig.model_type,
                       parse_config=SigudraConfig.parse, model_spec=SigudraConfig.model_spec,
                       weight_plan=sigudra_weight_plan, checkpoint_dtype=lambda c: "bfloat16",
                       sizes_from_shapes=SigudraConfig.with_ranks)

register_architecture(SIGUDRA, replace=True)
