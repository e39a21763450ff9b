"""Bevuvik as a registry entry: configuration, parts and checkpoint names.

Checkpoint names: ``embed``, ``final.norm``, ``head``, with looped layers ``loop.in`` [width, 2 width]; per layer i
``l<i>.norm1``, the mixer's tensors ``l<i>.mix.*`` and, with a feed-forward, ``l<i>.mlp.{gate,up,down}``:

    attention     q, k, v, o, each with a bias ``.b``; lq1, lk1, lq2, lk2
    parallel      left.{q,k,v,o}, left.out; right.{q,k,v} with .conv, right.{b,a,g}, right.A_log, right.dt_bias,
                  right.norm, right.o, right.out

Linear weights are [out, in].  The rows of the projections that read a mixer's input are packed into one matrix, in the
order that the parts name.
"""
from __future__ import annotations

from typing import List

from ..config.bevuvik import BevuvikConfig, CappedDeltaPair, DifferentialMixer
from ..config.registry import Architecture, register_architecture
from ..weights.plan import SourceTensor, WeightBinding


def _differential(m: DifferentialMixer, w: int, src: str, dst: str) -> List[WeightBinding]:
    q, k, v = m.heads * 2 * m.dim, m.kv_heads * 2 * m.dim, m.kv_heads * m.vdim
    return [
        WeightBinding(dst + "qkv_proj", (SourceTensor(src + "q", (q, w)), SourceTensor(src + "k", (k, w)),
                                         SourceTensor(src + "v", (v, w)))),
        WeightBinding(dst + "qkv_bias", (SourceTensor(src + "q.b", (q,)), SourceTensor(src + "k.b", (k,)),
                                         SourceTensor(src + "v.b", (v,)))),
        WeightBinding(dst + "lambdas", tuple(SourceTensor(src + n, (m.dim,)) for n in ("lq1", "lk1", "lq2", "lk2"))),
        WeightBinding(dst + "o_proj", (SourceTensor(src + "o", (w, m.heads * m.vdim)),)),
        WeightBinding(dst + "o_bias", (SourceTensor(src + "o.b", (w,)),))]


def _pair(m: CappedDeltaPair, w: int, src: str, dst: str) -> List[WeightBinding]:
    ls, ld, rs, rd = src + "left.", dst + "left.", src + "right.", dst + "right."
    q, k, v = m.heads * m.dim, m.kv_heads * m.dim, m.kv_heads * m.vdim
    rqk, rv = m.right_kv_heads * m.right_dim, m.right_heads * m.right_vdim
    return [
        WeightBinding(ld + "qkv_proj", (SourceTensor(ls + "q", (q, w)), SourceTensor(ls + "k", (k, w)),
                                        SourceTensor(ls + "v", (v, w)))),
        WeightBinding(ld + "o_proj", (SourceTensor(ls + "o", (w, m.heads * m.vdim)),)),
        WeightBinding(rd + "in_proj", (
            SourceTensor(rs + "q", (rqk, w)), SourceTensor(rs + "k", (rqk, w)), SourceTensor(rs + "v", (rv, w)),
            SourceTensor(rs + "g", (rv, w)), SourceTensor(rs + "a", (m.right_heads, w)),
            SourceTensor(rs + "b", (m.right_heads, w)))),
        WeightBinding(rd + "conv", (SourceTensor(rs + "q.conv", (rqk, m.conv)), SourceTensor(rs + "k.conv", (rqk, m.conv)),
                                    SourceTensor(rs + "v.conv", (rv, m.conv)))),
        WeightBinding(rd + "decay_bias", (SourceTensor(rs + "dt_bias", (m.right_heads,)),)),
        WeightBinding(rd + "a_log", (SourceTensor(rs + "A_log", (m.right_heads,)),)),
        WeightBinding(rd + "norm", (SourceTensor(rs + "norm", (m.right_vdim,), "norm"),)),
        WeightBinding(rd + "o_proj", (SourceTensor(rs + "o", (w, rv)),)),
        WeightBinding(dst + "left_out", (SourceTensor(ls + "out", (w,), "norm"),)),
        WeightBinding(dst + "right_out", (SourceTensor(rs + "out", (w,), "norm"),))]


def bevuvik_weight_plan(c: BevuvikConfig) -> List[WeightBinding]:
    w = c.width
    plan = [WeightBinding("embedding.weight", (SourceTensor("embed", (c.vocab, w)),))]
    if c.loop is not None:
        plan.append(WeightBinding("stream_inputs.loop.weight", (SourceTensor("loop.in", (w, 2 * w)),)))
    for i, l in enumerate(c.layers):
        src, dst = f"l{i}.", f"layers.{i}."
        plan.append(WeightBinding(dst + "input_norm.weight", (SourceTensor(src + "norm1", (w,), "norm"),)))
        mixer = _differential if isinstance(l.mixer, DifferentialMixer) else _pair
        plan += mixer(l.mixer, w, src + "mix.", dst + "mixer.")
        if l.ff is not None:
            f, ff = src + "mlp.", l.ff.ff
            plan += [WeightBinding(dst + "feed_forward.gate_up_proj", (SourceTensor(f + "gate", (ff, w)),
                                                                       SourceTensor(f + "up", (ff, w)))),
                     WeightBinding(dst + "feed_forward.down_proj", (SourceTensor(f + "down", (w, ff)),))]
    plan.append(WeightBinding("final_norm.weight", (SourceTensor("final.norm", (w,), "norm"),)))
    plan.append(WeightBinding("lm_head.weight", (SourceTensor("head", (c.vocab, w)),)))
    return plan


BEVUVIK = Architecture(name=BevuvikConfig.architecture, model_type=BevuvikConfig.model_type,
                       parse_config=BevuvikConfig.parse, model_spec=BevuvikConfig.model_spec,
                       weight_plan=bevuvik_weight_plan, checkpoint_dtype=lambda c: "bfloat16")

register_architecture(BEVUVIK, replace=True)
