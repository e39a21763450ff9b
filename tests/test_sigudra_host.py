"""Sigudra on the host: configuration, registry, weight plan, cache plan, and the plain implementation's own checks."""
import copy
import math

import pytest
import torch

import plain_sigudra as P
import sigudra_kit as K
from llm_infer_rust_b200 import ConfigError, resolve_architecture

ALL = dict(K.CONFIGS, window=K.ONLY_WINDOW, delta=K.ONLY_DELTA, gla=K.ONLY_GLA, one=K.ONE_EXPERT)


def test_the_architecture_is_found_by_its_name_and_every_size_comes_from_the_file():
    raw = K.as_given(K.CONFIGS["S1"])
    arch = resolve_architecture(raw)
    assert arch.name == "Sigudra"
    c = arch.parse_config(raw)
    assert (c.vocab, c.width, c.eps, len(c.layers)) == (97, 40, 1e-5, 5)
    assert (c.bigram.buckets, c.bigram.mul_prev, c.bigram.mul_cur) == (53, 31, 5)
    g, p, d = c.layers[0].mixer, c.layers[1].mixer, c.layers[2].mixer
    assert (g.heads, g.dim, g.vdim, g.tau, g.decay_rank) == (3, 20, 12, 8.0, 5)
    assert (p.heads, p.kv_heads, p.dim, p.vdim, p.scale, p.window, p.right_width, p.blocks, p.conv) == \
        (4, 2, 12, 20, 0.3, 24, 36, 3, 4)
    assert (d.heads, d.kv_heads, d.dim, d.vdim, d.conv, d.decay_rank, d.gate_rank) == (6, 2, 12, 16, 4, 7, 9)
    assert (c.layers[0].ff.kind, c.layers[0].ff.ff, c.layers[0].ff.experts, c.layers[0].ff.top) == ("moe", 20, 5, 2)
    assert c.layers[1].ff.kind == "dense" and c.layers[1].ff.ff == 28 and c.layers[3].ff is None
    spec = arch.model_spec(c)
    assert spec.embedding.kind == "pair_embedding" and spec.final_norm.kind == "output_layer_norm"
    assert not spec.lm_head["tied"] and "feed_forward" not in spec.layers[3].parts
    left, right = spec.layers[1]["mixer"]["left"], spec.layers[1]["mixer"]["right"]
    assert left["window"] == 24 and left["gate"] == "head" and left["qk_norm_scope"] == "projection"
    assert left.get("position_encoding") is None and right["blocks"] == 3
    assert spec.layers[0]["mixer"]["decay"] == "logistic" and spec.layers[2]["mixer"]["delta"]
    assert spec.layers[0]["feed_forward"]["weights_on"] == "input" and spec.layers[0]["feed_forward"]["scores"] == "sigmoid"
    none = arch.parse_config(K.as_given(K.CONFIGS["S3"]))
    assert none.bigram is None and arch.model_spec(none).embedding.kind == "token_embedding"
    assert none.layers[1].mixer.window is None


@pytest.mark.parametrize("change,message", [
    (lambda r: r.pop("vocab"), "vocab"),
    (lambda r: r.pop("norm"), "norm"),
    (lambda r: r["embedding"]["bigram"].pop("mul_cur"), "mul_cur"),
    (lambda r: r["layers"][0].update(type="mamba"), "type"),
    (lambda r: r["layers"][0]["mixer"].pop("tau"), "tau"),
    (lambda r: r["layers"][1]["mixer"].pop("right"), "right"),
    (lambda r: r["layers"][1]["mixer"]["left"].pop("scale"), "scale"),
    (lambda r: r["layers"][1]["mixer"]["left"].update(dim=7), "dim"),
    (lambda r: r["layers"][1]["mixer"]["right"].update(blocks=5), "blocks"),
    (lambda r: r["layers"][2]["mixer"].update(kv_heads=4), "kv_heads"),
    (lambda r: r["layers"][2]["mixer"].pop("conv"), "conv"),
    (lambda r: r["layers"][2]["mixer"].update(conv=9), "taps"),
    (lambda r: r["layers"][1]["mlp"].update(kind="experts"), "mlp.kind"),
    (lambda r: r["layers"][0]["mlp"]["router"].update(top=6), "top"),
    (lambda r: r["layers"][0]["mlp"]["expert"].pop("ff"), "ff"),
])
def test_a_configuration_that_lacks_or_contradicts_is_refused(change, message):
    raw = copy.deepcopy(K.as_given(K.CONFIGS["S1"]))
    change(raw)
    with pytest.raises(ConfigError, match=message):
        resolve_architecture(raw).parse_config(raw)


@pytest.mark.parametrize("name", sorted(ALL))
def test_the_weight_plan_names_every_tensor_of_a_checkpoint_once(name):
    raw = K.as_given(ALL[name])
    arch = resolve_architecture(raw)
    plan = arch.weight_plan(arch.parse_config(raw))
    names = [s.name for b in plan for s in b.sources]
    assert len(names) == len(set(names))
    w = K.random_weights(ALL[name], 1)
    assert {s.name: tuple(s.shape) for b in plan for s in b.sources} == {n: tuple(t.shape) for n, t in w.items()}


def test_ranks_come_from_the_tensors_shapes_and_are_missed_without_them(tmp_path):
    from llm_infer_rust_b200.weights import read_model_config
    raw = K.CONFIGS["S1"]
    arch = resolve_architecture(K.as_file(raw))
    c = arch.parse_config(K.as_file(raw))
    with pytest.raises(ConfigError, match="rank"):
        arch.model_spec(c)
    with pytest.raises(ConfigError, match="rank"):
        arch.weight_plan(c)
    w = K.random_weights(raw, 1)
    folder = K.write_model(str(tmp_path / "m"), K.as_file(raw), w)
    found, completed = read_model_config(folder)
    c = found.parse_config(completed)
    assert c == arch.parse_config(K.as_given(raw))
    assert c.layers[2].mixer.decay_rank == 7 and c.layers[2].mixer.gate_rank == 9 and c.layers[4].mixer.decay_rank == 11


def test_parts_inside_a_part_have_parameters_states_and_pages():
    from llm_infer_rust_b200.cache import plan_cache
    from llm_infer_rust_b200.parts import DecoderModel
    raw = K.as_given(K.CONFIGS["S1"])
    arch = resolve_architecture(raw)
    c = arch.parse_config(raw)
    model = DecoderModel(arch.model_spec(c), torch.float32, torch.device("cpu"))
    assert set(model.parameter_shapes()) == {b.param for b in arch.weight_plan(c)}
    assert model.parameter_shapes()["layers.1.mixer.right.gates"] == (6, 12, 12)
    plan = plan_cache(model, 8, 4)
    assert [(g.window, g.entries) for g in plan.groups] == [(24, [1]), (30, [3])]
    assert plan.block_states[1]["mixer.right.state"].shape == (36,) and plan.block_states[1]["mixer.right.conv"].shape == (3, 36)
    assert plan.block_states[2]["mixer.state"].shape == (6, 12, 16) and plan.block_states[2]["mixer.conv"].shape == (3, 144)
    assert set(plan.block_states[0]) == {"mixer.state"}
    assert plan.embedding_states["last_token"].dtype == torch.int32
    weight = torch.arange(6 * 12 * 12, dtype=torch.float32).view(6, 12, 12)
    model.bind_parameter("layers.1.mixer.right.gates", weight)
    stored = model.parameter("layers.1.mixer.right.gates")            # per block, its r rows and then its i rows
    assert torch.equal(stored[1, :12], weight[1]) and torch.equal(stored[1, 12:], weight[4])


# ----------------------------------------------------------------------------- the plain implementation's own checks
def test_plain_pieces_against_numbers_worked_by_hand():
    f = lambda *x: torch.tensor(x, dtype=torch.float64)
    assert torch.allclose(P.layer_norm(f(1.0, 3.0), f(2.0, 0.5), 0.0), f(-2.0, 0.5))
    assert torch.allclose(P.rms_norm(f(3.0, 4.0), f(1.0, 1.0), 0.0), f(3.0, 4.0) / math.sqrt(12.5))
    assert torch.allclose(P.unit(f(3.0, 4.0), 0.0), f(0.6, 0.8))
    assert abs(float(P.softplus(f(0.0))) - math.log(2)) < 1e-15 and abs(float(P.softplus(f(800.0))) - 800.0) < 1e-12
    assert abs(float(P.gelu_tanh(f(1.0))) - 0.8411919906082768) < 1e-12
    x = torch.tensor([[1.0], [2.0], [3.0]], dtype=torch.float64)
    assert torch.allclose(P.causal_conv(x, torch.tensor([[10.0, 1.0]], dtype=torch.float64)), torch.tensor([[1.0], [12.0], [23.0]], dtype=torch.float64))
    assert P.bigram_rows([4, 1, 4], 10, 7, 3) == [10, (4 * 7 + 1 * 3) % 10, (7 + 12) % 10]
    assert torch.equal(P.window_mask(4, 2), torch.tensor([[1, 0, 0, 0], [1, 1, 0, 0], [0, 1, 1, 0], [0, 0, 1, 1]], dtype=torch.bool))


def test_plain_recurrences_on_a_state_of_one_number():
    one = lambda *x: torch.tensor(x, dtype=torch.float64).view(-1, 1, 1)
    q, k, v, g = one(1.0, 1.0), one(1.0, 2.0), one(3.0, 5.0), one(0.5, 0.25)
    o, S = P.gla_scan(q, k, v, g)
    assert o.flatten().tolist() == [3.0, 0.25 * 3.0 + 10.0] and float(S) == 10.75
    beta = torch.tensor([[1.0], [0.5]], dtype=torch.float64)
    o, S = P.delta_scan(q, k, v, g, beta)               # S = 3; then S = 0.75, u = 0.5 (5 - 1.5) = 1.75, S = 0.75 + 3.5
    assert o.flatten().tolist() == [3.0, 4.25] and float(S) == 4.25
    # beta 1 and a unit key: the read-out of a key just written is its value
    o, _ = P.delta_scan(one(1.0), one(1.0), one(7.0), one(0.9), torch.ones(1, 1, dtype=torch.float64))
    assert float(o) == 7.0
    log_a = torch.log(torch.tensor([[0.6], [0.8]], dtype=torch.float64))
    S = P.lru_scan(log_a, torch.tensor([[1.0], [10.0]], dtype=torch.float64))
    assert torch.allclose(S.flatten(), torch.tensor([0.8, 0.8 * 0.8 + 0.6 * 10.0], dtype=torch.float64))


def test_plain_experts_take_their_score_on_the_input():
    f = lambda *x: torch.tensor(x, dtype=torch.float64)
    w = {"router": f(1.0, 3.0).view(2, 1)}
    for e, s in ((0, 1.0), (1, 2.0)):
        w[f"e{e}.gate"], w[f"e{e}.up"], w[f"e{e}.down"] = f(s).view(1, 1), f(1.0).view(1, 1), f(1.0).view(1, 1)
    y = P.experts_ff(f(0.5).view(1, 1), w, "", {"router": {"top": 1}})
    h = 0.5 / (1 + math.exp(-1.5))                       # the score of expert 1, on the input
    assert abs(float(y) - 2 * h / (1 + math.exp(-2 * h)) * h) < 1e-12


def test_plain_model_is_causal_and_starts_every_sequence_afresh():
    raw = K.CONFIGS["S1"]
    w = K.random_weights(raw, 3)
    ids = K.tokens(raw["vocab"], 40, 2)
    full = K.oracle(raw, w, ids)
    assert abs(full[:25] - K.oracle(raw, w, ids[:25])).max() < 1e-9
    # the first token is seen far behind the window: a lost state would show
    other = [(ids[0] + 1) % raw["vocab"]] + ids[1:]
    assert abs(full[39] - K.oracle(raw, w, other)[39]).max() > 1e-4
