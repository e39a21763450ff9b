"""Bevuvik on the host: configuration, registry, weight plan, run list and cache plan, and the plain implementation's own
checks."""
import copy
import math

import pytest
import torch

import bevuvik_kit as K
import plain_bevuvik as P
from llm_infer_rust_b200 import ConfigError, resolve_architecture

ALL = dict(K.CONFIGS, diff=K.ONLY_DIFF, pair=K.ONLY_PAIR)


def test_the_architecture_is_found_by_its_name_and_every_size_comes_from_the_file():
    raw = K.CONFIGS["B1"]
    arch = resolve_architecture(raw)
    assert arch.name == "Bevuvik"
    c = arch.parse_config(raw)
    assert (c.vocab, c.width, c.eps, c.residual_mult, len(c.layers)) == (97, 40, 1e-5, 0.4, 4)
    a, p = c.layers[1].mixer, c.layers[0].mixer
    assert (a.heads, a.kv_heads, a.dim, a.vdim, a.scale, a.diff, a.window) == (4, 2, 12, 20, 0.28, 0.35, 24)
    assert (a.rot.base, a.rot.dims, a.rot.scaling.factor, a.rot.scaling.original, a.rot.scaling.fast, a.rot.scaling.slow) == \
        (50000.0, 8, 4.0, 64, 16.0, 1.0)
    assert (p.heads, p.kv_heads, p.dim, p.vdim, p.scale, p.softcap, p.rot.dims) == (4, 2, 12, 14, 0.3, 8.0, 6)
    assert (p.right_heads, p.right_kv_heads, p.right_dim, p.right_vdim, p.conv) == (6, 2, 12, 16, 3)
    assert (c.layers[0].ff.ff, c.layers[0].ff.limit) == (28, 1.0) and c.layers[2].ff is None
    spec = arch.model_spec(c)
    assert [(e.layer, e.input) for e in spec.run_list] == [(0, None), (1, "loop"), (2, None), (1, "loop"), (2, None), (3, None)]
    assert all(e.reads is None for e in spec.run_list)
    assert not spec.lm_head["tied"] and "feed_forward" not in spec.layers[2].parts
    assert spec.layers[1].block["residual_mult"] == 0.4 and spec.layers[1]["mixer"]["bias"] and spec.layers[1]["mixer"]["out_bias"]
    assert spec.layers[0]["mixer"]["right"]["decay_per"] == "head" and spec.layers[0]["mixer"]["right"]["q_scale"] == 12 ** -0.5
    encodings = spec.position_encodings
    assert encodings[spec.layers[1]["mixer"]["position_encoding"]]["pairing"] == "interleaved"
    assert encodings[spec.layers[0]["mixer"]["left"]["position_encoding"]]["pairing"] == "half_split"
    none = arch.parse_config(K.CONFIGS["B4"])
    assert none.loop is None and none.layers[0].mixer.rot is None and none.layers[1].mixer.softcap is None
    assert not arch.model_spec(none).stream_inputs
    whole = arch.model_spec(arch.parse_config(K.CONFIGS["B3"]))
    assert [(e.layer, e.input is not None) for e in whole.run_list] == [(0, True), (1, False)] * 3 + [(2, False)]


@pytest.mark.parametrize("change,message", [
    (lambda r: r.pop("vocab"), "vocab"),
    (lambda r: r.pop("norm"), "norm"),
    (lambda r: r.pop("residual_mult"), "residual_mult"),
    (lambda r: r["layers"][0].update(type="mamba"), "type"),
    (lambda r: r["layers"][1]["mixer"].pop("diff"), "diff"),
    (lambda r: r["layers"][1]["mixer"].update(kv_heads=3), "kv_heads"),
    (lambda r: r["layers"][1]["mixer"]["rot"].update(dims=14), "dims"),
    (lambda r: r["layers"][1]["mixer"]["rot"]["scaling"].pop("slow"), "slow"),
    (lambda r: r["layers"][1]["mixer"].update(vdim=7), "vdim"),
    (lambda r: r["layers"][0]["mixer"].pop("right"), "right"),
    (lambda r: r["layers"][0]["mixer"]["left"].pop("scale"), "scale"),
    (lambda r: r["layers"][0]["mixer"]["right"].update(conv=9), "taps"),
    (lambda r: r["layers"][0]["mixer"]["right"].update(kv_heads=4), "kv_heads"),
    (lambda r: r["layers"][0]["mlp"].pop("limit"), "limit"),
    (lambda r: r["layers"][0]["mlp"].update(kind="moe"), "mlp.kind"),
    (lambda r: r["loop"].update(stop=5), "loop"),
    (lambda r: r["loop"].update(times=0), "times"),
])
def test_a_configuration_that_lacks_or_contradicts_is_refused(change, message):
    raw = copy.deepcopy(K.CONFIGS["B1"])
    change(raw)
    with pytest.raises(ConfigError, match=message):
        resolve_architecture(raw).parse_config(raw)


@pytest.mark.parametrize("name", sorted(ALL))
def test_the_weight_plan_names_every_tensor_of_a_checkpoint_once(name):
    raw = ALL[name]
    arch = resolve_architecture(raw)
    plan = arch.weight_plan(arch.parse_config(raw))
    names = [s.name for b in plan for s in b.sources]
    assert len(names) == len(set(names))
    w = K.random_weights(raw, 1)
    assert {s.name: tuple(s.shape) for b in plan for s in b.sources} == {n: tuple(t.shape) for n, t in w.items()}


def test_every_pass_has_pages_and_states_of_its_own_and_shares_its_weights():
    from llm_infer_rust_b200.cache import plan_cache
    from llm_infer_rust_b200.parts import DecoderModel
    raw = K.CONFIGS["B1"]
    arch = resolve_architecture(raw)
    c = arch.parse_config(raw)
    model = DecoderModel(arch.model_spec(c), torch.float32, torch.device("cpu"))
    assert set(model.parameter_shapes()) == {b.param for b in arch.weight_plan(c)}
    assert model.parameter_shapes()["stream_inputs.loop.weight"] == (40, 80)
    plan = plan_cache(model, 8, 4)
    # runs 0 and 5 once; 1 and 3 the same attention layer, 2 and 4 the same pair
    assert [(g.window, g.entries) for g in plan.groups] == [(None, [0, 2, 4]), (24, [1, 3]), (30, [5])]
    for run in (2, 4):
        assert plan.block_states[run]["mixer.right.state"].shape == (2, 20, 8)
        assert plan.block_states[run]["mixer.right.conv"].shape == (3, 56)
    spec = model.blocks[1].mixer.cache_spec()
    assert (spec.num_kv_heads, spec.head_dim, spec.v_head_dim) == (2, 24, 20)     # a key row holds both maps' keys


def test_lambda_is_taken_from_the_four_vectors():
    from llm_infer_rust_b200.parts import DecoderModel
    raw = K.ONLY_DIFF
    arch = resolve_architecture(raw)
    model = DecoderModel(arch.model_spec(arch.parse_config(raw)), torch.float32, torch.device("cpu"))
    w = K.random_weights(raw, 3)
    names = [f"l0.mix.{n}" for n in ("lq1", "lk1", "lq2", "lk2")]
    model.bind_parameter("layers.0.mixer.lambdas", torch.cat([w[n] for n in names]))
    want = P.diff_lambda(*(w[n].double() for n in names), 0.4)
    assert abs(model.blocks[0].mixer._lambda - float(want)) < 1e-12


@pytest.mark.parametrize("dims,base,scaling", [(16, 20000.0, (2.0, 128, 20.0, 1.5)), (8, 50000.0, (4.0, 64, 16.0, 1.0)),
                                               (32, 1e6, (16.0, 4096, 32.0, 1.0)), (4, 10.0, (8.0, 7, 4.0, 3.9)), (6, 77.0, None)])
def test_scaled_frequencies_and_their_gain(dims, base, scaling):
    from llm_infer_rust_b200.config.spec import PartSpec
    from llm_infer_rust_b200.parts import BuildEnv, build_part
    spec = {"rotary_dim": dims, "theta": base, "pairing": "interleaved"}
    named = dict(zip(("factor", "original", "fast", "slow"), scaling)) if scaling else None
    if named:
        spec["yarn"] = named
    part = build_part("position_encoding", PartSpec("rotary_frequencies", spec), BuildEnv(torch.float32, torch.device("cpu"), {}))
    freq, gain = P.yarn(dims, base, named)
    torch.testing.assert_close(part.inv_freq.double(), freq, rtol=1e-6, atol=0)
    assert abs(part.gain - gain) < 1e-12


# ----------------------------------------------------------------------------- the plain implementation's own checks
def test_plain_pieces_against_numbers_worked_by_hand():
    f = lambda *x: torch.tensor(x, dtype=torch.float64)
    assert torch.allclose(P.rms_norm(f(3.0, 4.0), f(1.0, 2.0), 0.0), f(3.0, 8.0) / math.sqrt(12.5))
    assert torch.allclose(P.unit(f(3.0, 4.0), 0.0), f(0.6, 0.8))
    assert abs(float(P.softplus(f(0.0))) - math.log(2)) < 1e-15
    x = f(1.0, 2.0, 3.0).view(3, 1)
    assert P.causal_conv(x, f(10.0, 1.0).view(1, 2)).flatten().tolist() == [1.0, 12.0, 23.0]
    assert P.window_mask(4, 2).long().tolist() == [[1, 0, 0, 0], [1, 1, 0, 0], [0, 1, 1, 0], [0, 0, 1, 1]]
    g = P.clamped_glu(f(5.0, -1.0), f(0.5, -9.0), 2.0)
    assert torch.allclose(g, f(2.0 / (1 + math.exp(-3.404)) * 1.5, -1.0 / (1 + math.exp(1.702)) * -1.0))
    # two maps that agree leave (1 - lambda) of their output, whose size the norm takes out again
    a = f(3.0, 4.0).view(1, 1, 2)
    assert torch.allclose(P.difference(a, a, 0.25, 0.5, 0.0), 0.5 * a / math.sqrt(12.5))
    assert torch.allclose(P.difference(a, 2 * a, 1.5, 0.5, 0.0), -0.5 * a / math.sqrt(12.5))


def test_plain_rotation_and_frequencies():
    f = lambda *x: torch.tensor(x, dtype=torch.float64)
    freq, gain = P.yarn(4, 100.0, None)
    assert torch.allclose(freq, f(1.0, 0.1)) and gain == 1.0
    x = torch.zeros(2, 1, 5, dtype=torch.float64)
    x[1, 0] = f(1.0, 2.0, 3.0, 4.0, 5.0)
    near = P.rotate(x, freq, 1.0, True)[1, 0]
    half = P.rotate(x, freq, 2.0, False)[1, 0]
    c, s, c2, s2 = math.cos(1), math.sin(1), math.cos(0.1), math.sin(0.1)
    assert torch.allclose(near, f(c - 2 * s, 2 * c + s, 3 * c2 - 4 * s2, 4 * c2 + 3 * s2, 5.0))
    assert torch.allclose(half, f(2 * (c - 3 * s), 2 * (2 * c2 - 4 * s2), 2 * (3 * c + s), 2 * (4 * c2 + 2 * s2), 5.0))
    # the highest frequencies are kept, the lowest divided by the factor
    freq, gain = P.yarn(32, 1e4, {"factor": 8.0, "original": 512, "fast": 32.0, "slow": 1.0})
    plain = P.frequencies(32, 1e4)
    assert freq[0] == plain[0] and abs(float(freq[-1] * 8 / plain[-1]) - 1) < 1e-12 and plain[6] / 8 < freq[6] < plain[6]
    assert abs(gain - (0.1 * math.log(8.0) + 1.0)) < 1e-15


def test_plain_recurrence_on_a_state_of_one_number():
    one = lambda *x: torch.tensor(x, dtype=torch.float64).view(-1, 1, 1)
    head = lambda *x: torch.tensor(x, dtype=torch.float64).view(-1, 1)
    o, S = P.delta_scan(one(1.0, 1.0), one(1.0, 2.0), one(3.0, 5.0), head(0.5, 0.25), head(1.0, 0.5))
    assert o.flatten().tolist() == [3.0, 4.25] and float(S) == 4.25      # S = 3; S = 0.75, u = 0.5 (5 - 1.5), S = 0.75 + 3.5


def test_plain_loop_runs_its_layers_in_turn():
    assert P.layer_runs(K.CONFIGS["B1"]) == [(0, False), (1, True), (2, False), (1, True), (2, False), (3, False)]
    assert P.layer_runs(K.CONFIGS["B4"]) == [(0, False), (1, False), (2, False)]
    arch = resolve_architecture(K.CONFIGS["B2"])
    runs = arch.model_spec(arch.parse_config(K.CONFIGS["B2"])).run_list
    assert P.layer_runs(K.CONFIGS["B2"]) == [(e.layer, e.input is not None) for e in runs]


@pytest.mark.parametrize("name", ["B1", "B3"])
def test_plain_model_is_causal_and_remembers_its_first_token(name):
    raw = K.CONFIGS[name]
    w = K.random_weights(raw, 3)
    ids = K.tokens(raw["vocab"], 40, 2)
    full = K.oracle(raw, w, ids)
    assert abs(full[:25] - K.oracle(raw, w, ids[:25])).max() < 1e-9
    other = [(ids[0] + 1) % raw["vocab"]] + ids[1:]
    assert abs(full[39] - K.oracle(raw, w, other)[39]).max() > 1e-4
