"""Sigudra through the engine against the plain implementation (``plain_sigudra.py``), in float32 and bfloat16.

Mechanisms alone (kernels against the plain functions, and one-layer models), whole prompts against token-by-token
decoding, portions down to two tokens, batches of unequal requests against each alone, pages and slots that are freed
and used again, keys that stand out just inside and just outside a window, far keys and slowly forgetting states, the
first tokens of a sequence, long decoding, drawn configurations, greedy generation through the scheduler, and trace
replay through ``bin/trace_run``.
"""
import numpy as np
import pytest
import torch

import plain_sigudra as P
import sigudra_kit as K

pytestmark = pytest.mark.gpu

PORTIONS = [2, 37, 3, 16, 64, 5, 1, 22]
DTYPES = [torch.float32, torch.bfloat16]


def cut(total, sizes):
    out, k = [], 0
    while total > 0:
        n = min(total, sizes[k % len(sizes)])
        out.append(n)
        total -= n
        k += 1
    return out


@pytest.fixture(scope="module")
def models(tmp_path_factory):
    """name -> (config, weights, folder stored in bfloat16)."""
    out = {}
    named = dict(K.CONFIGS, window=K.ONLY_WINDOW, delta=K.ONLY_DELTA, gla=K.ONLY_GLA, one=K.ONE_EXPERT)
    for i, (name, raw) in enumerate(named.items()):
        w = K.clear_weights(raw, 500 + i, K.tokens(raw["vocab"], 150, 3), tries=6)
        out[name] = (raw, w, K.write_model(str(tmp_path_factory.mktemp("sigudra_" + name)), K.as_file(raw), w))
    return out


def _i32(x, dev="cuda"):
    return torch.tensor(x, dtype=torch.int32, device=dev)


def close(got, want, dtype, f32=3e-5, bf16=2e-2):
    tol = f32 if dtype == torch.float32 else bf16
    scale = max(1.0, float(want.abs().max()))
    err = float((got.detach().cpu().double() - want).abs().max())
    assert err <= tol * scale, f"off by {err:.3e}, allowed {tol * scale:.3e}"


# ----------------------------------------------------------------------------- mechanisms alone
@pytest.mark.parametrize("y_dtype", DTYPES)
@pytest.mark.parametrize("width", [44, 70, 264, 13000])
def test_layer_norm_on_the_output_and_the_mean_of_two_normed_branches(width, y_dtype):
    """x <- x + LN(y) in place on a float32 stream, with the rounded copy; the same with the mean of two RMS-normed
    branches in place of y (one kernel); and the layer norm of chosen rows.  The rows have a mean far from zero."""
    from llm_infer_rust_b200.kernels import ops
    dev = torch.device("cuda")
    g = torch.Generator().manual_seed(width)
    T, eps = 7, 1e-5
    x = torch.randn(T, width, generator=g) * 3 + 2
    a, b = ((torch.randn(T, width, generator=g) * s + m).to(y_dtype) for s, m in ((5, 9), (0.3, -1)))
    w, wa, wb = (1.0 + 0.3 * torch.randn(width, generator=g) for _ in range(3))
    want = x.double() + P.layer_norm(a.double(), w.double(), eps)
    both = 0.5 * (P.rms_norm(a.double(), wa.double(), eps) + P.rms_norm(b.double(), wb.double(), eps))
    want_pair = x.double() + P.layer_norm(both, w.double(), eps)
    want_rms = x.double() + P.rms_norm(both, w.double(), eps)
    pair = ops.NormedPair(a.to(dev), b.to(dev), wa.to(dev), wb.to(dev), eps)
    for cast_to in (torch.bfloat16, torch.float32, None):
        for call, expect in ((lambda s: ops.norm_add(s, a.to(dev), w.to(dev), eps, cast_to=cast_to, center=True), want),
                             (lambda s: ops.norm_add_pair(s, pair, w.to(dev), eps, cast_to=cast_to, center=True), want_pair),
                             (lambda s: ops.norm_add_pair(s, pair, w.to(dev), eps, cast_to=cast_to), want_rms)):
            stream = x.to(dev).clone()
            got = call(stream)
            close(stream, expect, torch.float32)
            if cast_to is torch.bfloat16:
                assert torch.equal(got, stream.to(torch.bfloat16))
            elif cast_to is torch.float32:
                assert got.data_ptr() == stream.data_ptr()
            else:
                assert got is None
    rows = [5, 0, 5, 2]
    for out_dtype in DTYPES:
        got = ops.norm_rows(x.to(dev), w.to(dev), eps, out_dtype, rows=_i32(rows), center=True)
        close(got, P.layer_norm(x.double(), w.double(), eps)[rows], out_dtype)


@pytest.mark.parametrize("dtype", DTYPES)
def test_pair_table_across_portions_and_slots(dtype):
    """Rows of several requests in one step, some beginning their sequence, some going on from the token that an earlier
    step left in their slot; products of ids and multipliers beyond 32 bits."""
    from llm_infer_rust_b200.kernels import ops
    dev = torch.device("cuda")
    g = torch.Generator().manual_seed(3)
    vocab, width, buckets, mp, mc = 120, 36, 41, 2000000011, 1999999973
    table, pairs = (K.bf16_values(torch.randn(n, width, generator=g)) for n in (vocab, buckets + 1))
    seqs = [K.tokens(vocab, n, n) for n in (9, 1, 14)]
    seqs[2][0] = seqs[2][1] = 7
    slots, last = [3, 1, 2], torch.full((5, 1), -99, dtype=torch.int32, device=dev)
    got = [[] for _ in seqs]
    at = [0, 0, 0]
    for portions in ([4, 1, 1], [1, 0, 2], [2, 0, 1], [2, 0, 10]):
        live = [r for r in range(3) if portions[r]]
        ctx = K.step_context([(slots[r], at[r], portions[r]) for r in live])
        ids = [t for r in live for t in seqs[r][at[r]:at[r] + portions[r]]]
        out = ops.pair_embedding(_i32(ids), table.to(dev, dtype), pairs.to(dev, dtype), last, ctx, buckets, mp, mc, torch.float32)
        k = 0
        for r in live:
            got[r].append(out[k:k + portions[r]].cpu())
            k += portions[r]
            at[r] += portions[r]
    for r, seq in enumerate(seqs):
        want = table[torch.tensor(seq)] + pairs[torch.tensor(P.bigram_rows(seq, buckets, mp, mc))]
        assert torch.equal(torch.cat(got[r]), want)
        assert int(last[slots[r]]) == seq[-1]
    ops.check_errors(dev)


# heads, kv heads, d, dv, taps, decay rank, gate rank
STATES = [(6, 2, 12, 16, 4, 7, 9), (2, 2, 64, 64, 2, 16, 8), (3, 3, 10, 6, 1, 3, 4), (4, 1, 32, 64, 3, 8, 16),
          (2, 2, 128, 128, 4, 16, 24), (2, 1, 136, 264, 3, 5, 2), (1, 1, 260, 36, 2, 8, 8), (2, 2, 96, 192, 5, 8, 8),
          (1, 1, 4, 4, 8, 1, 1)]


def _state_layer(H, G, d, dv, taps, ra, rg, kind, seed):
    """A layer's tensors (float32, bfloat16-representable) and its part, on the device."""
    from llm_infer_rust_b200.config.spec import PartSpec
    from llm_infer_rust_b200.parts import BuildEnv
    from llm_infer_rust_b200.parts.linear_state import ChannelDecayAttention
    width = 24
    raw = K.config(16, width, 1e-5, [K.delta(H, G, d, dv, taps, (ra, rg)) if kind == "delta" else K.gla(H, d, dv, 6.0, ra)])
    w = K.random_weights(raw, seed)
    spec = {"hidden_size": width, "num_heads": H, "num_kv_heads": G if kind == "delta" else H, "head_dim": d, "v_head_dim": dv,
            "eps": 1e-5, "q_scale": d ** -0.5, "decay_rank": ra}
    names = ("q", "k", "v", "a1", "g1", "b") if kind == "delta" else ("q", "k", "v", "g", "a1")
    if kind == "delta":
        spec.update(conv_taps=taps, qkv_silu=True, qk_unit_eps=1e-6, decay="softplus", delta=True, gate="low_rank_sigmoid",
                    gate_rank=rg)
    else:
        spec.update(decay="logistic", tau=6.0, gate="silu")
    p = "l0.mix."

    def part(dtype):
        m = ChannelDecayAttention(PartSpec("channel_decay_attention", spec), BuildEnv(dtype, torch.device("cuda"), {}))
        bind = {"in_proj": torch.cat([w[p + n] for n in names]), "a2": w[p + "a2"], "norm": w[p + "norm"], "o_proj": w[p + "o"],
                "decay_bias": w[p + ("dt_bias" if kind == "delta" else "a2.b")]}
        if kind == "delta":
            bind.update(conv=torch.cat([w[p + n + ".conv"] for n in "qkv"]), a_log=w[p + "A_log"], g2=w[p + "g2"])
        for n, t in bind.items():
            m.bind(n, t.to("cuda", dtype))
        assert not m.missing_params()
        return m
    return raw, w, part, width


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("kind", ["delta", "gla"])
@pytest.mark.parametrize("sizes", STATES)
def test_a_state_layer_in_portions_beside_others_in_scrambled_slots(sizes, kind, dtype):
    """Two sequences and a third that joins late, in steps of unequal portions, decoded tokens among them (steps of single
    tokens take the fused kernel where it fits), states of earlier users in every slot: the layer's output at every
    token against the plain one on the whole sequence."""
    from llm_infer_rust_b200.cache.paged import LayerCache
    H, G, d, dv, taps, ra, rg = sizes
    raw, w, make, width = _state_layer(H, G, d, dv, taps, ra, rg, kind, 31 + d)
    part = make(dtype)
    g = torch.Generator().manual_seed(d + dv)
    lengths = [61, 40, 13]
    xs = [K.bf16_values(torch.randn(n, width, generator=g)) for n in lengths]
    cache = LayerCache(states={"mixer." + n: torch.full((6,) + tuple(s.shape), 37.0, device="cuda") for n, s in part.state_specs().items()})
    slots, at = [4, 2, 1], [0, 0, 0]
    got = [[] for _ in xs]
    steps = [[5, 1, 0], [1, 2, 0], [1, 1, 0], [33, 1, 2], [2, 9, 3]] + [[1, 1, 1]] * 8 + [[11, 0, 0], [0, 18, 0]]
    for portions in steps:
        live = [r for r in range(3) if portions[r]]
        ctx = K.step_context([(slots[r], at[r], portions[r]) for r in live])
        x = torch.cat([xs[r][at[r]:at[r] + portions[r]] for r in live]).to("cuda", dtype)
        y = part.forward(x, ctx, cache)
        k = 0
        for r in live:
            got[r].append(y[k:k + portions[r]].float().cpu())
            k += portions[r]
            at[r] += portions[r]
    assert at == lengths
    wd = {n: t.double() for n, t in w.items()}
    plain = P.channel_delta if kind == "delta" else P.gla
    m = dict(raw["layers"][0]["mixer"])
    for r, x in enumerate(xs):
        close(torch.cat(got[r]), plain(x.double(), wd, "l0.mix.", m, 1e-5), dtype, 3e-5, 3e-2)


@pytest.mark.parametrize("heads,kv,d,dv,delta", [(2, 1, 48, 40, True), (2, 2, 128, 96, True), (3, 3, 64, 32, False), (1, 1, 20, 260, True)])
def test_recurrence_with_strong_and_weak_decays(heads, kv, d, dv, delta):
    """The scan alone in float: decays from 1 (nothing is ever forgotten) to 0 (a token wipes a channel), keys that repeat
    (the delta rule replaces the value), rows that go on from a given state; a row cut in four is the same up to rounding."""
    import ctypes
    from llm_infer_rust_b200.kernels import ops
    g = torch.Generator().manual_seed(d)
    T = 75
    q, k = torch.randn(T, kv, d, generator=g), P.unit(torch.randn(T, kv, d, generator=g))
    k[40:50] = k[10:20]
    v = torch.randn(T, heads, dv, generator=g)
    decay = torch.exp(-torch.exp(3.0 * torch.randn(T, heads, d, generator=g) - 3.0))
    decay[7, :, ::3] = 0.0
    decay[:, :, 1::3] = 1.0
    beta = torch.rand(T, heads, generator=g)
    beta[45] = 1.0
    start = torch.randn(heads, d, dv, generator=g)
    rep = heads // kv
    args = (q.double().repeat_interleave(rep, 1), k.double().repeat_interleave(rep, 1), v.double(), decay.double())
    want, S = P.delta_scan(*args, beta.double(), start.double()) if delta else P.gla_scan(*args, start.double())
    dev = "cuda"
    state = torch.full((3, heads, d, dv), 5.0, device=dev)
    state[2] = start.to(dev)
    from llm_infer_rust_b200.kernels.build import load_cuda_library
    lib = load_cuda_library("state_scan.cu")

    def scan(lo, hi):
        parts = [t[lo:hi].reshape(hi - lo, -1).to(dev).contiguous() for t in (q, k, v, decay, beta)]
        out = torch.empty((hi - lo, heads * dv), device=dev)
        ctx = K.step_context([(2, 9 + lo, hi - lo)])
        p = [ctypes.c_void_p(t.data_ptr()) for t in parts]
        rc = lib.b200_state_scan(p[0], p[1], p[2], p[3], p[4] if delta else None, ctypes.c_void_p(out.data_ptr()),
                                 ctypes.c_void_p(state.data_ptr()), ctypes.c_void_p(ctx.cu_q.data_ptr()),
                                 ctypes.c_void_p(ctx.prefix_len.data_ptr()), ctypes.c_void_p(ctx.state_slots.data_ptr()), 1,
                                 heads, kv, d, dv, 0, ctypes.c_void_p(torch.cuda.current_stream().cuda_stream))
        assert rc == 0
        torch.cuda.synchronize()
        return out.cpu()
    whole = scan(0, T)
    close(whole.reshape(T, heads, dv), want, torch.float32, 1e-5)
    close(state[2], S, torch.float32, 1e-5)
    after = state[2].clone()
    state[2] = start.to(dev)
    cut_up = torch.cat([scan(0, 2), scan(2, 33), scan(33, 34), scan(34, T)])
    close(cut_up, whole.double(), torch.float32, 1e-5)
    close(state[2], after.cpu().double(), torch.float32, 1e-5)
    assert float(state[1].min()) == 5.0


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("width,blocks,taps", [(36, 3, 4), (64, 4, 5), (30, 1, 1), (22, 1, 2), (512, 2, 3), (264, 3, 8)])
def test_gated_recurrent_unit_in_portions_beside_others(width, blocks, taps, dtype):
    """The recurrent block as a part: steps of single tokens (few rows, and more than the few-row kernel takes), steps of
    unequal rows across the windows of 32 tokens that the scan is cut into, slots full of an earlier user's state."""
    from llm_infer_rust_b200.cache.paged import LayerCache
    from llm_infer_rust_b200.config.spec import PartSpec
    from llm_infer_rust_b200.parts import BuildEnv
    from llm_infer_rust_b200.parts.gated_lru import GatedLRU
    hidden = 20
    raw = K.config(16, hidden, 1e-5, [K.parallel(2, 1, 4, 4, 0.5, None, width, blocks, taps)])
    w = K.random_weights(raw, width)
    part = GatedLRU(PartSpec("gated_lru", {"hidden_size": hidden, "width": width, "blocks": blocks, "conv_taps": taps}),
                    BuildEnv(dtype, torch.device("cuda"), {}))
    p = "l0.mix.right."
    bind = {"yx_proj": torch.cat([w[p + "y"], w[p + "x"]]), "y_bias": w[p + "y.b"], "x_bias": w[p + "x.b"], "conv": w[p + "conv"],
            "conv_bias": w[p + "conv.b"], "gates": torch.cat([w[p + "ra"], w[p + "ri"]]), "r_bias": w[p + "ra.b"],
            "i_bias": w[p + "ri.b"], "lam": w[p + "lam"], "o_proj": w[p + "o"]}
    for n, t in bind.items():
        part.bind(n, t.to("cuda", dtype))
    assert not part.missing_params()
    g = torch.Generator().manual_seed(width)
    N = 19                                            # more rows than the few-row kernel takes
    lengths = [140, 50] + [7] * (N - 2)
    xs = [K.bf16_values(torch.randn(n, hidden, generator=g)) for n in lengths]
    cache = LayerCache(states={"mixer." + n: torch.full((N + 1,) + tuple(s.shape), 37.0, device="cuda") for n, s in part.state_specs().items()})
    slots = (torch.randperm(N, generator=g) + 1).tolist()
    at = [0] * N
    got = [[] for _ in xs]
    rest = [0] * (N - 2)
    steps = [[1] * N, [3, 1] + [1] * (N - 2), [70, 2] + [2] * (N - 2), [1] * N, [1, 1] + rest, [31, 33] + rest, [1, 1] + rest,
             [32, 10] + rest] + [[0, 0] + [2] * (N - 2)]
    for portions in steps:
        live = [r for r in range(N) if portions[r]]
        ctx = K.step_context([(slots[r], at[r], portions[r]) for r in live])
        y = part.forward(torch.cat([xs[r][at[r]:at[r] + portions[r]] for r in live]).to("cuda", dtype), ctx, cache)
        k = 0
        for r in live:
            got[r].append(y[k:k + portions[r]].float().cpu())
            k += portions[r]
            at[r] += portions[r]
    assert at == lengths
    wd = {n: t.double() for n, t in w.items()}
    for r, x in enumerate(xs):
        close(torch.cat(got[r]), P.gated_recurrent_unit(x.double(), wd, p), dtype, 3e-5, 3e-2)


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("column,channels,total", [(0, 24, 24), (8, 40, 64), (3, 21, 29)])
def test_convolution_of_a_column_range_with_biases(column, channels, total, dtype):
    """An input bias that the zeros before the start do not get, an output bias, columns inside a wider matrix; a row that
    goes on from its state."""
    from llm_infer_rust_b200.kernels import ops
    g = torch.Generator().manual_seed(total)
    taps, T = 3, 17
    x = K.bf16_values(torch.randn(T, total, generator=g))
    w, bias, out_bias = torch.randn(channels, taps, generator=g), torch.randn(channels, generator=g), torch.randn(channels, generator=g)
    want = P.causal_conv(x[:, column:column + channels].double() + bias.double(), w.double()) + out_bias.double()
    state = torch.full((3, taps - 1, channels), 9.0, device="cuda")
    out = []
    for lo, hi in ((0, 1), (1, 2), (2, 9), (9, 10), (10, T)):
        y = ops.causal_taps(x[lo:hi].to("cuda", dtype).contiguous(), w.cuda(), state, K.step_context([(1, lo, hi - lo)]), dtype,
                            channels=channels, column=column, bias=bias.cuda(), out_bias=out_bias.cuda())
        out.append(y.float().cpu())
    close(torch.cat(out), want, dtype)
    assert float(state[2].min()) == 9.0


@pytest.mark.parametrize("dtype", DTYPES)
def test_per_head_norm_with_weights_gates_and_the_tanh_gelu(dtype):
    from llm_infer_rust_b200.kernels import ops
    g = torch.Generator().manual_seed(8)
    T, H, dv, eps = 9, 3, 20, 1e-5
    o = torch.randn(T, H * dv, generator=g) * 3
    packed = K.bf16_values(torch.randn(T, H * dv + 7, generator=g) * 2)
    w = 1 + 0.3 * torch.randn(dv, generator=g)
    for gate, act in (("silu", P.silu), ("sigmoid", P.sigmoid)):
        want = P.rms_norm(o.double().reshape(T, H, dv), w.double(), eps).reshape(T, -1) * act(packed.double()[:, 5:5 + H * dv])
        got = ops.head_unit_norm_gate(o.cuda(), packed.to("cuda", dtype), 5, H, dv, eps, weight=w.cuda(), gate=gate)
        close(got, want, dtype)
    for width in (35, 40):
        gu = K.bf16_values(torch.randn(T, 2 * width, generator=g) * 3).double()
        close(ops.glu_columns(gu.to("cuda", dtype), "gelu_tanh"), P.gelu_tanh(gu[:, :width]) * gu[:, width:], dtype)


@pytest.mark.parametrize("rows,width,ff", [(1, 64, 40), (8, 264, 136), (16, 128, 520), (300, 256, 384)])
def test_gated_feed_forward_with_the_activation_in_the_products(rows, width, ff):
    """gelu_tanh(gate) * up as the epilogue of the few-row products (both kinds) and of the tcgen05 product, and the part
    that chooses among them; the silu builds beside them are left as they were."""
    from llm_infer_rust_b200.config.spec import PartSpec
    from llm_infer_rust_b200.kernels import ops
    from llm_infer_rust_b200.parts import BuildEnv, build_part
    g = torch.Generator().manual_seed(rows)
    dev, bf = torch.device("cuda"), torch.bfloat16
    x = K.bf16_values(torch.randn(rows, width, generator=g))
    w = K.bf16_values(torch.randn(2 * ff, width, generator=g) * 1.5 * width ** -0.5)
    down = K.bf16_values(torch.randn(width, ff, generator=g) * ff ** -0.5)
    a, b = x.double() @ w[:ff].double().T, x.double() @ w[ff:].double().T
    want = {"gelu_tanh": P.gelu_tanh(a) * b, "silu": P.silu(a) * b}
    for act in want:
        if rows <= 16:
            close(ops.few_row_glu(x.to(dev, bf), w.to(dev, bf), act), want[act], bf)
            if ops.stream_ok(rows, w.to(dev, bf), bf, ops.EPI_SWIGLU, False):
                close(ops.stream_linear(x.to(dev, bf), w.to(dev, bf), ops.EPI_SWIGLU, glu=act), want[act], bf)
        else:
            close(ops.gemm_tc(x.to(dev, bf), w.to(dev, bf), ops.GEMM_SWIGLU, glu=act), want[act], bf)
    for dtype in DTYPES:
        part = build_part("feed_forward", PartSpec("gated_act", {"hidden_size": width, "intermediate_size": ff,
                                                                 "activation": "gelu_tanh"}), BuildEnv(dtype, dev, {}))
        part.bind("gate_up_proj", w.to(dev, dtype))
        part.bind("down_proj", down.to(dev, dtype))
        close(part.forward(x.to(dev, dtype)), want["gelu_tanh"] @ down.double().T, dtype)
    ops.check_errors(dev)


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("tokens,width,ff,experts,top", [(1, 40, 24, 5, 2), (3, 33, 20, 4, 1), (70, 44, 20, 4, 1), (300, 64, 48, 3, 3),
                                                         (130, 248, 88, 12, 4), (700, 184, 136, 9, 2)])
def test_experts_with_weights_on_their_input(tokens, width, ff, experts, top, dtype):
    """Every kind of product (few pairs, tiles, tcgen05), experts with many, few and no tokens, and weights so far from
    one that a weight on the output instead would show: the activation is not linear."""
    from llm_infer_rust_b200.kernels import ops
    dev = torch.device("cuda")
    g = torch.Generator().manual_seed(tokens + top)
    w = {}
    for e in range(experts):
        w[f"e{e}.gate"] = K.bf16_values(torch.randn(ff, width, generator=g) * 2.0 * width ** -0.5)
        w[f"e{e}.up"] = K.bf16_values(torch.randn(ff, width, generator=g) * width ** -0.5)
        w[f"e{e}.down"] = K.bf16_values(torch.randn(width, ff, generator=g) * ff ** -0.5)
    choice = torch.stack([torch.randperm(experts, generator=g)[:top] for _ in range(tokens)])
    choice[: min(tokens, 40)] = choice[0]
    gains = 0.05 + 0.9 * torch.rand(tokens, top, generator=g)
    x = K.bf16_values(torch.randn(tokens, width, generator=g))
    wd = {n: t.double() for n, t in w.items()}
    want, swapped = torch.zeros(tokens, width, dtype=torch.float64), torch.zeros(tokens, width, dtype=torch.float64)
    for t in range(tokens):
        for e, s in zip(choice[t].tolist(), gains[t].double()):
            want[t] += P.expert(s * x[t:t + 1].double(), wd, f"e{e}.")[0]
            swapped[t] += s * P.expert(x[t:t + 1].double(), wd, f"e{e}.")[0]
    assert float((want - swapped).abs().max()) > 0.1
    gate_up = torch.cat([torch.cat([w[f"e{e}.gate"], w[f"e{e}.up"]]) for e in range(experts)]).view(experts, 2 * ff, width)
    down = torch.cat([w[f"e{e}.down"] for e in range(experts)]).view(experts, width, ff)
    args = (x.to(dev, dtype), choice.to(dev, torch.int32), gains.to(dev), gate_up.to(dev, dtype).contiguous(),
            down.to(dev, dtype).contiguous(), "silu")
    close(ops.routed_experts(*args, gains_on_input=True), want, dtype)
    close(ops.routed_experts(*args), swapped, dtype)
    if dtype == torch.bfloat16 and width % 8 == 0 and ff % 8 == 0 and tokens * top >= 128:
        for tensor_memory in (True, False):
            close(ops.routed_experts(*args, gains_on_input=True, tensor_memory=tensor_memory), want, dtype)
    ops.check_errors(dev)


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("tokens,width,experts,top", [(1, 40, 8, 3), (19, 44, 15, 1), (70, 64, 5, 5), (130, 33, 16, 2)])
def test_router_takes_sigmoid_scores_as_they_are(tokens, width, experts, top, dtype):
    from llm_infer_rust_b200.kernels import ops
    g = torch.Generator().manual_seed(tokens)
    x = K.bf16_values(torch.randn(tokens, width, generator=g))
    w = K.bf16_values(torch.randn(experts, width, generator=g) * 3.0 * width ** -0.5)
    s = P.sigmoid(x.double() @ w.double().T)
    want = s.topk(top, -1)
    choice, gains = ops.expert_router(x.to("cuda", dtype), w.to("cuda", dtype), top, scores="sigmoid")
    assert torch.equal(choice.cpu().long(), want.indices)
    torch.testing.assert_close(gains.cpu().double(), want.values, rtol=2e-5, atol=1e-7)
    # logits so large that many scores are 1 in 32 bits: the larger logit is chosen all the same
    big = K.bf16_values(w * 12.0)
    z = x.double() @ big.double().T
    choice, gains = ops.expert_router(x.to("cuda", dtype), big.to("cuda", dtype), top, scores="sigmoid")
    assert torch.equal(choice.cpu().long(), z.topk(top, -1).indices)


def _attend_in_portions(q, k, v, portions, dtype, window, scale, page=8):
    """q [T, H, d], k [T, G, d], v [T, G, dv] stored in pages handed out in a scrambled order and read by the attention
    kernels portion by portion; the outputs [T, H, dv]."""
    from llm_infer_rust_b200.kernels import ops
    dev = torch.device("cuda")
    T, H, d = q.shape
    G, dv = k.shape[1], v.shape[2]
    pages = -(-T // page)
    order = torch.randperm(pages, generator=torch.Generator().manual_seed(7)) + 1
    k_cache = torch.full((pages + 1, G, page, d), 55.0, device=dev, dtype=dtype)        # stale values everywhere
    v_cache = torch.full((pages + 1, G, page, dv), 55.0, device=dev, dtype=dtype)
    table = order.to(torch.int32).reshape(1, -1).to(dev)
    out, at = [], 0
    for n in portions:
        for p_ in range(at, at + n):
            k_cache[int(order[p_ // page]), :, p_ % page] = k[p_].to(dev, dtype)
            v_cache[int(order[p_ // page]), :, p_ % page] = v[p_].to(dev, dtype)
        qo = q[at:at + n].reshape(n, -1).to(dev, dtype).contiguous()
        o = torch.empty((n, H * dv), device=dev, dtype=dtype)
        args = (table, _i32([0, n]), _i32([at + n]))
        if n > 1:
            ops.prefill_attention(qo, k_cache, v_cache, o, *args, _i32([at]), _i32([0]), 1, n, H, G, d, page, window,
                                  scale, v_head_dim=dv, precise_weights=True)
        else:
            splits = 1 if at <= 40 else (2 if at <= 80 else 3)
            scratch = torch.empty(max(ops.decode_scratch_floats(1, H, max(d, dv), splits), 1), device=dev)
            ops.decode_attention(qo, k_cache, v_cache, o, scratch, *args, _i32([0]), 1, H, G, d, page, window, scale,
                                 splits, v_head_dim=dv, precise_weights=True)
        out.append(o.cpu().float().reshape(n, H, dv))
        at += n
    ops.check_errors(dev)
    return torch.cat(out)


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("size", [24, 5, 8, 1, 33, None])
@pytest.mark.parametrize("d,dv,H,G", [(12, 14, 4, 2), (32, 32, 8, 1), (48, 96, 4, 2), (96, 48, 6, 1), (16, 256, 2, 1)])
def test_keys_at_a_windows_edges_and_the_first_key(size, d, dv, H, G, dtype):
    """For chosen queries, in prompt portions and decoded alone, the key just OUTSIDE the window is made to fit the query
    far better than any other (it would take all the weight if it were seen), and for others the window's last key, or the
    very first key of the sequence; values wider and narrower than keys."""
    g = torch.Generator().manual_seed((size or 0) + d)
    T = 100
    q = K.bf16_values(torch.randn(T, H, d, generator=g))
    k = K.bf16_values(torch.randn(T, G, d, generator=g))
    v = K.bf16_values(torch.randn(T, G, dv, generator=g))
    portions = [30, 2, 9, 1, 1, 1, 20, 1, 1, 17] + [1] * 17
    assert sum(portions) == T
    for i in (25, 31, 41, 42, 43, 55, 63, 64, 70, 83, 90, 99):
        edge = (i - size) if size else 0                                      # the last key that is NOT seen
        for j, boost in ((edge, 6.0), (edge + 1, 4.0), (0, 3.0)):
            if 0 <= j <= i:
                k[j, :, :] = K.bf16_values(boost * q[i, 0:1, :] / q[i, 0].norm() * 2.0)
    rep = H // G
    want = P.softmax_attention(q.double(), k.double().repeat_interleave(rep, 1), v.double().repeat_interleave(rep, 1), 0.7,
                               P.window_mask(T, size))
    got = _attend_in_portions(q, k, v, portions, dtype, size, 0.7)
    close(got, want, dtype, 2e-5, 3e-2)


# ----------------------------------------------------------------------------- models
@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("name", ["S1", "S2", "S3", "S4", "window", "delta", "gla", "one"])
def test_whole_decoded_and_in_portions(name, dtype, models):
    if name == "one" and dtype == "bfloat16":
        pytest.skip("one expert a token: a near tie between two experts shows in full; compared in float32")
    raw, w, folder = models[name]
    T = 150
    ids = K.tokens(raw["vocab"], T, 3)
    want, unsure = K.oracle_and_close_calls(raw, w, ids)
    eng = K.make_engine(folder, dtype, page_size=8, pool_tokens=256)
    tol = K.tolerance(name, dtype)
    K.check_clear(K.run_alone(eng, 1, ids, [T]), want, unsure, dtype, "whole", tol)
    K.check_clear(K.run_alone(eng, 2, ids, [T - 40] + [1] * 40), want, unsure, dtype, "last 40 decoded", tol)
    K.check_clear(K.run_alone(eng, 3, ids, cut(T, PORTIONS)), want, unsure, dtype, "in portions", tol)
    K.check_clear(K.run_alone(eng, 4, ids[:24], [1] * 24), want[:24], unsure[:24], dtype, "token by token from the first", tol)
    K.check_clear(K.run_alone(eng, 5, ids[:61], [2] * 30 + [1]), want[:61], unsure[:61], dtype, "two tokens at a time", tol)
    assert eng.cache.manager.check() == ""


def test_every_layer_against_the_plain_stream(models):
    """The float32 stream after every layer, whole and cut into portions."""
    from llm_infer_rust_b200.engine import StepEntry
    raw, w, folder = models["S1"]
    ids = K.tokens(raw["vocab"], 60, 5)
    layers = []
    P.forward(raw, w, ids, dtype=torch.float64, layers_out=layers)
    eng = K.make_engine(folder, "float32", page_size=8, pool_tokens=128)
    caught = []
    for block in eng.model.blocks:
        def wrapped(h, residual, ctx, cache, inner=block.forward):
            out = inner(h, residual, ctx, cache)
            caught.append(out[0].detach().cpu().double().clone())
            return out
        block.forward = wrapped
    eng.open_request(1)
    for lo, hi in ((0, 33), (33, 35), (35, 60)):
        eng.step([StepEntry(1, ids[lo:hi], [])])
    n = len(raw["layers"])
    for i in range(n):
        got = torch.cat([caught[s * n + i] for s in range(3)])
        torch.testing.assert_close(got, layers[i], rtol=3e-5, atol=3e-5, msg=lambda m, i=i: f"layer {i}: {m}")


def drawn_config(seed):
    """A configuration whose every size, option and layer order is drawn: any model of the design must run as it is."""
    import random
    rng = random.Random(seed)
    even = lambda lo, hi: 2 * rng.randint(lo // 2, hi // 2)

    def feed_forward():
        kind = rng.choice(["none", "dense", "moe", "moe"])
        if kind == "none":
            return None
        if kind == "dense":
            return K.dense(rng.randint(8, 64))
        experts = rng.randint(2, 12)
        return K.moe(rng.randint(8, 40), experts, rng.randint(1 if experts > 4 else 2, min(experts, 4)))

    def size():
        return rng.choice([16, 32, 48, 64]) if rng.random() < 0.5 else rng.randint(3, 40)

    layers = []
    for _ in range(rng.randint(2, 5)):
        kind = rng.choice(["delta", "gla", "parallel"])
        kv = rng.randint(1, 3)
        if kind == "delta":
            layers.append(K.delta(kv * rng.randint(1, 3), kv, size(), size(), rng.randint(1, 6), (rng.randint(1, 20), rng.randint(1, 20)),
                                  feed_forward()))
        elif kind == "gla":
            layers.append(K.gla(rng.randint(1, 5), size(), size(), rng.choice([1.0, 4.0, 16.0, 50.0]), rng.randint(1, 20), feed_forward()))
        else:
            blocks = rng.randint(1, 4)
            dim = rng.choice([16, 32, 64]) if rng.random() < 0.5 else even(4, 40)
            layers.append(K.parallel(kv * rng.randint(1, 4), kv, dim, dim if rng.random() < 0.5 else even(4, 40),
                                     rng.uniform(0.1, 0.5), rng.choice([None, rng.randint(1, 70)]), blocks * rng.randint(4, 16),
                                     blocks, rng.randint(1, 6), feed_forward()))
    bigram = rng.choice([None, (rng.randint(2, 200), rng.randint(1, 200), rng.randint(1, 200))])
    return K.config(rng.randint(50, 300), rng.randint(24, 96), rng.choice([1e-5, 1e-6, 3e-4]), layers, bigram)


@pytest.mark.parametrize("seed", range(10))
def test_configurations_drawn_at_random(seed, tmp_path):
    raw = drawn_config(seed)
    T = 90
    ids = K.tokens(raw["vocab"], T, seed)
    w = K.clear_weights(raw, 700 + seed, ids)
    folder = K.write_model(str(tmp_path / "m"), K.as_file(raw), w)
    want, unsure = K.oracle_and_close_calls(raw, w, ids)
    for dtype in ("float32", "bfloat16"):
        eng = K.make_engine(folder, dtype, page_size=(4, 8, 16)[seed % 3], pool_tokens=256)
        K.check_clear(K.run_alone(eng, 1, ids, [T]), want, unsure, dtype, f"{seed} whole")
        K.check_clear(K.run_alone(eng, 2, ids, [T - 30] + [1] * 30), want, unsure, dtype, f"{seed} last 30 decoded")
        K.check_clear(K.run_alone(eng, 3, ids, cut(T, [2, 17, 3, 40, 1, 5])), want, unsure, dtype, f"{seed} in portions")
        assert eng.cache.manager.check() == ""
        del eng


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_far_tokens(dtype, models):
    """Prompts of hundreds of tokens over many pages: attention so sharp that the best key inside the window takes nearly
    all of a position's weight, and states that remember hundreds of tokens (the plain logits at the end move when the
    first token is another one)."""
    for name in ("window", "delta", "gla"):
        raw, w, folder = models[name]
        T = 400
        ids = K.tokens(raw["vocab"], T, 11)
        want = K.oracle(raw, w, ids)
        if name != "window":
            other = K.oracle(raw, w, [(ids[0] + 1) % raw["vocab"]] + ids[1:])
            assert np.abs(want[300:] - other[300:]).max() > 3 * K.TOL["float32"] * np.abs(want).max()
        eng = K.make_engine(folder, dtype, page_size=16, pool_tokens=448)
        tol = K.tolerance(name, dtype)
        K.check(K.run_alone(eng, 1, ids, [T]), want, dtype, name + " whole", tol)
        K.check(K.run_alone(eng, 2, ids, [T - 70, 37, 2] + [1] * 31), want, dtype, name + " tail decoded", tol)
        K.check(K.run_alone(eng, 3, ids, cut(T, [127, 2, 16, 129, 15, 1 + 16 * 6, 14])), want, dtype, name + " in portions", tol)
        del eng


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("name", ["S1", "S2"])
def test_mixed_batches_with_pages_and_slots_used_again(name, dtype, models):
    """Up to three live requests of unequal length in a pool that holds far less than all of them: portions of some
    beside decoded tokens of others, and every position's logits as alone."""
    from llm_infer_rust_b200.engine import StepEntry
    from replay_driver import mixed_schedule
    raw, w, folder = models[name]
    lengths = {"a": 90, "b": 37, "c": 120, "d": 5, "e": 64, "f": 101}
    reqs = {r: (K.tokens(raw["vocab"], n, 20 + i), max(2, n - 12 - i)) for i, (r, n) in enumerate(lengths.items())}
    want = {r: K.oracle_and_close_calls(raw, w, ids) for r, (ids, _) in reqs.items()}
    eng = K.make_engine(folder, dtype, page_size=8, pool_tokens=320, max_requests=3)
    got = {r: [] for r in reqs}
    number = {r: i + 1 for i, r in enumerate(reqs)}
    opened = set()
    for entries, end in mixed_schedule(reqs, 320, seed=4, max_live=3):
        batch = []
        for r, toks, wanted in entries:
            if r not in opened:
                eng.open_request(number[r])
                opened.add(r)
            batch.append(StepEntry(number[r], list(toks), list(wanted)))
        logits = eng.step(batch).cpu().numpy()
        at = 0
        for r, toks, _ in entries:
            got[r].append(logits[at:at + len(toks)].copy())
            at += len(toks)
        for r in end:
            eng.close_request(number[r])
        assert eng.cache.manager.check() == ""
    eng.check_kernel_errors()
    for r in reqs:
        K.check_clear(np.concatenate(got[r]), *want[r], dtype, f"request {r} in mixed batches")


def test_pages_and_slots_that_are_used_again_hold_nothing_of_their_last_user(models):
    """One request at a time in a pool of a few pages and one state slot: the second gets what the first one left full."""
    raw, w, folder = models["S1"]
    eng = K.make_engine(folder, "float32", page_size=4, pool_tokens=64, max_requests=1)
    first, second = K.tokens(raw["vocab"], 50, 1), K.tokens(raw["vocab"], 33, 2)
    K.check(K.run_alone(eng, 1, first, [20, 30]), K.oracle(raw, w, first), "float32", "first user", K.TOL["float32"])
    K.check(K.run_alone(eng, 2, second, [1, 1, 31]), K.oracle(raw, w, second), "float32", "second user", K.TOL["float32"])
    K.check(K.run_alone(eng, 3, first, [50]), K.oracle(raw, w, first), "float32", "third user", K.TOL["float32"])


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_long_decoding(dtype, models):
    raw, w, folder = models["S2"]
    ids = K.tokens(raw["vocab"], 260, 8)
    eng = K.make_engine(folder, dtype, page_size=16, pool_tokens=320)
    K.check_clear(K.run_alone(eng, 1, ids, [6] + [1] * 254), *K.oracle_and_close_calls(raw, w, ids), dtype,
                  "254 tokens decoded one by one")


@pytest.mark.parametrize("dtype,graphs,portion_graphs", [("float32", 0, 0), ("bfloat16", 0, 0), ("bfloat16", 4, 0),
                                                         ("bfloat16", 4, 64)])
def test_greedy_generation_through_the_scheduler(dtype, graphs, portion_graphs, models):
    """``Engine.generate``: prompts cut by the scheduler's token budget, more prompts than slots, decode graphs in
    bfloat16, and graphs of prompt portions whose shape comes again.  float32: the tokens are the plain
    implementation's; bfloat16: every generated token is one whose plain logit is within a small margin of the best."""
    from llm_infer_rust_b200 import SamplingParams
    raw, w, folder = models["S2"]
    prompts = [K.tokens(raw["vocab"], n, 40 + n) for n in (5, 23, 1, 12, 30, 64, 50)]
    eng = K.make_engine(folder, dtype, page_size=8, pool_tokens=512, max_requests=3, cuda_graph_bs=graphs,
                        chunked_prefill_size=16, max_prefill_tokens_per_batch=16,
                        prefill_cuda_graph_max_tokens=portion_graphs)
    results = eng.generate(prompts, SamplingParams(max_tokens=12, ignore_eos=True))
    eng.check_kernel_errors()
    for prompt, res in zip(prompts, results):
        assert len(res.tokens) == 12
        logits, unsure = K.oracle_and_close_calls(raw, w, prompt + res.tokens)
        for i, tok in enumerate(res.tokens):
            row = logits[len(prompt) - 1 + i]
            if dtype == "bfloat16" and unsure[len(prompt) - 1 + i]:
                continue
            margin = 1e-4 if dtype == "float32" else 0.08 * max(1.0, np.abs(row).max())
            assert row[tok] >= row.max() - margin, f"token {i} of a prompt of {len(prompt)}: {tok} is not the best"


def test_trace_replay_as_a_user_runs_it(models, tmp_path):
    from replay_driver import Replay, run_alone
    raw, w, folder = models["S1"]
    ids = K.tokens(raw["vocab"], 70, 9)
    want, unsure = K.oracle_and_close_calls(raw, w, ids)
    for dtype in ("bfloat16", "float32"):
        rp = Replay(folder, dtype, 128, str(tmp_path / dtype), raw["vocab"], ["--page-size", "8"])
        try:
            K.check_clear(run_alone(rp, "x", ids, [33, 2, 3] + [1] * 32), want, unsure, dtype, "replay",
                          1e-4 if dtype == "float32" else None)
        finally:
            assert rp.close() == 0


def test_command_line_random_weights_mode(tmp_path):
    """The command line writes a random Sigudra model from a configuration and serves it; the same folder through
    ``Engine.generate`` gives the same tokens."""
    import json
    import os
    import subprocess
    import sys
    from llm_infer_rust_b200 import SamplingParams
    root = os.path.dirname(os.path.dirname(os.path.abspath(__file__)))
    cfg = tmp_path / "cfg.json"
    cfg.write_text(json.dumps(K.as_given(K.CONFIGS["S1"])))
    made = tmp_path / "made"
    cmd = [sys.executable, "-m", "llm_infer_rust_b200", "--model-path", str(made), "--random-weights", "--config",
           str(cfg), "--seed", "5", "--dtype", "float32", "--page-size", "4", "--max-total-tokens", "256",
           "--max-running-req", "2", "--max-seq-len", "64", "--cuda-graph-bs", "0", "--prompt-ids", "1,2,3",
           "--prompt-ids", "9,8,7,6,5", "--max-tokens", "6", "--ignore-eos"]
    done = subprocess.run(cmd, cwd=root, capture_output=True, text=True, timeout=600)
    assert done.returncode == 0, done.stderr
    lines = [json.loads(x) for x in done.stdout.strip().splitlines()]
    eng = K.make_engine(str(made), "float32", page_size=4, pool_tokens=256, max_requests=2)
    want = eng.generate([[1, 2, 3], [9, 8, 7, 6, 5]], SamplingParams(max_tokens=6, ignore_eos=True))
    assert [x["output_ids"] for x in lines] == [r.tokens for r in want]
    eng.check_kernel_errors()
