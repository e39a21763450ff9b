"""Bevuvik through the engine against the plain implementation (``plain_bevuvik.py``), in float32 and bfloat16.

Mechanisms alone (kernels against the plain functions, and one-layer models), whole prompts against token-by-token
decoding, portions down to two tokens, batches of unequal requests against each alone, pages and slots that are freed
and used again, keys that stand out just inside and just outside a window, far keys and slowly forgetting states, the
first tokens of a sequence, long decoding, drawn configurations, greedy generation through the scheduler, and trace
replay through ``bin/trace_run``.
"""
import numpy as np
import pytest
import torch

import bevuvik_kit as K
import plain_bevuvik as P

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
    for i, (name, raw) in enumerate(dict(K.CONFIGS, diff=K.ONLY_DIFF, pair=K.ONLY_PAIR).items()):
        w = K.random_weights(raw, 600 + i)
        out[name] = (raw, w, K.write_model(str(tmp_path_factory.mktemp("bevuvik_" + name)), raw, w))
    return out


def _i32(x, dev="cuda"):
    return torch.tensor(x, dtype=torch.int32, device=dev)


def close(got, want, dtype, f32=3e-5, bf16=2e-2):
    tol = f32 if dtype == torch.float32 else bf16
    scale = max(1.0, float(want.abs().max()))
    err = float((got.detach().cpu().double() - want).abs().max())
    assert err <= tol * scale, f"off by {err:.3e}, allowed {tol * scale:.3e}"


# ----------------------------------------------------------------------------- mechanisms alone
@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("width", [44, 70, 264, 13000])
def test_the_owed_sum_and_the_norm_behind_it(width, dtype):
    """x <- x + m (y + bias + f), or with the mean of two normed branches in place of y, then the norm, chosen rows of it,
    or the sum itself as columns of a wider matrix with the stream left alone."""
    from llm_infer_rust_b200.kernels import ops
    dev = torch.device("cuda")
    g = torch.Generator().manual_seed(width)
    T, eps, m = 7, 1e-5, 0.37
    x = torch.randn(T, width, generator=g) * 3 + 1
    a, b, f = ((torch.randn(T, width, generator=g) * s).to(dtype) for s in (5, 0.3, 2))
    bias, w, wa, wb = (1.0 + 0.5 * torch.randn(width, generator=g) for _ in range(4))
    d = lambda t: t.double()
    pair = 0.5 * (P.rms_norm(d(a), d(wa), eps) + P.rms_norm(d(b), d(wb), eps))
    on = lambda t: t.to(dev)
    branches = ops.NormedPair(on(a), on(b), on(wa), on(wb), eps)
    cases = [(dict(y=on(a)), d(a)), (dict(y=on(a), bias=on(bias)), d(a) + d(bias)), (dict(y=on(a), add=on(f)), d(a) + d(f)),
             (dict(y=on(a), add=on(f), bias=on(bias)), d(a) + d(f) + d(bias)), (dict(y=branches), pair),
             (dict(y=branches, add=on(f)), pair + d(f)), ({}, 0 * d(a))]
    for kw, total in cases:
        want = d(x) + m * total
        for out_dtype in DTYPES:
            stream = on(x).clone()
            got = ops.residual_sum(stream, mult=m, weight=on(w), eps=eps, out_dtype=out_dtype, **kw)
            close(stream, want, torch.float32)
            close(got, P.rms_norm(want, d(w), eps), out_dtype, bf16=5e-3)
            rows = [5, 0, 2]
            stream = on(x).clone()
            got = ops.residual_sum(stream, mult=m, weight=on(w), eps=eps, out_dtype=out_dtype, rows=_i32(rows), store=False, **kw)
            close(got, P.rms_norm(want, d(w), eps)[rows], out_dtype, bf16=5e-3)
            wide = torch.full((T, 2 * width + 3), 7.0, device=dev, dtype=out_dtype)
            ops.residual_sum(stream, mult=m, out=wide, column=width, store=False, **kw)
            assert torch.equal(stream.cpu(), x)
            close(wide[:, width:2 * width], want, out_dtype, bf16=5e-3)
            assert bool((wide[:, :width] == 7.0).all()) and bool((wide[:, 2 * width:] == 7.0).all())


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("whole_rows", [False, True])
@pytest.mark.parametrize("H,G,d,dv,dims,maps,interleaved", [
    (4, 2, 12, 20, 8, 2, True), (3, 1, 32, 16, 32, 2, True), (4, 2, 24, 16, 12, 2, True), (2, 2, 9, 6, 2, 2, False),
    (5, 5, 16, 16, 6, 1, False), (3, 3, 40, 8, 32, 1, False), (2, 1, 16, 32, 16, 2, False), (2, 1, 8, 8, 0, 2, True)])
def test_heads_before_attention(H, G, d, dv, dims, maps, interleaved, whole_rows, dtype):
    """Biases, scaled frequencies with a gain, both pairings, and two maps a head: keys of both in one cache row, query
    vectors zero outside their own map's columns; rows of whole 16-byte pieces (eight columns a thread) and others."""
    from llm_infer_rust_b200.kernels import ops
    dev = torch.device("cuda")
    g = torch.Generator().manual_seed(d)
    T, page = 11, 4
    n = (H + G) * maps * d + G * dv
    packed = K.bf16_values(torch.randn(T, n + (8 - n % 8 if whole_rows else 5), generator=g))
    bias = torch.randn(n, generator=g)
    freq, gain = P.yarn(dims, 1000.0, {"factor": 4.0, "original": 32, "fast": 8.0, "slow": 0.5}) if dims else P.rotation({})
    q = torch.full((T, H * maps * maps * d), 9.0, device=dev, dtype=dtype)
    k_cache = torch.full((6, G, page, maps * d), 9.0, device=dev, dtype=dtype)
    v_cache = torch.full((6, G, page, dv), 9.0, device=dev, dtype=dtype)
    order = [4, 2, 5]
    slots = [order[t // page] * page + t % page for t in range(T)]
    slots[7] = 0                                             # a padding row stores nothing
    ops.heads_prepare(packed.to(dev, dtype), q, k_cache, v_cache, _i32(list(range(T))), _i32(slots), H * maps, G, d, dv,
                      bias=bias.to(dev), inv_freq=freq.float().to(dev) if dims else None, rot_dims=dims, interleaved=interleaved, maps=maps,
                      rot_gain=gain)
    x = packed[:, :n].double() + bias.double()
    wq = P.rotate(x[:, :H * maps * d].reshape(T, H * maps, d), freq, gain, interleaved)
    wk = P.rotate(x[:, H * maps * d:(H + G) * maps * d].reshape(T, G * maps, d), freq, gain, interleaved).reshape(T, G, maps * d)
    wv = x[:, (H + G) * maps * d:].reshape(T, G, dv)
    got = q.view(T, H, maps, maps, d)
    for a in range(maps):
        for b in range(maps):
            if a == b:
                close(got[:, :, a, a], wq.reshape(T, H, maps, d)[:, :, a], dtype, 1e-5, 1e-2)
            else:
                assert bool((got[:, :, a, b] == 0).all())
    for t in range(T):
        rows = (k_cache[order[t // page], :, t % page], v_cache[order[t // page], :, t % page])
        if slots[t] == 0:
            assert all(bool((r == 9.0).all()) for r in rows)
        else:
            close(rows[0], wk[t], dtype, 1e-5, 1e-2)
            close(rows[1], wv[t], dtype, 1e-5, 1e-2)
    ops.check_errors(dev)


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("heads,dv", [(3, 20), (2, 64), (1, 7)])
def test_difference_of_two_outputs(heads, dv, dtype):
    from llm_infer_rust_b200.kernels import ops
    a = torch.randn(9, heads, 2, dv, generator=torch.Generator().manual_seed(dv)).to(dtype)
    a[4] = 0.0                                               # eps inside the root keeps a zero vector zero
    want = P.difference(a[:, :, 0].double(), a[:, :, 1].double(), 0.7, 0.4, 1e-5)
    got = ops.head_difference(a.reshape(9, -1).cuda(), heads, dv, 0.7, 0.6, 1e-5)
    close(got.view(9, heads, dv), want, dtype, 1e-5, 5e-3)


def _attend(q, k, v, portions, dtype, window, scale, softcap=0.0, difference=None, page=8, splits_from=40):
    """q [T, vectors, d], k [T, G, d], v [T, G, dv] stored in pages handed out in a scrambled order and read by the
    attention kernels portion by portion; the outputs [T, heads, dv] (with ``difference``, half as many heads)."""
    from llm_infer_rust_b200.kernels import ops
    dev = torch.device("cuda")
    T, H, d = q.shape
    G, dv = k.shape[1], v.shape[2]
    pages = -(-T // page)
    order = torch.randperm(pages, generator=torch.Generator().manual_seed(7)) + 1
    k_cache = torch.full((pages + 1, G, page, d), 55.0, device=dev, dtype=dtype)        # stale values everywhere
    v_cache = torch.full((pages + 1, G, page, dv), 55.0, device=dev, dtype=dtype)
    table = order.to(torch.int32).reshape(1, -1).to(dev)
    fused = difference is not None and ops.fuses_difference(dtype, H, G, d, page, dv)
    kw = dict(v_head_dim=dv, softcap=softcap, precise_weights=True, difference=difference if fused else None)
    out, at = [], 0
    for n in portions:
        for p_ in range(at, at + n):
            k_cache[int(order[p_ // page]), :, p_ % page] = k[p_].to(dev, dtype)
            v_cache[int(order[p_ // page]), :, p_ % page] = v[p_].to(dev, dtype)
        qo = q[at:at + n].reshape(n, -1).to(dev, dtype).contiguous()
        o = torch.empty((n, (H // 2 if fused else H) * dv), device=dev, dtype=dtype)
        args = (table, _i32([0, n]), _i32([at + n]))
        if n > 1:
            ops.prefill_attention(qo, k_cache, v_cache, o, *args, _i32([at]), _i32([0]), 1, n, H, G, d, page, window, scale, **kw)
        else:
            splits = 1 + max(0, at - splits_from) // 15                      # one, clusters of two and four, and others
            scratch = torch.empty(max(ops.decode_scratch_floats(1, H, max(d, dv), splits), 1), device=dev)
            ops.decode_attention(qo, k_cache, v_cache, o, scratch, *args, _i32([0]), 1, H, G, d, page, window, scale,
                                 splits, **kw)
        if difference is not None and not fused:
            o = ops.head_difference(o, H // 2, dv, *difference)
        out.append(o.cpu().float().reshape(n, -1, dv))
        at += n
    ops.check_errors(dev)
    return torch.cat(out)


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("size", [24, 5, 8, 1, 33, None])
@pytest.mark.parametrize("d,dv,H,G", [(12, 14, 4, 2), (16, 32, 8, 1), (24, 64, 3, 1), (64, 128, 2, 2), (32, 16, 6, 2), (8, 208, 5, 5)])
def test_maps_at_a_windows_edges_and_the_first_key(d, dv, H, G, size, dtype):
    """For chosen queries, in prompt portions and decoded alone, the key just OUTSIDE the window is made to fit one map's
    query far better than any other (it would take all of that map's weight if it were seen), and for others the window's
    last key, or the very first key of the sequence; the maps differ, so that one standing for the other would show."""
    g = torch.Generator().manual_seed((size or 0) + d)
    T, lam, diff, eps = 100, 0.6, 0.35, 1e-5
    q = K.bf16_values(torch.randn(T, H, 2, d, generator=g))
    k = K.bf16_values(torch.randn(T, G, 2, d, generator=g))
    v = K.bf16_values(torch.randn(T, G, dv, generator=g))
    portions = [30, 2, 9, 1, 1, 1, 20, 1, 1, 17] + [1] * 17
    assert sum(portions) == T
    for n, i in enumerate((25, 31, 41, 42, 43, 55, 63, 64, 70, 83, 90, 99)):
        edge = (i - size) if size else 0                                      # the last key that is NOT seen
        for j, boost in ((edge, 6.0), (edge + 1, 4.0), (0, 3.0)):
            if 0 <= j <= i:
                k[j, :, n % 2] = K.bf16_values(boost * q[i, 0:1, n % 2] / q[i, 0, n % 2].norm() * 2.0)
    mask = P.window_mask(T, size)
    maps = [P.softmax_attention(q[:, :, a].double(), k[:, :, a].double(), v.double(), 0.7, mask) for a in range(2)]
    want = P.difference(maps[0], maps[1], lam, diff, eps)
    rows = torch.zeros(T, H, 2, 2, d)
    rows[:, :, 0, 0], rows[:, :, 1, 1] = q[:, :, 0], q[:, :, 1]
    got = _attend(rows.reshape(T, 2 * H, 2 * d), k.reshape(T, G, 2 * d), v, portions, dtype, size, 0.7,
                  difference=(lam, 1.0 - diff, eps))
    close(got, want, dtype, 3e-5, 3e-2)


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("d,dv,H,G", [(12, 14, 4, 2), (32, 32, 8, 1), (16, 48, 6, 2), (64, 16, 3, 3), (144, 256, 2, 1)])
def test_capped_scores_far_keys_and_values_of_another_width(d, dv, H, G, dtype):
    """Scores of tens under a cap of a few: the best key's share is set by the cap; the best key is far back."""
    g = torch.Generator().manual_seed(d + dv)
    T = 130
    q, k, v = (K.bf16_values(torch.randn(T, n, w, generator=g)) for n, w in ((H, d), (G, d), (G, dv)))
    for i in (40, 77, 100, 129):
        k[i // 9] = K.bf16_values(5.0 * q[i, :1] / q[i, 0].norm() * 3.0)
    want = P.softmax_attention(q.double(), k.double(), v.double(), 0.9, P.window_mask(T, None), softcap=4.0)
    got = _attend(q, k, v, [35, 2, 1, 1, 50, 1, 9] + [1] * 31, dtype, None, 0.9, softcap=4.0)
    close(got, want, dtype, 3e-5, 3e-2)


# heads, kv heads, d, dv, taps
STATES = [(6, 2, 12, 16, 3), (2, 2, 64, 64, 2), (3, 3, 10, 6, 1), (4, 1, 32, 64, 4), (2, 2, 128, 128, 4), (2, 1, 136, 264, 3),
          (1, 1, 260, 36, 2), (2, 2, 96, 192, 5), (1, 1, 4, 4, 8)]


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("column", [0, 16])
@pytest.mark.parametrize("sizes", STATES)
def test_a_delta_rule_with_one_decay_a_head_in_portions_beside_others(sizes, column, dtype):
    """Two sequences and a third that joins late, in steps of unequal portions, decoded tokens among them (steps of single
    tokens take the fused kernel where it fits), states of earlier users in every slot, the packed projection also as a
    column range of a wider matrix: the layer's output at every token against the plain one on the whole sequence."""
    from llm_infer_rust_b200.cache.paged import LayerCache
    from llm_infer_rust_b200.config.spec import PartSpec
    from llm_infer_rust_b200.kernels import ops
    from llm_infer_rust_b200.parts import BuildEnv, build_part
    H, G, d, dv, taps = sizes
    width = 24
    raw = K.config(16, width, 1e-5, 1.0, [K.pair((1, 1, 4, 4, 1.0, None, None), (H, G, d, dv, taps))])
    w = K.random_weights(raw, 31 + d)
    p = "l0.mix.right."
    part = build_part("mixer", PartSpec("channel_decay_attention", {
        "hidden_size": width, "num_heads": H, "num_kv_heads": G, "head_dim": d, "v_head_dim": dv, "eps": 1e-5,
        "conv_taps": taps, "qkv_silu": True, "qk_unit_eps": 1e-6, "q_scale": d ** -0.5, "decay": "softplus",
        "decay_per": "head", "delta": True, "gate": "silu"}), BuildEnv(dtype, torch.device("cuda"), {}))
    for n, t in {"in_proj": torch.cat([w[p + n] for n in ("q", "k", "v", "g", "a", "b")]), "norm": w[p + "norm"],
                 "o_proj": w[p + "o"], "decay_bias": w[p + "dt_bias"], "a_log": w[p + "A_log"],
                 "conv": torch.cat([w[p + n + ".conv"] for n in "qkv"])}.items():
        part.bind(n, t.to("cuda", dtype))
    assert not part.missing_params()
    g = torch.Generator().manual_seed(d + dv)
    lengths = [61, 40, 13]
    xs = [K.bf16_values(torch.randn(n, width, generator=g)) for n in lengths]
    cache = LayerCache(states={"mixer." + n: torch.full((6,) + tuple(s.shape), 37.0, device="cuda") for n, s in part.state_specs().items()})
    slots, at = [4, 2, 1], [0, 0, 0]
    got = [[] for _ in xs]
    for portions in [[5, 1, 0], [1, 2, 0], [1, 1, 0], [33, 1, 2], [2, 9, 3]] + [[1, 1, 1]] * 8 + [[11, 0, 0], [0, 18, 0]]:
        live = [r for r in range(3) if portions[r]]
        ctx = K.step_context([(slots[r], at[r], portions[r]) for r in live])
        x = torch.cat([xs[r][at[r]:at[r] + portions[r]] for r in live]).to("cuda", dtype)
        packed = ops.linear(x, part.params["in_proj"])
        if column:
            packed = torch.cat([torch.full((packed.shape[0], column), 3.0, device="cuda", dtype=dtype), packed], 1).contiguous()
        y = part.forward_packed(packed, column, ctx, cache)
        k = 0
        for r in live:
            got[r].append(y[k:k + portions[r]].float().cpu())
            k += portions[r]
            at[r] += portions[r]
    assert at == lengths
    wd = {n: t.double() for n, t in w.items()}
    for r, x in enumerate(xs):
        close(torch.cat(got[r]), P.gated_delta(x.double(), wd, p, raw["layers"][0]["mixer"]["right"], 1e-5), dtype, 3e-5, 3e-2)


@pytest.mark.parametrize("rows,heads,kv,d,dv", [(1, 2, 1, 48, 40), (1, 2, 2, 128, 96), (3, 8, 4, 64, 128), (1, 1, 1, 20, 260)])
def test_recurrence_with_strong_and_weak_decays(rows, heads, kv, d, dv):
    """The scan alone in float: decays from 1 (nothing is ever forgotten) to 0 (a token wipes the state), keys that repeat
    (the delta rule replaces the value), rows that go on from a given state; a row cut in four is the same up to rounding."""
    import ctypes
    from llm_infer_rust_b200.kernels import ops
    from llm_infer_rust_b200.kernels.build import load_cuda_library
    g = torch.Generator().manual_seed(d)
    T = 75
    q, k = torch.randn(rows, T, kv, d, generator=g), P.unit(torch.randn(rows, T, kv, d, generator=g))
    k[:, 40:50] = k[:, 10:20]
    v = torch.randn(rows, T, heads, dv, generator=g)
    decay = torch.exp(-torch.exp(3.0 * torch.randn(rows, T, heads, generator=g) - 3.0))
    decay[:, 7], decay[:, 20:30] = 0.0, 1.0
    beta = torch.rand(rows, T, heads, generator=g)
    beta[:, 45] = 1.0
    start = torch.randn(rows, heads, d, dv, generator=g)
    rep = heads // kv
    want = [P.delta_scan(q[r].double().repeat_interleave(rep, 1), k[r].double().repeat_interleave(rep, 1), v[r].double(),
                         decay[r].double(), beta[r].double(), start[r].double()) for r in range(rows)]
    lib = load_cuda_library("state_scan.cu", {"STATE_HEAD_BLOCKS": ops.state_head_blocks(d)})
    state = torch.full((rows + 2, heads, d, dv), 5.0, device="cuda")

    def scan(lo, hi):
        parts = [t[:, lo:hi].reshape(rows * (hi - lo), -1).cuda().contiguous() for t in (q, k, v, decay, beta)]
        out = torch.empty((rows * (hi - lo), heads * dv), device="cuda")
        ctx = K.step_context([(rows + 1 - r, 9 + lo, hi - lo) for r in range(rows)])
        ptr = lambda t: ctypes.c_void_p(t.data_ptr())
        rc = lib.b200_state_scan(*[ptr(t) for t in parts], ptr(out), ptr(state), ptr(ctx.cu_q), ptr(ctx.prefix_len),
                                 ptr(ctx.state_slots), rows, heads, kv, d, dv, 1,
                                 ctypes.c_void_p(torch.cuda.current_stream().cuda_stream))
        assert rc == 0
        torch.cuda.synchronize()
        return out.view(rows, hi - lo, heads, dv).cpu()

    def begin():
        for r in range(rows):
            state[rows + 1 - r] = start[r].cuda()
    begin()
    whole = scan(0, T)
    for r in range(rows):
        close(whole[r], want[r][0], torch.float32, 1e-5)
        close(state[rows + 1 - r], want[r][1], torch.float32, 1e-5)
    begin()
    cut_up = torch.cat([scan(0, 2), scan(2, 33), scan(33, 34), scan(34, T)], 1)
    close(cut_up, whole.double(), torch.float32, 1e-5)
    assert float(state[1].min()) == 5.0


@pytest.mark.parametrize("rows,width,ff", [(1, 64, 48), (5, 96, 130), (16, 256, 200), (40, 64, 48), (300, 2048, 640)])
def test_clamped_feed_forward_with_the_activation_in_the_products(rows, width, ff):
    """g' sigmoid(1.702 g') (u' + 1) as the epilogue of the few-row products (both kinds) and of the tcgen05 product, and
    the part that chooses among them; the clamps bite on both sides."""
    from llm_infer_rust_b200.config.spec import PartSpec
    from llm_infer_rust_b200.kernels import ops
    from llm_infer_rust_b200.parts import BuildEnv, build_part
    g = torch.Generator().manual_seed(rows)
    dev, bf, limit = torch.device("cuda"), torch.bfloat16, 0.8
    x = K.bf16_values(torch.randn(rows, width, generator=g))
    w = K.bf16_values(torch.randn(2 * ff, width, generator=g) * 1.5 * width ** -0.5)
    down = K.bf16_values(torch.randn(width, ff, generator=g) * ff ** -0.5)
    a, b = x.double() @ w[:ff].double().T, x.double() @ w[ff:].double().T
    assert float(a.max()) > limit and float(b.max()) > limit and float(b.min()) < -limit and float(a.min()) < -limit
    want = P.clamped_glu(a, b, limit)
    args = (x.to(dev, bf), w.to(dev, bf))
    if rows <= 16:
        close(ops.few_row_glu(*args, "clamped_swish", limit, 1.702), want, bf)
        if ops.stream_ok(rows, args[1], bf, ops.EPI_SWIGLU, False):
            close(ops.stream_linear(*args, ops.EPI_SWIGLU, glu="clamped_swish", limit=limit, alpha=1.702), want, bf)
    else:
        close(ops.gemm_tc(*args, ops.GEMM_SWIGLU, glu="clamped_swish", limit=limit, alpha=1.702), want, bf)
    for dtype in DTYPES:
        part = build_part("feed_forward", PartSpec("gated_act", {"hidden_size": width, "intermediate_size": ff,
                                                                 "activation": "clamped_swish", "limit": limit}), BuildEnv(dtype, dev, {}))
        part.bind("gate_up_proj", w.to(dev, dtype))
        part.bind("down_proj", down.to(dev, dtype))
        close(part.forward(x.to(dev, dtype)), want @ down.double().T, dtype)
    ops.check_errors(dev)


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("tokens,width", [(1, 40), (9, 64), (50, 72)])
def test_a_pass_begins_with_the_product_of_stream_and_embedding(tokens, width, dtype):
    """Twice in a row, the second time with a sum still owed to the stream: x0 is the first input both times."""
    from llm_infer_rust_b200.config.spec import PartSpec
    from llm_infer_rust_b200.parts import BuildEnv, build_part
    from llm_infer_rust_b200.parts.norm import OwedSum
    g = torch.Generator().manual_seed(tokens)
    part = build_part("stream_input", PartSpec("concat_input", {"width": width}), BuildEnv(dtype, torch.device("cuda"), {}))
    weight = K.bf16_values(torch.randn(width, 2 * width, generator=g) * (2 * width) ** -0.5)
    part.bind("weight", weight.to("cuda", dtype))
    x0, y = (K.bf16_values(torch.randn(tokens, width, generator=g)) for _ in range(2))
    stream = x0.cuda()
    kept = part.begin(stream)
    stream, residual = part.forward(stream, None, kept)
    assert residual is None and stream.dtype == torch.float32
    want = torch.cat([x0, x0], 1).double() @ weight.double().T
    close(stream, want, dtype, 1e-5, 1e-2)
    stream, residual = part.forward(OwedSum(y.to("cuda", dtype), None, 0.5), stream, kept)
    want = torch.cat([want + 0.5 * y.double(), x0.double()], 1) @ weight.double().T
    close(stream, want, dtype, 1e-5, 1e-2)


# ----------------------------------------------------------------------------- models
@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("name", ["B1", "B2", "B3", "B4", "diff", "pair"])
def test_whole_decoded_and_in_portions(name, dtype, models):
    raw, w, folder = models[name]
    T = 150
    ids = K.tokens(raw["vocab"], T, 3)
    want = K.oracle(raw, w, ids)
    eng = K.make_engine(folder, dtype, page_size=8, pool_tokens=256)
    tol = K.tolerance(name, dtype)
    K.check_most(K.run_alone(eng, 1, ids, [T]), want, dtype, "whole", tol)
    K.check_most(K.run_alone(eng, 2, ids, [T - 40] + [1] * 40), want, dtype, "last 40 decoded", tol)
    K.check_most(K.run_alone(eng, 3, ids, cut(T, PORTIONS)), want, dtype, "in portions", tol)
    K.check_most(K.run_alone(eng, 4, ids[:24], [1] * 24), want[:24], dtype, "token by token from the first", tol)
    K.check_most(K.run_alone(eng, 5, ids[:61], [2] * 30 + [1]), want[:61], dtype, "two tokens at a time", tol)
    assert eng.cache.manager.check() == ""


def test_every_layer_run_against_the_plain_stream(models):
    """The float32 stream after every layer run (looped layers count each time), whole and cut into portions."""
    from llm_infer_rust_b200.engine import StepEntry
    from llm_infer_rust_b200.kernels import ops
    for name in ("B1", "B3"):
        raw, w, folder = models[name]
        ids = K.tokens(raw["vocab"], 60, 5)
        layers = []
        K.oracle(raw, w, ids, layers)
        eng = K.make_engine(folder, "float32", page_size=8, pool_tokens=128)
        caught = []
        for block in eng.model.blocks:
            def wrapped(h, residual, ctx, cache, inner=block.forward):
                owed, stream = inner(h, residual, ctx, cache)
                caught.append(ops.residual_sum(stream, y=owed.y, add=owed.add, bias=owed.bias, mult=owed.mult,
                                               store=False).cpu().double())
                return owed, stream
            block.forward = wrapped
        eng.open_request(1)
        for lo, hi in ((0, 33), (33, 35), (35, 60)):
            eng.step([StepEntry(1, ids[lo:hi], [])])
        n = len(layers)
        assert len(caught) == 3 * n == 3 * len(P.layer_runs(raw))
        for i in range(n):
            got = torch.cat([caught[s * n + i] for s in range(3)])
            torch.testing.assert_close(got, layers[i], rtol=3e-5, atol=3e-5, msg=lambda m, i=i: f"{name}, layer run {i}: {m}")


def drawn_config(seed):
    """A configuration whose every size, option and layer order is drawn: any model of the design must run as it is."""
    import random
    rng = random.Random(seed)
    even = lambda lo, hi: 2 * rng.randint(lo // 2, hi // 2)

    def feed_forward():
        return None if rng.random() < 0.2 else K.dense(rng.randint(8, 64), rng.uniform(0.5, 4.0))

    def width(step=1):
        return step * rng.randint(1, 64 // step) if rng.random() < 0.5 else rng.choice([16, 32, 48, 64])

    def rotation(dim, scaled):
        dims = 2 * rng.randint(1, dim // 2)
        scaling = (rng.choice([2.0, 8.0, 40.0]), rng.choice([30, 256, 4096]), rng.uniform(8, 40), rng.uniform(0.5, 4)) if scaled else None
        return K.rot(rng.choice([50.0, 1e4, 5e5]), dims, scaling)

    layers = []
    for _ in range(rng.randint(2, 4)):
        kv, group = rng.randint(1, 3), rng.randint(1, 4)
        if rng.random() < 0.5:
            dim = rng.choice([8, 16, 32]) if rng.random() < 0.5 else rng.randint(2, 40)
            layers.append(K.attention(kv * group, kv, dim, rng.choice([2 * dim, even(4, 40), 16 * rng.randint(1, 6)]),
                                      rng.uniform(0.1, 0.5), rng.uniform(0.1, 0.8),
                                      rotation(dim, rng.random() < 0.7), rng.choice([None, rng.randint(1, 70)]), feed_forward()))
        else:
            dim = rng.choice([16, 32, 64]) if rng.random() < 0.5 else even(4, 40)
            right_kv = rng.randint(1, 3)
            layers.append(K.pair((kv * group, kv, dim, rng.choice([dim, even(4, 40), 16 * rng.randint(1, 6)]), rng.uniform(0.1, 0.5),
                                  rng.choice([2.0, 10.0, 50.0]), rotation(dim, False)),
                                 (right_kv * rng.randint(1, 3), right_kv, width(), width(), rng.randint(1, 6)), feed_forward()))
    n = len(layers)
    start = rng.randint(0, n - 1)
    loop = rng.choice([None, (start, rng.randint(start + 1, n), rng.randint(1, 3))])
    return K.config(rng.randint(50, 300), rng.randint(24, 96), rng.choice([1e-5, 1e-6, 3e-4]), rng.uniform(0.2, 1.0), layers, loop)


@pytest.mark.parametrize("seed", range(10))
def test_configurations_drawn_at_random(seed, tmp_path):
    raw = drawn_config(seed)
    T = 90
    ids = K.tokens(raw["vocab"], T, seed)
    w = K.random_weights(raw, 700 + seed)
    folder = K.write_model(str(tmp_path / "m"), raw, w)
    want = K.oracle(raw, w, ids)
    for dtype in ("float32", "bfloat16"):
        eng = K.make_engine(folder, dtype, page_size=(4, 8, 16)[seed % 3], pool_tokens=256)
        K.check_most(K.run_alone(eng, 1, ids, [T]), want, dtype, f"{seed} whole")
        K.check_most(K.run_alone(eng, 2, ids, [T - 30] + [1] * 30), want, dtype, f"{seed} last 30 decoded")
        K.check_most(K.run_alone(eng, 3, ids, cut(T, [2, 17, 3, 40, 1, 5])), want, dtype, f"{seed} in portions")
        assert eng.cache.manager.check() == ""
        del eng


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_far_tokens(dtype, models):
    """Prompts of hundreds of tokens over many pages: maps so sharp that the best key inside the window takes nearly all of
    a position's weight, attention without a window beside states that remember hundreds of tokens (the plain logits at
    the end move when the first token is another one)."""
    for name in ("diff", "pair", "B3"):
        raw, w, folder = models[name]
        T = 400
        ids = K.tokens(raw["vocab"], T, 11)
        want = K.oracle(raw, w, ids)
        if name != "diff":
            other = K.oracle(raw, w, [(ids[0] + 1) % raw["vocab"]] + ids[1:])
            assert np.abs(want[300:] - other[300:]).max() > 3 * K.TOL["float32"] * np.abs(want).max()
        eng = K.make_engine(folder, dtype, page_size=16, pool_tokens=448)
        tol = K.tolerance(name, dtype)
        K.check_most(K.run_alone(eng, 1, ids, [T]), want, dtype, name + " whole", tol)
        K.check_most(K.run_alone(eng, 2, ids, [T - 70, 37, 2] + [1] * 31), want, dtype, name + " tail decoded", tol)
        K.check_most(K.run_alone(eng, 3, ids, cut(T, [127, 2, 16, 129, 15, 1 + 16 * 6, 14])), want, dtype, name + " in portions", tol)
        del eng


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("name", ["B1", "B2"])
def test_mixed_batches_with_pages_and_slots_used_again(name, dtype, models):
    """Up to three live requests of unequal length in a pool that holds far less than all of them: portions of some
    beside decoded tokens of others, and every position's logits as alone."""
    from llm_infer_rust_b200.engine import StepEntry
    from replay_driver import mixed_schedule
    raw, w, folder = models[name]
    lengths = {"a": 90, "b": 37, "c": 120, "d": 5, "e": 64, "f": 101}
    reqs = {r: (K.tokens(raw["vocab"], n, 20 + i), max(2, n - 12 - i)) for i, (r, n) in enumerate(lengths.items())}
    want = {r: K.oracle(raw, w, ids) for r, (ids, _) in reqs.items()}
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
        K.check_most(np.concatenate(got[r]), want[r], dtype, f"request {r} in mixed batches")


def test_pages_and_slots_that_are_used_again_hold_nothing_of_their_last_user(models):
    """One request at a time in a pool of a few pages and one state slot: the second gets what the first one left full."""
    raw, w, folder = models["B1"]
    eng = K.make_engine(folder, "float32", page_size=4, pool_tokens=64, max_requests=1)
    first, second = K.tokens(raw["vocab"], 50, 1), K.tokens(raw["vocab"], 33, 2)
    K.check(K.run_alone(eng, 1, first, [20, 30]), K.oracle(raw, w, first), "float32", "first user", K.TOL["float32"])
    K.check(K.run_alone(eng, 2, second, [1, 1, 31]), K.oracle(raw, w, second), "float32", "second user", K.TOL["float32"])
    K.check(K.run_alone(eng, 3, first, [50]), K.oracle(raw, w, first), "float32", "third user", K.TOL["float32"])


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_long_decoding(dtype, models):
    raw, w, folder = models["B2"]
    ids = K.tokens(raw["vocab"], 260, 8)
    eng = K.make_engine(folder, dtype, page_size=16, pool_tokens=320)
    K.check_most(K.run_alone(eng, 1, ids, [6] + [1] * 254), K.oracle(raw, w, ids), dtype, "254 tokens decoded one by one")


@pytest.mark.parametrize("dtype,graphs,portion_graphs", [("float32", 0, 0), ("bfloat16", 0, 0), ("bfloat16", 4, 0),
                                                         ("bfloat16", 4, 64)])
def test_greedy_generation_through_the_scheduler(dtype, graphs, portion_graphs, models):
    """``Engine.generate``: prompts cut by the scheduler's token budget, more prompts than slots, decode graphs in
    bfloat16, and graphs of prompt portions whose shape comes again.  float32: the tokens are the plain
    implementation's; bfloat16: every generated token is one whose plain logit is within a small margin of the best."""
    from llm_infer_rust_b200 import SamplingParams
    raw, w, folder = models["B2"]
    prompts = [K.tokens(raw["vocab"], n, 40 + n) for n in (5, 23, 1, 12, 30, 64, 50)]
    eng = K.make_engine(folder, dtype, page_size=8, pool_tokens=512, max_requests=3, cuda_graph_bs=graphs,
                        chunked_prefill_size=16, max_prefill_tokens_per_batch=16,
                        prefill_cuda_graph_max_tokens=portion_graphs)
    results = eng.generate(prompts, SamplingParams(max_tokens=12, ignore_eos=True))
    eng.check_kernel_errors()
    for prompt, res in zip(prompts, results):
        assert len(res.tokens) == 12
        logits = K.oracle(raw, w, prompt + res.tokens)
        for i, tok in enumerate(res.tokens):
            row = logits[len(prompt) - 1 + i]
            margin = 1e-4 if dtype == "float32" else 0.08 * max(1.0, np.abs(row).max())
            assert row[tok] >= row.max() - margin, f"token {i} of a prompt of {len(prompt)}: {tok} is not the best"


def test_trace_replay_as_a_user_runs_it(models, tmp_path):
    from replay_driver import Replay, run_alone
    raw, w, folder = models["B1"]
    ids = K.tokens(raw["vocab"], 70, 9)
    want = K.oracle(raw, w, ids)
    for dtype in ("bfloat16", "float32"):
        rp = Replay(folder, dtype, 128, str(tmp_path / dtype), raw["vocab"], ["--page-size", "8"])
        try:
            K.check_most(run_alone(rp, "x", ids, [33, 2, 3] + [1] * 32), want, dtype, "replay", 1e-4 if dtype == "float32" else None)
        finally:
            assert rp.close() == 0


def test_command_line_random_weights_mode(tmp_path):
    """The command line writes a random Bevuvik model from a configuration and serves it; the same folder through
    ``Engine.generate`` gives the same tokens."""
    import json
    import os
    import subprocess
    import sys
    from llm_infer_rust_b200 import SamplingParams
    root = os.path.dirname(os.path.dirname(os.path.abspath(__file__)))
    cfg = tmp_path / "cfg.json"
    cfg.write_text(json.dumps(K.CONFIGS["B1"]))
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
