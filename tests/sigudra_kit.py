"""Small Sigudra configurations, random weights for them and helpers that run them through the engine.

The configurations differ from one another in every size and option: head counts and groups, key and value widths, taps
from one to five, ranks, windows of many sizes (also the page's size, one position, or none), blocks of the recurrent
unit, dense, routed (one to all experts a token) and absent feed-forwards, with and without the pair table.  Weights are
drawn with torch's generator and are representable in bfloat16, so that the float32 engine, the bfloat16 engine and the
plain implementation read the same numbers.
"""
from __future__ import annotations

import contextlib
from types import SimpleNamespace
from typing import Dict, List, Sequence, Tuple

import numpy as np
import torch

import plain_sigudra as P
from kefetar_kit import bf16_values, check, make_engine, run_alone, tokens  # noqa: F401  (shared helpers)
from mukenex_kit import write_model  # noqa: F401


def delta(heads, kv_heads, dim, vdim, conv, ranks, mlp=None):
    """ranks: (decay, gate)."""
    return {"type": "channel_delta", "mixer": {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "conv": conv},
            "mlp": mlp, "_ranks": tuple(ranks)}


def gla(heads, dim, vdim, tau, rank, mlp=None):
    return {"type": "gla", "mixer": {"heads": heads, "dim": dim, "vdim": vdim, "tau": tau}, "mlp": mlp, "_ranks": (rank,)}


def parallel(heads, kv_heads, dim, vdim, scale, window, width, blocks, conv, mlp=None):
    left = {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "scale": scale}
    if window is not None:
        left["mask"] = {"size": window}
    return {"type": "parallel", "mixer": {"left": left, "right": {"width": width, "blocks": blocks, "conv": conv}}, "mlp": mlp}


def dense(ff):
    return {"kind": "dense", "ff": ff}


def moe(ff, experts, top):
    return {"kind": "moe", "expert": {"ff": ff}, "router": {"experts": experts, "top": top}}


def config(vocab, width, eps, layers, bigram=None):
    """bigram: (buckets, mul_prev, mul_cur) or None."""
    raw = {"architecture": "Sigudra", "vocab": vocab, "width": width, "norm": {"eps": eps}, "layers": layers}
    if bigram is not None:
        raw["embedding"] = {"bigram": dict(zip(("buckets", "mul_prev", "mul_cur"), bigram))}
    return raw


def as_file(raw: dict) -> dict:
    """The configuration as a config.json has it: without the ranks, which only the tensors' shapes tell."""
    return dict(raw, layers=[{k: v for k, v in l.items() if k != "_ranks"} for l in raw["layers"]])


def as_given(raw: dict) -> dict:
    """The configuration with the ranks named in it (for a model that has no checkpoint to ask)."""
    layers = []
    for l in as_file(raw)["layers"]:
        src = raw["layers"][len(layers)]
        if "_ranks" in src:
            l = dict(l, mixer=dict(l["mixer"], **dict(zip(("decay_rank", "gate_rank"), src["_ranks"]))))
        layers.append(l)
    return dict(raw, layers=layers)


CONFIGS = {
    # grouped heads in the delta rule, a window that is no multiple of a page, values wider than keys on the attention
    # side, odd widths everywhere, a layer without a feed-forward
    "S1": config(97, 40, 1e-5, [
        gla(3, 20, 12, 8.0, 5, moe(20, 5, 2)),
        parallel(4, 2, 12, 20, 0.3, 24, 36, 3, 4, dense(28)),
        delta(6, 2, 12, 16, 4, (7, 9), moe(16, 7, 3)),
        parallel(2, 2, 10, 6, 0.4, 30, 22, 1, 2),
        gla(2, 8, 24, 3.0, 11)], (53, 31, 5)),
    # sizes of the tensor-core and few-row kernels, every expert for every token, a window one longer than two pages
    "S2": config(211, 64, 1e-6, [
        delta(2, 2, 64, 64, 2, (16, 8), dense(96)),
        parallel(8, 2, 32, 32, 0.18, 33, 64, 4, 5, moe(24, 3, 3)),
        gla(4, 32, 64, 16.0, 16, moe(32, 6, 2)),
        delta(4, 1, 32, 64, 3, (8, 16), dense(24))], (101, 7, 3)),
    # taps of one, a state that is no whole 16-byte piece, heads wider than 128, no window, no pair table
    "S3": config(73, 72, 3e-6, [
        delta(3, 3, 10, 6, 1, (3, 4), moe(40, 4, 2)),
        parallel(2, 1, 16, 16, 0.25, None, 30, 5, 1, dense(48)),
        gla(1, 160, 136, 5.0, 6, dense(40)),
        delta(2, 1, 136, 264, 3, (5, 2))]),
    # multipliers whose products leave 32 bits, the window of one page
    "S4": config(150, 48, 1e-4, [
        parallel(3, 3, 24, 24, 0.2, 8, 48, 2, 3, dense(32)),
        gla(2, 24, 40, 1.0, 1)], (89, 2000000011, 1999999973)),
}

# One layer alone: attention whose best key takes nearly all of the weight; a state that forgets slowly.
ONLY_WINDOW = config(89, 36, 1e-5, [parallel(4, 2, 12, 14, 3.0, 48, 24, 2, 3)], (31, 3, 2))
ONLY_DELTA = config(89, 48, 1e-5, [delta(4, 2, 16, 24, 4, (6, 6))], (31, 3, 2))
ONLY_GLA = config(89, 48, 1e-5, [gla(3, 16, 24, 64.0, 6)])
# One expert a token: a near tie between the two best experts would show in full, so this one is compared in float32.
ONE_EXPERT = config(61, 32, 1e-5, [gla(2, 8, 8, 4.0, 3, moe(12, 6, 1))], (17, 5, 3))


def random_weights(raw: dict, seed: int) -> Dict[str, torch.Tensor]:
    """Checkpoint tensors by name, float32 with bfloat16-representable values.  Decays are spread from channels that
    forget within a few tokens to channels that remember hundreds.  Keys resemble queries: a first token's read-out is
    (q . k) v before its norm, whose sign rounding would decide if q . k were a sum of unrelated terms."""
    g = torch.Generator().manual_seed(seed)

    def normal(*shape, std=1.0, mean=0.0):
        return bf16_values(mean + std * torch.randn(tuple(shape), generator=g))

    w, width = {}, raw["width"]
    w["embed"] = normal(raw["vocab"], width)
    big = (raw.get("embedding") or {}).get("bigram")
    if big:
        w["bigram"] = normal(big["buckets"] + 1, width)
    w["final.norm"] = normal(width, std=0.2, mean=1.0)
    w["head"] = normal(raw["vocab"], width, std=width ** -0.5)
    wide = 2.0 * width ** -0.5
    for i, layer in enumerate(raw["layers"]):
        p, m = f"l{i}.mix.", layer["mixer"]
        w[f"l{i}.norm1"] = normal(width, std=0.3, mean=1.0)
        if layer["type"] == "channel_delta":
            H, G, d, dv = m["heads"], m["kv_heads"], m["dim"], m["vdim"]
            ra, rg = layer["_ranks"]
            for name, n in (("q", G * d), ("k", G * d), ("v", H * dv)):
                w[p + name] = normal(n, width, std=wide)
                w[p + name + ".conv"] = normal(n, m["conv"], std=0.6)
            for name in ("", ".conv"):
                w[p + "k" + name] = bf16_values(0.9 * w[p + "q" + name] + 0.4 * w[p + "k" + name])
            w[p + "b"] = normal(H, width, std=width ** -0.5)
            w[p + "A_log"] = normal(H, std=0.7)
            w[p + "a1"], w[p + "a2"] = normal(ra, width, std=width ** -0.5), normal(H * d, ra, std=ra ** -0.5)
            w[p + "dt_bias"] = normal(H * d, std=2.0, mean=-3.0)
            w[p + "g1"], w[p + "g2"] = normal(rg, width, std=width ** -0.5), normal(H * dv, rg, std=rg ** -0.5)
            w[p + "norm"] = normal(dv, std=0.3, mean=1.0)
            w[p + "o"] = normal(width, H * dv, std=(H * dv) ** -0.5)
        elif layer["type"] == "gla":
            H, d, dv = m["heads"], m["dim"], m["vdim"]
            (ra,) = layer["_ranks"]
            for name, n in (("q", H * d), ("k", H * d), ("v", H * dv), ("g", H * dv)):
                w[p + name] = normal(n, width, std=width ** -0.5)
            w[p + "k"] = bf16_values(0.9 * w[p + "q"] + 0.4 * w[p + "k"])
            w[p + "a1"], w[p + "a2"] = normal(ra, width, std=width ** -0.5), normal(H * d, ra, std=ra ** -0.5)
            w[p + "a2.b"] = normal(H * d, std=2.0, mean=1.0)
            w[p + "norm"] = normal(dv, std=0.3, mean=1.0)
            w[p + "o"] = normal(width, H * dv, std=(H * dv) ** -0.5)
        else:
            l, r = m["left"], m["right"]
            H, G, d, dv, n = l["heads"], l["kv_heads"], l["dim"], l["vdim"], r["width"]
            for name, rows in (("q", H * d), ("k", G * d), ("v", G * dv), ("g", H)):
                w[p + "left." + name] = normal(rows, width, std=wide if name in "qk" else width ** -0.5)
            w[p + "left.q.norm"], w[p + "left.k.norm"] = normal(H * d, std=0.3, mean=1.0), normal(G * d, std=0.3, mean=1.0)
            w[p + "left.o"] = normal(width, H * dv, std=(H * dv) ** -0.5)
            for name in ("y", "x"):
                w[p + "right." + name] = normal(n, width, std=width ** -0.5)
                w[p + "right." + name + ".b"] = normal(n, std=0.5)
            w[p + "right.conv"], w[p + "right.conv.b"] = normal(n, r["conv"], std=0.6), normal(n, std=0.3)
            size = n // r["blocks"]
            for name in ("ra", "ri"):
                w[p + "right." + name] = normal(r["blocks"], size, size, std=size ** -0.5)
                w[p + "right." + name + ".b"] = normal(r["blocks"], size, std=0.5)
            w[p + "right.lam"] = normal(n, std=2.0, mean=-4.0)
            w[p + "right.o"] = normal(width, n, std=n ** -0.5)
            w[p + "left.out"], w[p + "right.out"] = normal(width, std=0.3, mean=1.0), normal(width, std=0.3, mean=1.0)
        mlp = layer.get("mlp")
        if not mlp:
            continue
        f = f"l{i}.mlp."
        w[f"l{i}.norm2"] = normal(width, std=0.3, mean=1.0)
        if mlp["kind"] == "dense":
            w[f + "gate"], w[f + "up"] = normal(mlp["ff"], width, std=width ** -0.5), normal(mlp["ff"], width, std=width ** -0.5)
            w[f + "down"] = normal(width, mlp["ff"], std=mlp["ff"] ** -0.5)
        else:
            ff = mlp["expert"]["ff"]
            # a router whose logits lie far apart: close calls between experts are rare
            w[f + "router"] = normal(mlp["router"]["experts"], width, std=2.5 * width ** -0.5)
            for e in range(mlp["router"]["experts"]):
                w[f"{f}e{e}.gate"] = normal(ff, width, std=width ** -0.5)
                w[f"{f}e{e}.up"] = normal(ff, width, std=width ** -0.5)
                w[f"{f}e{e}.down"] = normal(width, ff, std=ff ** -0.5)
    return w


@contextlib.contextmanager
def one_thread():
    """The plain implementation is thousands of tiny operations: on a machine of many cores each of them costs more in
    waking threads than in arithmetic."""
    threads = torch.get_num_threads()
    torch.set_num_threads(1)
    try:
        yield
    finally:
        torch.set_num_threads(threads)


def oracle(raw: dict, weights: Dict[str, torch.Tensor], ids: Sequence[int]) -> np.ndarray:
    """The plain implementation's logits in float64, [T, vocab]."""
    with one_thread():
        return P.forward(raw, weights, list(ids), dtype=torch.float64).numpy()


CLOSE_CALL = 0.2        # router logits (which have a spread of two and a half); what a bfloat16 engine's rounding can move them by
AFTER_CLOSE_CALL = 2     # tokens that a short convolution and a state carry a close call on to, visibly


def oracle_and_close_calls(raw: dict, weights: Dict[str, torch.Tensor], ids: Sequence[int]):
    """The plain logits [T, vocab] and, per position, whether it or one of the few before it went through a close call: a
    token whose router chose within ``CLOSE_CALL`` of another expert may take the other one in bfloat16, which its own
    logits show, and those of the tokens after it whose convolutions and states carry on from there."""
    margins: List[torch.Tensor] = []
    with one_thread():
        logits = P.forward(raw, weights, list(ids), dtype=torch.float64, margins_out=margins).numpy()
    close = np.zeros(len(ids), dtype=bool)
    for m in margins:
        for t in np.nonzero((m < CLOSE_CALL).numpy())[0]:
            close[t:t + 1 + AFTER_CLOSE_CALL] = True
    return logits, close


def clear_weights(raw: dict, seed: int, ids: Sequence[int], tries: int = 12) -> Dict[str, torch.Tensor]:
    """Of ``tries`` random weight sets, the one with the fewest close calls of its routers on ``ids``."""
    best, fewest = None, 1 << 30
    for k in range(tries):
        w = random_weights(raw, seed + 1000 * k)
        margins: List[torch.Tensor] = []
        with one_thread():
            P.forward(raw, w, list(ids), dtype=torch.float64, margins_out=margins)
        n = sum(int((m < CLOSE_CALL).sum()) for m in margins)
        if n < fewest:
            best, fewest = w, n
        if n == 0:
            break
    return best


def check_clear(got: np.ndarray, want: np.ndarray, close: np.ndarray, dtype: str, what: str, tol: float = None) -> None:
    """``check`` on every position in float32.  In bfloat16, on the positions that no close call touches (the others must
    not be most of them), and one position in fifty (or one) may lie beyond the bound, though not beyond four times it: the
    norms on the outputs magnify the rounding of an output whose terms cancel.  The float32 run, which allows no exception,
    is the one that shows a wrong mechanism."""
    tol = TOL[dtype] if tol is None else tol
    if dtype == "bfloat16":
        assert len(close) < 16 or close.mean() < 0.6, f"{what}: too many close calls for the test to mean much"
        got, want = got[~close], want[~close]
        if not len(got):
            return
        bound = tol * max(1.0, float(np.abs(want).max()))
        err = np.abs(got.astype(np.float64) - want).max(axis=1)
        beyond = np.nonzero(err > bound)[0]
        if 0 < beyond.size <= max(1, len(err) // 50) and err.max() <= 4.0 * bound:
            keep = np.ones(len(err), dtype=bool)
            keep[beyond] = False
            got, want = got[keep], want[keep]
    check(got, want, dtype, what, tol)


TOL = {"float32": 3e-5, "bfloat16": 7e-2}      # of the logits' scale; bfloat16: five layers with norms on their outputs
# The one-layer attention model has scores of tens: q and k rounded to bfloat16 (2^-9 each) move such a score by a tenth,
# and so a key's weight by a tenth.  Its bfloat16 bound is that share of the logits' scale; its float32 bound is the
# common one, and that is the run which shows a wrong key.
SHARP_BF16_TOL = 0.15


def tolerance(name: str, dtype: str) -> float:
    return SHARP_BF16_TOL if (name == "window" and dtype == "bfloat16") else TOL[dtype]


def step_context(rows: Sequence[Tuple[int, int, int]], device="cuda") -> SimpleNamespace:
    """The index arrays of a step for kernels under test; rows: (state slot, tokens before this step, tokens)."""
    def i32(x):
        return torch.tensor(x, dtype=torch.int32, device=device)
    counts = [n for _, _, n in rows]
    starts = np.concatenate([[0], np.cumsum(counts)]).tolist()
    return SimpleNamespace(
        num_rows=len(rows), num_tokens=sum(counts), num_prefill=sum(n != 1 for n in counts), max_q_len=max(counts),
        row_of_token=i32([r for r, n in enumerate(counts) for _ in range(n)]), cu_q=i32(starts),
        prefix_len=i32([p for _, p, _ in rows]), state_slots=i32([s for s, _, _ in rows]),
        positions=i32([p + j for _, p, n in rows for j in range(n)]))
