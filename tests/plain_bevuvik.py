"""A plain, slow Bevuvik: whole sequences on the CPU, one function per mechanism.

Written from the design's equations and nothing else; it shares no code with the package.  Everything is torch on
the CPU in ``dtype`` (float64 by default).  ``weights`` maps checkpoint tensor names to tensors, ``config`` is the
dict of a config.json.

    x = x0 = embed[token]
    before the first layer of every pass through the looped layers:   x <- loop.in [x; x0]
    per layer i:   h = R(x; norm1);   x <- x + m (mixer(h) + ff(h))        (one norm, both read it; m = residual_mult)
    logits = head R(x; final.norm)
"""
from __future__ import annotations

import math
from typing import Dict, List, Optional

import torch


# ------------------------------------------------------------------------------------------------ small pieces
def rms_norm(x: torch.Tensor, w: Optional[torch.Tensor], eps: float) -> torch.Tensor:
    """x / sqrt(mean(x^2) + eps) over the last axis, times w if there is one."""
    y = x / torch.sqrt((x * x).mean(-1, keepdim=True) + eps)
    return y if w is None else y * w


def unit(x: torch.Tensor, eps: float = 1e-6) -> torch.Tensor:
    """x / sqrt(sum x^2 + eps) over the last axis."""
    return x / torch.sqrt((x * x).sum(-1, keepdim=True) + eps)


def sigmoid(z: torch.Tensor) -> torch.Tensor:
    return 1.0 / (1.0 + torch.exp(-z))


def softplus(z: torch.Tensor) -> torch.Tensor:
    """log(1 + e^z), without overflow."""
    return torch.clamp(z, min=0.0) + torch.log1p(torch.exp(-z.abs()))


def silu(z: torch.Tensor) -> torch.Tensor:
    return z * sigmoid(z)


def causal_conv(x: torch.Tensor, w: torch.Tensor) -> torch.Tensor:
    """x [T, channels], w [channels, taps]: y[t] = sum_j w[:, j] x[t - taps + 1 + j], zeros before the start."""
    T, taps = x.shape[0], w.shape[1]
    padded = torch.cat([torch.zeros(taps - 1, x.shape[1], dtype=x.dtype), x])
    return sum(w[:, j] * padded[j:j + T] for j in range(taps))


# ------------------------------------------------------------------------------------------------ rotation
def frequencies(dims: int, base: float) -> torch.Tensor:
    return torch.tensor([base ** (-2.0 * i / dims) for i in range(dims // 2)], dtype=torch.float64)


def yarn(dims: int, base: float, scaling: Optional[dict]):
    """(frequencies, gain of cos and sin) with YaRN's blend of the plain and the divided frequencies."""
    f = frequencies(dims, base)
    if not scaling:
        return f, 1.0
    factor, original = scaling["factor"], scaling["original"]

    def where(turns):
        return dims * math.log(original / (2.0 * math.pi * turns)) / (2.0 * math.log(base))
    lo = max(math.floor(where(scaling["fast"])), 0)
    hi = min(math.ceil(where(scaling["slow"])), dims - 1)
    out = []
    for i in range(dims // 2):
        ramp = min(max((i - lo) / max(hi - lo, 0.001), 0.0), 1.0)
        out.append(f[i].item() / factor * ramp + f[i].item() * (1.0 - ramp))
    return torch.tensor(out, dtype=torch.float64), 0.1 * math.log(factor) + 1.0


def rotation(m: dict):
    """(frequencies, gain) of a mixer's rotation (none: no coordinate is turned)."""
    r = m.get("rot")
    return yarn(r["dims"], r["base"], r.get("scaling")) if r else (torch.zeros(0, dtype=torch.float64), 1.0)


def rotate(x: torch.Tensor, freq: torch.Tensor, gain: float, interleaved: bool) -> torch.Tensor:
    """x [T, heads, d] at positions 0..T-1: the first 2 len(freq) coordinates of every head are turned."""
    T, n = x.shape[0], len(freq)
    a = torch.arange(T, dtype=torch.float64)[:, None] * freq[None, :]
    c, s = (gain * torch.cos(a)).to(x.dtype)[:, None, :], (gain * torch.sin(a)).to(x.dtype)[:, None, :]
    out = x.clone()
    if interleaved:
        u, v = x[..., 0:2 * n:2], x[..., 1:2 * n:2]
        out[..., 0:2 * n:2], out[..., 1:2 * n:2] = u * c - v * s, v * c + u * s
    else:
        u, v = x[..., :n], x[..., n:2 * n]
        out[..., :n], out[..., n:2 * n] = u * c - v * s, v * c + u * s
    return out


# ------------------------------------------------------------------------------------------------ attention
def window_mask(T: int, size: Optional[int]) -> torch.Tensor:
    """[T, T] True where query i reads key j: 0 <= i - j < size (None: j <= i)."""
    back = torch.arange(T)[:, None] - torch.arange(T)[None, :]
    return (back >= 0) if size is None else (back >= 0) & (back < size)


def softmax_attention(q, k, v, scale: float, mask, softcap: Optional[float] = None) -> torch.Tensor:
    """q [T, H, d], k [T, G, d], v [T, G, dv]: query head h reads key/value head h // (H / G)."""
    rep = q.shape[1] // k.shape[1]
    s = torch.einsum("ihd,jhd->hij", q, k.repeat_interleave(rep, 1)) * scale
    if softcap:
        s = softcap * torch.tanh(s / softcap)
    s = s.masked_fill(~mask[None], float("-inf"))
    return torch.einsum("hij,jhd->ihd", torch.softmax(s, -1), v.repeat_interleave(rep, 1))


def diff_lambda(lq1, lk1, lq2, lk2, diff: float) -> torch.Tensor:
    return torch.exp((lq1 * lk1).sum()) - torch.exp((lq2 * lk2).sum()) + diff


def difference(a1: torch.Tensor, a2: torch.Tensor, lam, diff: float, eps: float) -> torch.Tensor:
    """a1 - lam a2 [T, H, dv], every head's vector divided by its root mean square, times (1 - diff)."""
    return rms_norm(a1 - lam * a2, None, eps) * (1.0 - diff)


def differential_attention(h: torch.Tensor, w: Dict[str, torch.Tensor], p: str, m: dict, eps: float) -> torch.Tensor:
    T = h.shape[0]
    H, G, d, dv = m["heads"], m["kv_heads"], m["dim"], m["vdim"]
    q = (h @ w[p + "q"].T + w[p + "q.b"]).reshape(T, H, 2, d)
    k = (h @ w[p + "k"].T + w[p + "k.b"]).reshape(T, G, 2, d)
    v = (h @ w[p + "v"].T + w[p + "v.b"]).reshape(T, G, dv)
    freq, gain = rotation(m)
    mask = window_mask(T, m["mask"]["size"] if m.get("mask") else None)
    a = [softmax_attention(rotate(q[:, :, i], freq, gain, True), rotate(k[:, :, i], freq, gain, True), v, m["scale"], mask)
         for i in range(2)]
    lam = diff_lambda(w[p + "lq1"], w[p + "lk1"], w[p + "lq2"], w[p + "lk2"], m["diff"])
    return difference(a[0], a[1], lam, m["diff"], eps).reshape(T, H * dv) @ w[p + "o"].T + w[p + "o.b"]


def capped_attention(h: torch.Tensor, w: Dict[str, torch.Tensor], p: str, m: dict) -> torch.Tensor:
    T = h.shape[0]
    H, G, d, dv = m["heads"], m["kv_heads"], m["dim"], m["vdim"]
    freq, _ = rotation(m)
    q = rotate((h @ w[p + "q"].T).reshape(T, H, d), freq, 1.0, False)
    k = rotate((h @ w[p + "k"].T).reshape(T, G, d), freq, 1.0, False)
    v = (h @ w[p + "v"].T).reshape(T, G, dv)
    a = softmax_attention(q, k, v, m["scale"], window_mask(T, None), m.get("softcap"))
    return a.reshape(T, H * dv) @ w[p + "o"].T


# ------------------------------------------------------------------------------------------------ the recurrence
def delta_scan(q: torch.Tensor, k: torch.Tensor, v: torch.Tensor, g: torch.Tensor, beta: torch.Tensor,
               start: Optional[torch.Tensor] = None):
    """Gated delta rule with one decay a head: q k [T, H, d], v [T, H, dv], g beta [T, H]; per head and token
    S <- g S;  u = beta (v - S^T k);  S <- S + k u^T;  o = S^T q.   Returns o [T, H, dv] and S [H, d, dv]."""
    T, H, d = q.shape
    S = torch.zeros(H, d, v.shape[2], dtype=q.dtype) if start is None else start.clone()
    out = []
    for t in range(T):
        S = g[t][:, None, None] * S
        u = beta[t][:, None] * (v[t] - torch.einsum("hdv,hd->hv", S, k[t]))
        S = S + k[t][:, :, None] * u[:, None, :]
        out.append(torch.einsum("hdv,hd->hv", S, q[t]))
    return torch.stack(out), S


def gated_delta(h: torch.Tensor, w: Dict[str, torch.Tensor], p: str, m: dict, eps: float) -> torch.Tensor:
    T = h.shape[0]
    H, G, d, dv = m["heads"], m["kv_heads"], m["dim"], m["vdim"]
    q, k, v = (silu(causal_conv(h @ w[p + n].T, w[p + n + ".conv"])) for n in ("q", "k", "v"))
    q = unit(q.reshape(T, G, d)) * d ** -0.5
    k = unit(k.reshape(T, G, d))
    beta = sigmoid(h @ w[p + "b"].T)
    g = torch.exp(-torch.exp(w[p + "A_log"]) * softplus(h @ w[p + "a"].T + w[p + "dt_bias"]))
    rep = H // G
    o, _ = delta_scan(q.repeat_interleave(rep, 1), k.repeat_interleave(rep, 1), v.reshape(T, H, dv), g, beta)
    o = rms_norm(o, w[p + "norm"], eps).reshape(T, H * dv)
    return (o * silu(h @ w[p + "g"].T)) @ w[p + "o"].T


def parallel(h: torch.Tensor, w: Dict[str, torch.Tensor], p: str, m: dict, eps: float) -> torch.Tensor:
    left = capped_attention(h, w, p + "left.", m["left"])
    right = gated_delta(h, w, p + "right.", m["right"], eps)
    return 0.5 * (rms_norm(left, w[p + "left.out"], eps) + rms_norm(right, w[p + "right.out"], eps))


MIXERS = {"attention": differential_attention, "parallel": parallel}


# ------------------------------------------------------------------------------------------------ feed-forward
def clamped_glu(gate: torch.Tensor, up: torch.Tensor, limit: float) -> torch.Tensor:
    g, u = torch.clamp(gate, max=limit), torch.clamp(up, min=-limit, max=limit)
    return g * sigmoid(1.702 * g) * (u + 1.0)


def dense_ff(h: torch.Tensor, w: Dict[str, torch.Tensor], p: str, limit: float) -> torch.Tensor:
    return clamped_glu(h @ w[p + "gate"].T, h @ w[p + "up"].T, limit) @ w[p + "down"].T


# ------------------------------------------------------------------------------------------------ the model
def layer_runs(config: dict) -> List[tuple]:
    """(layer, first of a pass) of every layer run, in order."""
    n = len(config["layers"])
    loop = config.get("loop") or {"start": n, "stop": n, "times": 1}
    runs = [(i, False) for i in range(loop["start"])]
    for _ in range(loop["times"]):
        runs += [(i, i == loop["start"]) for i in range(loop["start"], loop["stop"])]
    return runs + [(i, False) for i in range(loop["stop"], n)]


def forward(config: dict, weights: Dict[str, torch.Tensor], ids: List[int], dtype=torch.float64,
            layers_out: Optional[list] = None) -> torch.Tensor:
    """Logits [T, vocab] of one whole sequence.  ``layers_out`` receives x after every layer run."""
    w = {n: t.to(dtype) for n, t in weights.items()}
    eps, m = config["norm"]["eps"], config["residual_mult"]
    x0 = w["embed"][torch.tensor(ids)]
    x = x0
    for i, first in layer_runs(config):
        if first:
            x = torch.cat([x, x0], -1) @ w["loop.in"].T
        layer, p = config["layers"][i], f"l{i}."
        h = rms_norm(x, w[p + "norm1"], eps)
        y = MIXERS[layer["type"]](h, w, p + "mix.", layer["mixer"], eps)
        if layer.get("mlp"):
            y = y + dense_ff(h, w, p + "mlp.", layer["mlp"]["limit"])
        x = x + m * y
        if layers_out is not None:
            layers_out.append(x.clone())
    return rms_norm(x, w["final.norm"], eps) @ w["head"].T
