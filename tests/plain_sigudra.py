"""A plain, slow Sigudra: whole sequences on the CPU, one function per mechanism.

Written from the design's equations and nothing else; it shares no code with the package.  Everything is torch on
the CPU in ``dtype`` (float64 by default).  ``weights`` maps checkpoint tensor names to tensors, ``config`` is the
dict of a config.json.

    x_t = embed[token_t] + bigram[row(token_(t-1), token_t)]
    per layer i:   x <- x + LN(mixer(x); norm1);   x <- x + LN(ff(x); norm2)  (if the layer has a feed-forward)
    logits = head LN(x; final.norm)
"""
from __future__ import annotations

import math
from typing import Dict, List, Optional

import torch


# ------------------------------------------------------------------------------------------------ small pieces
def layer_norm(x: torch.Tensor, w: torch.Tensor, eps: float) -> torch.Tensor:
    """(x - mean) / sqrt(mean((x - mean)^2) + eps) * w over the last axis; no bias."""
    c = x - x.mean(-1, keepdim=True)
    return c / torch.sqrt((c * c).mean(-1, keepdim=True) + eps) * w


def rms_norm(x: torch.Tensor, w: torch.Tensor, eps: float) -> torch.Tensor:
    return x / torch.sqrt((x * x).mean(-1, keepdim=True) + eps) * w


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


def gelu_tanh(z: torch.Tensor) -> torch.Tensor:
    return 0.5 * z * (1.0 + torch.tanh(math.sqrt(2.0 / math.pi) * (z + 0.044715 * z ** 3)))


def causal_conv(x: torch.Tensor, w: torch.Tensor) -> torch.Tensor:
    """x [T, channels], w [channels, taps]: y[t] = sum_j w[:, j] x[t - taps + 1 + j], zeros before the start."""
    T, taps = x.shape[0], w.shape[1]
    padded = torch.cat([torch.zeros(taps - 1, x.shape[1], dtype=x.dtype), x])
    return sum(w[:, j] * padded[j:j + T] for j in range(taps))


# ------------------------------------------------------------------------------------------------ embedding
def bigram_rows(ids: List[int], buckets: int, mul_prev: int, mul_cur: int) -> List[int]:
    """The row of the second table for every token: the first token of a sequence has the last row (``buckets``)."""
    return [buckets if t == 0 else (ids[t - 1] * mul_prev + ids[t] * mul_cur) % buckets for t in range(len(ids))]


# ------------------------------------------------------------------------------------------------ recurrences
def delta_scan(q: torch.Tensor, k: torch.Tensor, v: torch.Tensor, g: torch.Tensor, beta: torch.Tensor,
               start: Optional[torch.Tensor] = None):
    """Gated delta rule, q k g [T, H, d], v [T, H, dv], beta [T, H]; per head and token
    S <- diag(g) S;  u = beta (v - S^T k);  S <- S + k u^T;  o = S^T q.   Returns o [T, H, dv] and S [H, d, dv]."""
    T, H, d = q.shape
    S = torch.zeros(H, d, v.shape[2], dtype=q.dtype) if start is None else start.clone()
    out = []
    for t in range(T):
        S = g[t][:, :, None] * S
        u = beta[t][:, None] * (v[t] - torch.einsum("hdv,hd->hv", S, k[t]))
        S = S + k[t][:, :, None] * u[:, None, :]
        out.append(torch.einsum("hdv,hd->hv", S, q[t]))
    return torch.stack(out), S


def gla_scan(q: torch.Tensor, k: torch.Tensor, v: torch.Tensor, alpha: torch.Tensor,
             start: Optional[torch.Tensor] = None):
    """S <- diag(alpha) S + k v^T;  o = S^T q.  Shapes as in ``delta_scan``."""
    T, H, d = q.shape
    S = torch.zeros(H, d, v.shape[2], dtype=q.dtype) if start is None else start.clone()
    out = []
    for t in range(T):
        S = alpha[t][:, :, None] * S + k[t][:, :, None] * v[t][:, None, :]
        out.append(torch.einsum("hdv,hd->hv", S, q[t]))
    return torch.stack(out), S


def lru_scan(log_a: torch.Tensor, drive: torch.Tensor, start: Optional[torch.Tensor] = None) -> torch.Tensor:
    """S_t = a_t S_(t-1) + sqrt(1 - a_t^2) drive_t with a = exp(log_a), element by element; S of every token [T, width]."""
    S = torch.zeros(log_a.shape[1], dtype=log_a.dtype) if start is None else start.clone()
    out = []
    for t in range(log_a.shape[0]):
        S = torch.exp(log_a[t]) * S + torch.sqrt(-torch.expm1(2.0 * log_a[t])) * drive[t]
        out.append(S)
    return torch.stack(out)


# ------------------------------------------------------------------------------------------------ mixers
def channel_delta(h: torch.Tensor, w: Dict[str, torch.Tensor], p: str, m: dict, eps: float) -> torch.Tensor:
    T = h.shape[0]
    H, G, d, dv = m["heads"], m["kv_heads"], m["dim"], m["vdim"]
    q, k, v = (silu(causal_conv(h @ w[p + n].T, w[p + n + ".conv"])) for n in ("q", "k", "v"))
    q = unit(q.reshape(T, G, d)) * d ** -0.5
    k = unit(k.reshape(T, G, d))
    rep = H // G
    beta = sigmoid(h @ w[p + "b"].T)
    z = ((h @ w[p + "a1"].T) @ w[p + "a2"].T + w[p + "dt_bias"]).reshape(T, H, d)
    g = torch.exp(-torch.exp(w[p + "A_log"])[None, :, None] * softplus(z))
    o, _ = delta_scan(q.repeat_interleave(rep, 1), k.repeat_interleave(rep, 1), v.reshape(T, H, dv), g, beta)
    gate = sigmoid((h @ w[p + "g1"].T) @ w[p + "g2"].T).reshape(T, H, dv)
    return (rms_norm(o, w[p + "norm"], eps) * gate).reshape(T, H * dv) @ w[p + "o"].T


def gla(h: torch.Tensor, w: Dict[str, torch.Tensor], p: str, m: dict, eps: float) -> torch.Tensor:
    T = h.shape[0]
    H, d, dv = m["heads"], m["dim"], m["vdim"]
    q = (h @ w[p + "q"].T).reshape(T, H, d) * d ** -0.5
    k = (h @ w[p + "k"].T).reshape(T, H, d)
    v = (h @ w[p + "v"].T).reshape(T, H, dv)
    z = (h @ w[p + "a1"].T) @ w[p + "a2"].T + w[p + "a2.b"]
    alpha = torch.exp(-softplus(-z) / m["tau"]).reshape(T, H, d)              # sigmoid(z)^(1 / tau)
    o, _ = gla_scan(q, k, v, alpha)
    o = rms_norm(o, w[p + "norm"], eps).reshape(T, H * dv)
    return (o * silu(h @ w[p + "g"].T)) @ w[p + "o"].T


def window_mask(T: int, size: Optional[int]) -> torch.Tensor:
    """[T, T] True where query i reads key j: 0 <= i - j < size (None: j <= i)."""
    back = torch.arange(T)[:, None] - torch.arange(T)[None, :]
    return (back >= 0) if size is None else (back >= 0) & (back < size)


def softmax_attention(q: torch.Tensor, k: torch.Tensor, v: torch.Tensor, scale: float, mask: torch.Tensor) -> torch.Tensor:
    s = (torch.einsum("ihd,jhd->hij", q, k) * scale).masked_fill(~mask[None], float("-inf"))
    return torch.einsum("hij,jhd->ihd", torch.softmax(s, -1), v)


def window_attention(h: torch.Tensor, w: Dict[str, torch.Tensor], p: str, m: dict, eps: float) -> torch.Tensor:
    """Grouped-query attention: one RMS norm over all of q's rows (and one over k's) before the split into heads, no
    rotation, a window, one sigmoid gate a head."""
    T = h.shape[0]
    H, G, d, dv = m["heads"], m["kv_heads"], m["dim"], m["vdim"]
    q = rms_norm(h @ w[p + "q"].T, w[p + "q.norm"], eps).reshape(T, H, d)
    k = rms_norm(h @ w[p + "k"].T, w[p + "k.norm"], eps).reshape(T, G, d)
    v = (h @ w[p + "v"].T).reshape(T, G, dv)
    rep = H // G
    mask = window_mask(T, m["mask"]["size"] if m.get("mask") else None)
    o = softmax_attention(q, k.repeat_interleave(rep, 1), v.repeat_interleave(rep, 1), m["scale"], mask)
    o = o * sigmoid(h @ w[p + "g"].T)[:, :, None]
    return o.reshape(T, H * dv) @ w[p + "o"].T


def block_products(u: torch.Tensor, blocks: torch.Tensor, bias: torch.Tensor) -> torch.Tensor:
    """u [T, width] in equal parts, part b times the square matrix blocks[b] [out, in], plus bias[b]."""
    T = u.shape[0]
    n, size, _ = blocks.shape
    return (torch.einsum("tbi,boi->tbo", u.reshape(T, n, size), blocks) + bias).reshape(T, n * size)


def gated_recurrent_unit(h: torch.Tensor, w: Dict[str, torch.Tensor], p: str) -> torch.Tensor:
    y = gelu_tanh(h @ w[p + "y"].T + w[p + "y.b"])
    u = causal_conv(h @ w[p + "x"].T + w[p + "x.b"], w[p + "conv"]) + w[p + "conv.b"]
    r = sigmoid(block_products(u, w[p + "ra"], w[p + "ra.b"]))
    i = sigmoid(block_products(u, w[p + "ri"], w[p + "ri.b"]))
    S = lru_scan(-8.0 * r * softplus(w[p + "lam"]), i * u)
    return (S * y) @ w[p + "o"].T


def parallel(h: torch.Tensor, w: Dict[str, torch.Tensor], p: str, m: dict, eps: float) -> torch.Tensor:
    left = window_attention(h, w, p + "left.", m["left"], eps)
    right = gated_recurrent_unit(h, w, p + "right.")
    return 0.5 * (rms_norm(left, w[p + "left.out"], eps) + rms_norm(right, w[p + "right.out"], eps))


MIXERS = {"channel_delta": channel_delta, "gla": gla, "parallel": parallel}


# ------------------------------------------------------------------------------------------------ feed-forward
def dense_ff(h: torch.Tensor, w: Dict[str, torch.Tensor], p: str) -> torch.Tensor:
    return (gelu_tanh(h @ w[p + "gate"].T) * (h @ w[p + "up"].T)) @ w[p + "down"].T


def expert(h: torch.Tensor, w: Dict[str, torch.Tensor], p: str) -> torch.Tensor:
    return (silu(h @ w[p + "gate"].T) * (h @ w[p + "up"].T)) @ w[p + "down"].T


def experts_ff(h: torch.Tensor, w: Dict[str, torch.Tensor], p: str, mlp: dict, margins: Optional[list] = None) -> torch.Tensor:
    """The ``top`` experts with the largest sigmoid scores; the score multiplies the expert's INPUT."""
    top = mlp["router"]["top"]
    z = h @ w[p + "router"].T
    if margins is not None and top < z.shape[1]:
        ranked = z.sort(-1, descending=True).values
        margins.append(ranked[:, top - 1] - ranked[:, top])
    s = sigmoid(z)
    chosen = s.topk(top, -1).indices
    out = torch.zeros_like(h)
    for t in range(h.shape[0]):
        for e in chosen[t].tolist():
            out[t] += expert(s[t, e] * h[t:t + 1], w, f"{p}e{e}.")[0]
    return out


# ------------------------------------------------------------------------------------------------ the model
def forward(config: dict, weights: Dict[str, torch.Tensor], ids: List[int], dtype=torch.float64,
            layers_out: Optional[list] = None, margins_out: Optional[list] = None) -> torch.Tensor:
    """Logits [T, vocab] of one whole sequence.  ``layers_out`` receives x after every layer, ``margins_out`` every
    router's distance (in logits) between the last expert chosen and the first one left out [T]."""
    w = {n: (t if not t.is_floating_point() else t.to(dtype)) for n, t in weights.items()}
    eps = config["norm"]["eps"]
    x = w["embed"][torch.tensor(ids)]
    big = (config.get("embedding") or {}).get("bigram")
    if big:
        x = x + w["bigram"][torch.tensor(bigram_rows(list(ids), big["buckets"], big["mul_prev"], big["mul_cur"]))]
    for i, layer in enumerate(config["layers"]):
        p = f"l{i}."
        y = MIXERS[layer["type"]](x, w, p + "mix.", layer["mixer"], eps)
        x = x + layer_norm(y, w[p + "norm1"], eps)
        mlp = layer.get("mlp")
        if mlp:
            y = dense_ff(x, w, p + "mlp.") if mlp["kind"] == "dense" else experts_ff(x, w, p + "mlp.", mlp, margins_out)
            x = x + layer_norm(y, w[p + "norm2"], eps)
        if layers_out is not None:
            layers_out.append(x.clone())
    return layer_norm(x, w["final.norm"], eps) @ w["head"].T
