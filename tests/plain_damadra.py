"""A plain, slow implementation of the Damadra architecture in float64: whole sequences, no cache, no batching, one function
per mechanism.  It imports nothing from the package; the tests compare the library against it.

A model is (cfg, weights): cfg the parsed config.json (a dict), weights a dict name -> float64 torch tensor.
"""

from __future__ import annotations

import math
from fractions import Fraction

import torch

F64 = torch.float64


def rms(x: torch.Tensor, eps: float) -> torch.Tensor:
    """x divided by its root mean square over the last axis, eps inside the root."""
    return x / torch.sqrt((x * x).mean(dim=-1, keepdim=True) + eps)


def silu(z: torch.Tensor) -> torch.Tensor:
    return z / (1.0 + torch.exp(-z))


def squared_relu(z: torch.Tensor) -> torch.Tensor:
    return torch.where(z > 0, z * z, torch.zeros_like(z))


# ------------------------------------------------------------------ the distance bias
def distance_bucket(n: int, rows: int, far: float) -> int:
    """Which of `rows` table rows belongs to a distance of n tokens: one row per distance below rows / 2, then rows whose
    borders grow geometrically up to `far`, the last row for everything beyond.  In whole numbers: the k-th of the m growing
    rows starts at the first n with (n / half)^m >= (far / half)^k."""
    half = rows // 2
    if n < half:
        return n
    m = rows - half
    step, span = Fraction(n, half) ** m, Fraction(far) / half
    k = 0
    while k < m - 1 and step >= span ** (k + 1):
        k += 1
    return half + k


def bias_matrix(rel: torch.Tensor, far: float, T: int) -> torch.Tensor:
    """rel [rows, H] -> [H, T, T]: entry (h, i, j) is the bias of query i and key j (zero where j > i)."""
    rows = rel.shape[0]
    by_distance = rel[[distance_bucket(n, rows, far) for n in range(T)]]  # [T, H]
    gap = torch.arange(T)[:, None] - torch.arange(T)[None, :]
    return by_distance[gap.clamp(min=0)].permute(2, 0, 1) * (gap >= 0)


# ------------------------------------------------------------------ attention
def causal(T: int, window: int = 0) -> torch.Tensor:
    """[T, T]: row i sees column j; window 0: every j <= i, else the last `window` positions."""
    gap = torch.arange(T)[:, None] - torch.arange(T)[None, :]
    return (gap >= 0) & ((gap < window) if window else torch.ones(T, T, dtype=torch.bool))


def query_temperature(positions: torch.Tensor, coef: float, every: int) -> torch.Tensor:
    return 1.0 + coef * torch.log(torch.div(positions + 1, every, rounding_mode="floor").to(F64) + 1.0)


def softmax_attention(q, k, v, scale: float, bias, window: int):
    """q [T, H, dim], k [T, G, dim], v [T, G, vdim], bias [H, T, T] -> [T, H, vdim]."""
    T, H = q.shape[0], q.shape[1]
    rep = H // k.shape[1]
    k, v = k.repeat_interleave(rep, dim=1), v.repeat_interleave(rep, dim=1)
    s = torch.einsum("ihd,jhd->hij", q, k) * scale + bias
    s = s.masked_fill(~causal(T, window)[None], -math.inf)
    e = torch.exp(s - s.amax(dim=-1, keepdim=True))
    return torch.einsum("hij,jhv->ihv", e / e.sum(dim=-1, keepdim=True), v)


def windowed_queries_keys_values(h, W, p, m, eps):
    """The mixer with a window: queries and keys normed over all heads at once, the values are the keys before their norm."""
    T, H, G, dim = h.shape[0], m["heads"], m["kv_heads"], m["dim"]
    q, k = h @ W[p + "q"].T, h @ W[p + "k"].T
    v = k.view(T, G, dim)
    q, k = rms(q, eps) * W[p + "q.norm"], rms(k, eps) * W[p + "k.norm"]
    return q.view(T, H, dim), k.view(T, G, dim), v


def full_queries(h, W, p, m, eps):
    """The mixer without a window: every query head normed on its own, then the temperature of its position."""
    T = h.shape[0]
    q = rms((h @ W[p + "q"].T).view(T, m["heads"], m["dim"]), eps) * W[p + "q.norm"]
    t = query_temperature(torch.arange(T), m["q_temp"]["coef"], m["q_temp"]["every"])
    return q * t[:, None, None]


def full_keys_values(h, W, p, m, eps):
    T, G = h.shape[0], m["kv_heads"]
    k = rms((h @ W[p + "k"].T).view(T, G, m["dim"]), eps) * W[p + "k.norm"]
    return k, (h @ W[p + "v"].T).view(T, G, m["vdim"])


def attend(q, k, v, W, p, m):
    T = q.shape[0]
    bias = bias_matrix(W[p + "rel"], m["bias_max"], T)
    window = int((m.get("mask") or {}).get("size") or 0)
    return softmax_attention(q, k, v, m["scale"], bias, window).reshape(T, -1) @ W[p + "o"].T


# ------------------------------------------------------------------ feed-forward
def dense_ff(h, W, p):
    return (silu(h @ W[p + "gate"].T) * (h @ W[p + "up"].T)) @ W[p + "down"].T


def expert(h, W, p):
    return squared_relu(h @ W[p + "up"].T) @ W[p + "down"].T


def route(h, W, p, top: int):
    """(chosen [T, top], weights [T, top]): softmax over everything the router scores; the largest score + correction are
    chosen, their weights are their scores as they are."""
    z = h @ W[p + "router"].T
    e = torch.exp(z - z.amax(dim=-1, keepdim=True))
    s = e / e.sum(dim=-1, keepdim=True)
    chosen = torch.sort(s + W[p + "correction"], dim=-1, descending=True, stable=True).indices[:, :top]
    return chosen, torch.gather(s, 1, chosen)


def moe_ff(h, W, p, router):
    """The first `experts` router outputs are experts, the `identity` ones behind them hand the input on."""
    chosen, weights = route(h, W, p, router["top"])
    y = torch.zeros_like(h)
    for t in range(h.shape[0]):
        for e, w in zip(chosen[t].tolist(), weights[t]):
            y[t] += w * (expert(h[t : t + 1], W, f"{p}e{e}.")[0] if e < router["experts"] else h[t])
    return y


# ------------------------------------------------------------------ the model
def plain_streams(cfg, W, toks):
    """(logits [T, vocab], the stream after every layer [layers, T, width])."""
    eps, m_res = float(cfg["norm"]["eps"]), float(cfg["residual_mult"])
    x = W["embed"][torch.as_tensor(list(toks), dtype=torch.long)] * float(cfg["embedding"]["scale"])
    after, kept = [], {}
    for i, layer in enumerate(cfg["layers"]):
        p, m = f"l{i}.", layer["mixer"]
        if layer["type"] == "attention":
            q, k, v = windowed_queries_keys_values(x, W, p + "mix.", m, eps)
        else:
            assert layer["type"] == "attention_2"
            q = full_queries(x, W, p + "mix.", m, eps)
            src = m.get("kv_from")
            if src is None:
                kept[i] = full_keys_values(x, W, p + "mix.", m, eps)
                src = i
            k, v = kept[src]
        x = x + m_res * rms(attend(q, k, v, W, p + "mix.", m), eps) * W[p + "norm1"]
        mlp = layer.get("mlp")
        if mlp:
            y = dense_ff(x, W, p + "mlp.") if mlp["kind"] == "dense" else moe_ff(x, W, p + "mlp.", mlp["router"])
            x = x + m_res * rms(y, eps) * W[p + "norm2"]
        after.append(x)
    return (rms(x, eps) * W["final.norm"]) @ W["head"].T, torch.stack(after)


def plain_logits(cfg, W, toks):
    return plain_streams(cfg, W, toks)[0]
