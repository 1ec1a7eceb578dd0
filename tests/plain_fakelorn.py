"""A plain, slow implementation of the Fakelorn architecture in float64: whole sequences, no cache, no batching, one function
per mechanism.  It imports nothing from the package; the tests compare the library against it.

A model is (cfg, weights): cfg the parsed config.json (a dict), weights a dict name -> float64 torch tensor.
"""

from __future__ import annotations

import math

import torch

F64 = torch.float64


def rms(x: torch.Tensor, eps: float) -> torch.Tensor:
    """x divided by its root mean square over the last axis, eps inside the root."""
    return x / torch.sqrt((x * x).mean(dim=-1, keepdim=True) + eps)


def grouped_norm(x: torch.Tensor, w: torch.Tensor, groups: int, eps: float) -> torch.Tensor:
    """Every one of `groups` equal consecutive parts of a row divided by its own root mean square, the whole times w."""
    T, d = x.shape
    return rms(x.view(T, groups, d // groups), eps).reshape(T, d) * w


def logistic(z: torch.Tensor) -> torch.Tensor:
    return 1.0 / (1.0 + torch.exp(-z))


def silu(z: torch.Tensor) -> torch.Tensor:
    return z * logistic(z)


def softplus(z: torch.Tensor) -> torch.Tensor:
    return torch.maximum(z, torch.zeros_like(z)) + torch.log1p(torch.exp(-z.abs()))


def softmax_rows(s: torch.Tensor, visible: torch.Tensor) -> torch.Tensor:
    """Softmax over the last axis of the entries where `visible` is true, zero elsewhere."""
    s = s.masked_fill(~visible, -math.inf)
    e = torch.exp(s - s.amax(dim=-1, keepdim=True))
    return e / e.sum(dim=-1, keepdim=True)


def causal(T: int, window: int = 0) -> torch.Tensor:
    """[T, T]: row i sees column j; window 0: every j <= i, else the last `window` positions."""
    gap = torch.arange(T)[:, None] - torch.arange(T)[None, :]
    return (gap >= 0) & ((gap < window) if window else torch.ones(T, T, dtype=torch.bool))


# ------------------------------------------------------------------ rotation
def frequencies(base: float, dims: int) -> torch.Tensor:
    return base ** (-2.0 * torch.arange(dims // 2, dtype=F64) / dims)


def rotate_halves(x: torch.Tensor, positions: torch.Tensor, base: float, dims: int) -> torch.Tensor:
    """x [T, heads, n]; number i of the first `dims` is paired with i + dims / 2, the rest pass unchanged."""
    if not dims:
        return x
    a = positions.to(F64)[:, None] * frequencies(base, dims)[None, :]
    c, s = torch.cos(a)[:, None, :], torch.sin(a)[:, None, :]
    half = dims // 2
    u, v = x[..., :half], x[..., half:dims]
    return torch.cat([u * c - v * s, v * c + u * s, x[..., dims:]], dim=-1)


# ------------------------------------------------------------------ differential attention in a window
def lambda_of(W, p: str, diff: float) -> torch.Tensor:
    return torch.exp((W[p + "lq1"] * W[p + "lk1"]).sum()) - torch.exp((W[p + "lq2"] * W[p + "lk2"]).sum()) + diff


def differential_maps(q, k, v, scale: float, window: int):
    """q [T, H, 2, dim], k [T, G, 2, dim], v [T, G, vdim] -> the two maps' outputs, each [T, H, vdim]."""
    T, H = q.shape[0], q.shape[1]
    rep = H // k.shape[1]
    k, v = k.repeat_interleave(rep, dim=1), v.repeat_interleave(rep, dim=1)
    vis = causal(T, window)
    out = []
    for a in (0, 1):
        s = torch.einsum("ihd,jhd->hij", q[:, :, a], k[:, :, a]) * scale
        out.append(torch.einsum("hij,jhv->ihv", softmax_rows(s, vis[None]), v))
    return out


def combine_maps(a1, a2, lam, diff: float, eps: float):
    return rms(a1 - lam * a2, eps) * (1.0 - diff)


def attention_mixer(h, W, p, m, eps):
    T, H, G, dim, vdim = h.shape[0], m["heads"], m["kv_heads"], m["dim"], m["vdim"]
    q = (h @ W[p + "q"].T).view(T, H, 2, dim)
    k = (h @ W[p + "k"].T).view(T, G, 2, dim)
    v = (h @ W[p + "v"].T).view(T, G, vdim)
    mask = m.get("mask") or {}
    a1, a2 = differential_maps(q, k, v, m["scale"], int(mask.get("size") or 0))
    o = combine_maps(a1, a2, lambda_of(W, p, m["diff"]), m["diff"], eps)
    return o.reshape(T, H * vdim) @ W[p + "o"].T


# ------------------------------------------------------------------ state-space layer
def short_convolution(x: torch.Tensor, w: torch.Tensor, b: torch.Tensor) -> torch.Tensor:
    """x [T, C], w [C, taps] (last column the current token's), b [C]; zeros before the start."""
    T, taps = x.shape[0], w.shape[1]
    padded = torch.cat([torch.zeros(taps - 1, x.shape[1], dtype=F64), x])
    return sum(padded[i : i + T] * w[:, i] for i in range(taps)) + b


def ssm_recurrence(x, B, C, dt, log_rate, D):
    """x [T, H, vdim], B and C [T, G, N], dt [T, H] -> y [T, H, vdim]; S_t = exp(-exp(log_rate) dt_t) S_(t-1) + dt_t B_t x_t^T,
    y_t = S_t^T C_t + D x_t."""
    T, H, vdim = x.shape
    rep = H // B.shape[1]
    B, C = B.repeat_interleave(rep, dim=1), C.repeat_interleave(rep, dim=1)
    S = torch.zeros(H, B.shape[2], vdim, dtype=F64)
    y = []
    for t in range(T):
        a = torch.exp(-torch.exp(log_rate) * dt[t])
        S = a[:, None, None] * S + dt[t][:, None, None] * B[t][:, :, None] * x[t][:, None, :]
        y.append(torch.einsum("hn,hnv->hv", C[t], S) + D[:, None] * x[t])
    return torch.stack(y)


def gate_then_norm(y, z, w, groups: int, eps: float):
    return grouped_norm(y * silu(z), w, groups, eps)


def mamba2_mixer(h, W, p, m, eps):
    T, H, vdim, N, G = h.shape[0], m["heads"], m["vdim"], m["state"], m["groups"]
    inner = H * vdim
    proj = h @ W[p + "in"].T
    z, xbc, dt = proj[:, :inner], proj[:, inner : 2 * inner + 2 * G * N], proj[:, 2 * inner + 2 * G * N :]
    xbc = silu(short_convolution(xbc, W[p + "conv"], W[p + "conv.b"]))
    x = xbc[:, :inner].view(T, H, vdim)
    B = xbc[:, inner : inner + G * N].view(T, G, N)
    C = xbc[:, inner + G * N :].view(T, G, N)
    y = ssm_recurrence(x, B, C, softplus(dt + W[p + "dt_bias"]), W[p + "A_log"], W[p + "D"])
    return gate_then_norm(y.reshape(T, inner), z, W[p + "norm"], m["norm_groups"], eps) @ W[p + "o"].T


# ------------------------------------------------------------------ latent attention
def latent_rows(h, W, p, m, eps):
    """What a layer keeps per position: the normed latent [T, rank] and the turned shared key part [T, rot_dim]."""
    rank = m["kv_rank"]
    raw = h @ W[p + "dkv"].T
    c = rms(raw[:, :rank], eps) * W[p + "dkv.norm"]
    kr = rotate_halves(raw[:, None, rank:], torch.arange(h.shape[0]), m["rot"]["base"], m["rot"]["dims"])[:, 0]
    return c, kr


def latent_queries(h, W, p, m, eps):
    """(unrotated [T, H, dim], turned [T, H, rot_dim]), through the queries' own latent."""
    T, H, dim, rot = h.shape[0], m["heads"], m["dim"], m["rot_dim"]
    c_q = rms(h @ W[p + "dq"].T, eps) * W[p + "dq.norm"]
    q = (c_q @ W[p + "uq"].T).view(T, H, dim + rot)
    return q[..., :dim], rotate_halves(q[..., dim:], torch.arange(T), m["rot"]["base"], m["rot"]["dims"])


def latent_attention_mixer(h, W, p, m, eps, rows):
    T, H, dim, vdim = h.shape[0], m["heads"], m["dim"], m["vdim"]
    c, kr = rows
    qn, qr = latent_queries(h, W, p, m, eps)
    k = (c @ W[p + "uk"].T).view(T, H, dim)
    v = (c @ W[p + "uv"].T).view(T, H, vdim)
    s = (torch.einsum("ihd,jhd->hij", qn, k) + torch.einsum("ihd,jd->hij", qr, kr)) * m["scale"]
    o = torch.einsum("hij,jhv->ihv", softmax_rows(s, causal(T)[None]), v).reshape(T, H * vdim)
    return (o * logistic(h @ W[p + "g"].T)) @ W[p + "o"].T


# ------------------------------------------------------------------ feed-forward
def gated_ff(h, W, p):
    return (silu(h @ W[p + "gate"].T) * (h @ W[p + "up"].T)) @ W[p + "down"].T


def route(h, W, p, top: int):
    """(chosen [T, top], weights [T, top]): the largest logits, softmax over the chosen ones only."""
    z = h @ W[p + "router"].T
    best, chosen = torch.sort(z, dim=-1, descending=True, stable=True)
    e = torch.exp(best[:, :top] - best[:, :1])
    return chosen[:, :top], e / e.sum(dim=-1, keepdim=True)


def moe_ff(h, W, p, mlp):
    chosen, weights = route(h, W, p, mlp["router"]["top"])
    y = torch.zeros(h.shape[0], W[p + "e0.down"].shape[0], dtype=F64)
    for t in range(h.shape[0]):
        for e, w in zip(chosen[t].tolist(), weights[t]):
            y[t] += w * gated_ff(h[t : t + 1], W, f"{p}e{e}.")[0]
    return y + gated_ff(h, W, p + "shared.") if mlp.get("shared") else y


# ------------------------------------------------------------------ the model
def residual_gate(h, W, name: str):
    return logistic(h @ W[name].T + W[name + ".b"])


def cap_logits(z, scale: float, cap: float):
    z = z * scale
    return cap * torch.tanh(z / cap) if cap else z


def plain_streams(cfg, W, toks):
    """(logits [T, vocab], the stream after every layer [layers, T, width])."""
    eps, groups = float(cfg["norm"]["eps"]), int(cfg["norm"]["groups"])
    x = W["embed"][torch.as_tensor(list(toks), dtype=torch.long)].clone()
    after, rows = [], {}
    for i, layer in enumerate(cfg["layers"]):
        p, m = f"l{i}.", layer["mixer"]
        h = grouped_norm(x, W[p + "norm1"], groups, eps)
        if layer["type"] == "attention":
            y = attention_mixer(h, W, p + "mix.", m, eps)
        elif layer["type"] == "mamba2":
            y = mamba2_mixer(h, W, p + "mix.", m, eps)
        else:
            assert layer["type"] == "latent_attention"
            src = m.get("kv_from")
            if src is None:
                rows[i] = latent_rows(h, W, p + "mix.", m, eps)
                src = i
            y = latent_attention_mixer(h, W, p + "mix.", m, eps, rows[src])
        x = x + residual_gate(h, W, p + "rg1") * y
        mlp = layer.get("mlp")
        if mlp:
            h = grouped_norm(x, W[p + "norm2"], groups, eps)
            y = gated_ff(h, W, p + "mlp.") if mlp["kind"] == "dense" else moe_ff(h, W, p + "mlp.", mlp)
            x = x + residual_gate(h, W, p + "rg2") * y
        after.append(x)
    h = grouped_norm(x, W["final.norm"], groups, eps)
    return cap_logits(h @ W["embed"].T, float(cfg.get("logit_scale") or 1.0), float(cfg.get("logit_softcap") or 0.0)), torch.stack(after)


def plain_logits(cfg, W, toks):
    return plain_streams(cfg, W, toks)[0]
