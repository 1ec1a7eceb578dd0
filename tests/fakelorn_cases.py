"""Small Fakelorn configurations and random weights for the tests, made without the library.

Weights are drawn so that every mechanism matters (activations of order one, peaked scores, gates on both sides of one half,
lambdas away from the constant, decays from quick forgetting to almost none, norm weights away from one), rounded to bfloat16
and written with the third-party safetensors package."""

import json
import os

import numpy as np
import torch


def _attn(heads, kv_heads, dim, vdim, scale, diff, window):
    m = {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "scale": scale, "diff": diff}
    if window:
        m["mask"] = {"size": window}
    return {"type": "attention", "mixer": m}


def _ssm(heads, vdim, state, groups, conv, norm_groups):
    return {"type": "mamba2", "mixer": {"heads": heads, "vdim": vdim, "state": state, "groups": groups, "conv": conv, "norm_groups": norm_groups}}


def _latent(heads, dim, rot_dim, vdim, q_rank, kv_rank, scale, base, kv_from=None):
    m = {"heads": heads, "dim": dim, "rot_dim": rot_dim, "vdim": vdim, "q_rank": q_rank, "kv_rank": kv_rank, "scale": scale, "rot": {"base": base, "dims": rot_dim}}
    if kv_from is not None:
        m["kv_from"] = kv_from
    return {"type": "latent_attention", "mixer": m}


def _dense(ff):
    return {"kind": "dense", "ff": ff}


def _moe(experts, top, ff, shared=0):
    m = {"kind": "moe", "router": {"experts": experts, "top": top}, "expert": {"ff": ff}}
    if shared:
        m["shared"] = {"ff": shared}
    return m


def _model(vocab, width, eps, groups, scale, cap, layers):
    cfg = {"architecture": "Fakelorn", "vocab": vocab, "width": width, "norm": {"eps": eps, "groups": groups}, "logit_scale": scale, "layers": layers}
    if cap:
        cfg["logit_softcap"] = cap
    return cfg


def config_a():
    """Six layers that differ in everything: a state-space layer first, sizes that are no multiples of 8, 6 heads on 2 with a window
    of 33, an attention without a window, two latent layers with latents of their own and a reader of the first that is not
    its neighbour, layers without feed-forward, parts of a norm of 32 numbers, two of five experts and all of three."""
    return _model(131, 96, 1e-5, 3, 0.25, 5.0, [
        dict(_ssm(3, 20, 24, 1, 3, 5), mlp=_dense(100)),
        dict(_latent(3, 12, 8, 20, 28, 24, 0.3, 500.0), mlp=_moe(5, 2, 24, 36)),
        dict(_attn(6, 2, 10, 12, 0.35, 0.2, 33), mlp=None),
        dict(_latent(2, 20, 8, 12, 9, 40, 0.25, 10000.0), mlp=_dense(40)),
        dict(_latent(4, 16, 8, 12, 20, 24, 0.25, 500.0, kv_from=1), mlp=None),
        dict(_attn(2, 2, 8, 8, 0.5, 0.7, 0), mlp=_moe(3, 3, 16)),
    ])


def config_b():
    """A width that no 16-byte-row kernel takes (68), whole rows as the only part of a norm, single heads, a window of one token, a
    negative constant in the difference, convolutions of one and two taps, no unrotated query part, one expert of one, no cap."""
    return _model(77, 68, 1e-6, 1, 3.0, 0.0, [
        dict(_attn(1, 1, 12, 24, 0.4, -0.3, 1), mlp=_moe(1, 1, 30, 10)),
        dict(_latent(1, 0, 16, 8, 68, 12, 0.5, 100.0), mlp=None),
        dict(_ssm(1, 36, 40, 1, 1, 1), mlp=_dense(70)),
        dict(_ssm(2, 8, 12, 2, 2, 4), mlp=_moe(6, 3, 12, 20)),
        dict(_latent(3, 7, 16, 9, 10, 12, 0.4, 100.0, kv_from=1), mlp=_dense(33)),
    ])


def config_c():
    """Sizes that the tensor-core kernels take: maps of 32 and 64 with values of 64 and 128, windows of 64 and 70, a latent of 64 with 16
    rotated numbers, a state of 128 x 64 with four heads on two groups."""
    return _model(160, 128, 1e-6, 4, 0.9, 20.0, [
        dict(_attn(4, 2, 32, 64, 0.2, 0.35, 64), mlp=_dense(256)),
        dict(_ssm(4, 64, 128, 2, 4, 4), mlp=_moe(8, 3, 48, 64)),
        dict(_latent(4, 32, 16, 32, 64, 64, 0.15, 10000.0), mlp=_moe(4, 1, 128, 96)),
        dict(_attn(3, 1, 64, 128, 0.12, 0.5, 70), mlp=_dense(128)),
        dict(_latent(8, 16, 16, 64, 32, 64, 0.18, 10000.0, kv_from=2), mlp=_dense(64)),
    ])


def config_d():
    """Eight layers of larger and odd sizes in another order: maps of 24 with values of 40 (padded tiles), windows of 130 and 200, ten heads
    on five, two sources of latents with two readers, a latent of 128, a state of 48 x 40 with six heads on three groups behind
    five taps, one of 160 x 24 (beyond the tensor-core form), twelve experts of which three, all of four, one of three."""
    return _model(1000, 384, 1e-5, 6, 0.75, 30.0, [
        dict(_latent(5, 24, 32, 40, 72, 128, 0.13, 50000.0), mlp=_moe(6, 2, 96, 40)),
        dict(_attn(10, 5, 24, 40, 0.2, 0.25, 130), mlp=_dense(512)),
        dict(_latent(3, 48, 16, 24, 40, 96, 0.12, 1000.0), mlp=_moe(4, 4, 128, 72)),
        dict(_ssm(6, 40, 48, 3, 5, 2), mlp=None),
        dict(_latent(6, 16, 32, 56, 48, 128, 0.14, 50000.0, kv_from=0), mlp=_dense(200)),
        dict(_attn(4, 4, 16, 72, 0.25, 0.8, 200), mlp=_moe(12, 3, 64, 200)),
        dict(_ssm(2, 24, 160, 1, 4, 3), mlp=_moe(3, 1, 256)),
        dict(_latent(2, 32, 16, 16, 24, 96, 0.15, 1000.0, kv_from=2), mlp=_dense(96)),
    ])


CONFIGS = {"a": config_a, "b": config_b, "c": config_c, "d": config_d}


def tensor_shapes(cfg):
    d, V = cfg["width"], cfg["vocab"]
    out = {"embed": (V, d), "final.norm": (d,)}
    for i, layer in enumerate(cfg["layers"]):
        p, m = f"l{i}.", layer["mixer"]
        out[p + "norm1"], out[p + "rg1"], out[p + "rg1.b"] = (d,), (d, d), (d,)
        q = p + "mix."
        H, vd = m["heads"], m["vdim"]
        if layer["type"] == "attention":
            G, dim = m["kv_heads"], m["dim"]
            out[q + "q"], out[q + "k"], out[q + "v"] = (H * 2 * dim, d), (G * 2 * dim, d), (G * vd, d)
            for name in ("lq1", "lk1", "lq2", "lk2"):
                out[q + name] = (dim,)
        elif layer["type"] == "mamba2":
            channels = H * vd + 2 * m["groups"] * m["state"]
            out[q + "in"] = (H * vd + channels + H, d)
            out[q + "conv"], out[q + "conv.b"] = (channels, m["conv"]), (channels,)
            out[q + "dt_bias"] = out[q + "A_log"] = out[q + "D"] = (H,)
            out[q + "norm"] = (H * vd,)
        else:
            rank, rot = m["kv_rank"], m["rot_dim"]
            out[q + "dq"], out[q + "dq.norm"] = (m["q_rank"], d), (m["q_rank"],)
            out[q + "uq"] = (H * (m["dim"] + rot), m["q_rank"])
            if m.get("kv_from") is None:
                out[q + "dkv"], out[q + "dkv.norm"] = (rank + rot, d), (rank,)
            out[q + "uk"], out[q + "uv"], out[q + "g"] = (H * m["dim"], rank), (H * vd, rank), (H * vd, d)
        out[q + "o"] = (d, H * vd)
        mlp = layer["mlp"]
        if mlp is None:
            continue
        out[p + "norm2"], out[p + "rg2"], out[p + "rg2.b"] = (d,), (d, d), (d,)
        q = p + "mlp."
        blocks = [("", mlp["ff"])] if mlp["kind"] == "dense" else [(f"e{j}.", mlp["expert"]["ff"]) for j in range(mlp["router"]["experts"])]
        if mlp["kind"] == "moe":
            out[q + "router"] = (mlp["router"]["experts"], d)
            if mlp.get("shared"):
                blocks.append(("shared.", mlp["shared"]["ff"]))
        for b, ff in blocks:
            out[q + b + "gate"] = out[q + b + "up"] = (ff, d)
            out[q + b + "down"] = (d, ff)
    return out


def random_weights(cfg, seed):
    """name -> bfloat16 torch tensor."""
    rng = np.random.default_rng(seed)
    out = {}
    for name, shape in tensor_shapes(cfg).items():
        last = name.rsplit(".", 1)[-1]
        if last in ("norm1", "norm2", "norm"):
            t = 1.0 + 0.3 * rng.standard_normal(shape)
        elif last in ("lq1", "lk1", "lq2", "lk2"):
            t = 1.2 * rng.standard_normal(shape) / np.sqrt(shape[0])
        elif last == "conv":
            t = 0.6 * rng.standard_normal(shape)
        elif last == "b":
            t = 0.7 * rng.standard_normal(shape)
        elif last == "A_log":
            t = -1.0 + rng.standard_normal(shape)
        elif last in ("dt_bias", "D"):
            t = rng.standard_normal(shape)
        elif name == "embed":
            t = rng.standard_normal(shape)
        elif last in ("q", "k", "uq", "uk", "gate", "up", "router", "rg1", "rg2"):
            t = 1.5 * rng.standard_normal(shape) / np.sqrt(max(shape[-1], 1))  # peaked scores, gates on both sides
        else:
            t = (0.5 if last in ("o", "down") else 1.0) * rng.standard_normal(shape) / np.sqrt(shape[-1])
        out[name] = torch.from_numpy(np.asarray(t, dtype=np.float32)).to(torch.bfloat16)
    return out


def write_model(folder, cfg, weights):
    from safetensors.torch import save_file

    os.makedirs(folder, exist_ok=True)
    with open(os.path.join(folder, "config.json"), "w") as f:
        json.dump(cfg, f)
    save_file({k: v.contiguous() for k, v in weights.items()}, os.path.join(folder, "model.safetensors"))
    return str(folder)


def as_float64(weights):
    return {k: v.to(torch.float64) for k, v in weights.items()}
