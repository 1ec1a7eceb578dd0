"""Small Damadra configurations and random weights for the tests, made without the library.

Weights are drawn so that every mechanism matters (scores of a few units, biases of a unit or two that differ from bucket to bucket,
norm weights away from one, corrections that change the choice of experts; scores much larger than these would turn the rounding of
a bfloat16 run into other choices of keys), rounded to bfloat16 and written with the third-party
safetensors package.  How many rows a layer's bias table has is not in a configuration: `ROWS` names it per configuration."""

import json
import os

import numpy as np
import torch


def _win(heads, kv_heads, dim, scale, bias_max, window):
    return {"type": "attention", "mixer": {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": dim, "scale": scale, "bias_max": bias_max, "mask": {"size": window}}}


def _full(heads, kv_heads, dim, vdim, scale, bias_max, coef, every, kv_from=None):
    m = {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "scale": scale, "bias_max": bias_max, "q_temp": {"coef": coef, "every": every}}
    if kv_from is not None:
        m["kv_from"] = kv_from
    return {"type": "attention_2", "mixer": m}


def _dense(ff):
    return {"kind": "dense", "ff": ff}


def _moe(experts, identity, top, ff):
    return {"kind": "moe", "router": {"experts": experts, "identity": identity, "top": top}, "expert": {"ff": ff}}


def _model(vocab, width, eps, scale, mult, layers):
    return {"architecture": "Damadra", "vocab": vocab, "width": width, "norm": {"eps": eps}, "embedding": {"scale": scale}, "residual_mult": mult, "layers": layers}


def config_a():
    """Six layers that differ in everything: sizes that are no multiples of 8, 6 heads on 2 with a window of 33, a reader that is not its
    source's neighbour, layers without feed-forward, three of five experts and two identities, all three of one expert and two."""
    return _model(131, 96, 1e-5, 3.0, 0.7, [
        dict(_full(3, 1, 10, 12, 0.35, 50, 0.3, 7), mlp=_moe(5, 2, 3, 24)),
        dict(_win(6, 2, 12, 0.4, 29, 33), mlp=None),
        dict(_full(4, 2, 20, 6, 0.25, 90, 0.4, 16), mlp=_dense(100)),
        dict(_full(5, 1, 10, 12, 0.5, 21, -0.1, 40, kv_from=0), mlp=_moe(1, 2, 3, 30)),
        dict(_win(2, 2, 8, 0.6, 200, 90), mlp=_dense(40)),
        dict(_full(2, 2, 20, 6, 0.3, 64, 0.5, 100, kv_from=2), mlp=None),
    ])


def config_b():
    """A width that no 16-byte-row kernel takes (68), single heads, a window of one token, a table of two rows, a temperature that
    steps at every token and one that falls, factors of one, one expert of one, more identities than experts."""
    return _model(77, 68, 1e-6, 1.0, 1.0, [
        dict(_win(1, 1, 12, 0.8, 9, 1), mlp=_moe(1, 0, 1, 30)),
        dict(_full(1, 1, 16, 8, 0.7, 5, 0.2, 1), mlp=None),
        dict(_win(3, 1, 7, 1.0, 12, 5), mlp=_moe(2, 6, 4, 12)),
        dict(_full(3, 1, 16, 8, 0.5, 5, -0.2, 3, kv_from=1), mlp=_dense(33)),
    ])


def config_c():
    """Sizes that the tensor-core kernels take: heads of 64 and 128 on both kinds, windows of 64 and 70, a table whose borders are whole
    numbers (16 rows up to 128), a reader with another number of query heads."""
    return _model(160, 128, 1e-6, 8.0, 0.6, [
        dict(_win(4, 2, 64, 0.25, 128, 64), mlp=_dense(256)),
        dict(_full(4, 2, 64, 64, 0.25, 128, 0.5, 32), mlp=_moe(9, 5, 3, 48)),
        dict(_win(3, 1, 128, 0.18, 100, 70), mlp=_moe(4, 1, 1, 128)),
        dict(_full(2, 1, 128, 128, 0.2, 128, 0.3, 50), mlp=_dense(128)),
        dict(_full(8, 2, 64, 64, 0.3, 40, 0.1, 9, kv_from=1), mlp=_dense(64)),
    ])


def config_d():
    """Larger and odd sizes in another order: keys of 40, 96 and 72 beside values of 24, 64 and 72 (padded tiles), ten heads on five, windows
    of 130 and 200, tables of many rows, twelve experts and four identities of which three, four of four experts."""
    return _model(1000, 384, 1e-5, 5.0, 0.9, [
        dict(_full(5, 5, 96, 64, 0.12, 300, 0.4, 64), mlp=_dense(512)),
        dict(_win(10, 5, 40, 0.2, 150, 130), mlp=None),
        dict(_full(6, 3, 40, 24, 0.2, 180, 0.3, 20), mlp=_moe(4, 0, 4, 72)),
        dict(_full(10, 5, 96, 64, 0.15, 500, 0.2, 33, kv_from=0), mlp=_moe(12, 4, 3, 64)),
        dict(_win(4, 4, 72, 0.18, 90, 200), mlp=_moe(6, 3, 2, 96)),
        dict(_full(9, 3, 40, 24, 0.2, 70, 0.3, 50, kv_from=2), mlp=_dense(200)),
    ])


CONFIGS = {"a": config_a, "b": config_b, "c": config_c, "d": config_d}
# seeds with which the tests' sequences bring no close call between two experts among their first tokens (a bfloat16 run may then choose
# the other one, and with few keys to look at every later token sees the difference)
SEEDS = {"a": 211, "b": 213, "c": 207, "d": 212}
ROWS = {"a": [8, 12, 26, 6, 10, 20], "b": [4, 2, 6, 2], "c": [16, 16, 32, 24, 12], "d": [40, 64, 30, 48, 20, 32]}  # rows of each layer's table


def tensor_shapes(cfg, rows):
    d, V = cfg["width"], cfg["vocab"]
    out = {"embed": (V, d), "head": (V, d), "final.norm": (d,)}
    for i, layer in enumerate(cfg["layers"]):
        p, m = f"l{i}.", layer["mixer"]
        q = p + "mix."
        H, G, dim, vd = m["heads"], m["kv_heads"], m["dim"], m["vdim"]
        windowed = layer["type"] == "attention"
        out[p + "norm1"] = (d,)
        out[q + "q"], out[q + "q.norm"] = (H * dim, d), (H * dim if windowed else dim,)
        if m.get("kv_from") is None:
            out[q + "k"], out[q + "k.norm"] = (G * dim, d), (G * dim if windowed else dim,)
            if not windowed:
                out[q + "v"] = (G * vd, d)
        out[q + "rel"], out[q + "o"] = (rows[i], H), (d, H * vd)
        mlp = layer["mlp"]
        if mlp is None:
            continue
        out[p + "norm2"] = (d,)
        q = p + "mlp."
        if mlp["kind"] == "dense":
            out[q + "gate"] = out[q + "up"] = (mlp["ff"], d)
            out[q + "down"] = (d, mlp["ff"])
            continue
        r, ff = mlp["router"], mlp["expert"]["ff"]
        out[q + "router"], out[q + "correction"] = (r["experts"] + r["identity"], d), (r["experts"] + r["identity"],)
        for j in range(r["experts"]):
            out[f"{q}e{j}.up"], out[f"{q}e{j}.down"] = (ff, d), (d, ff)
    return out


def random_weights(cfg, rows, seed):
    """name -> bfloat16 torch tensor."""
    rng = np.random.default_rng(seed)
    out = {}
    for name, shape in tensor_shapes(cfg, rows).items():
        last = name.rsplit(".", 1)[-1]
        if last in ("norm1", "norm2", "norm"):
            t = 1.0 + 0.3 * rng.standard_normal(shape)
        elif last == "rel":
            t = 1.2 * rng.standard_normal(shape)
        elif last == "correction":
            t = 0.2 * rng.standard_normal(shape)
        elif last == "router":
            t = 2.0 * rng.standard_normal(shape) / np.sqrt(shape[-1])  # (the last expert chosen then has a small weight beside the first)
        elif name == "embed":
            t = rng.standard_normal(shape) / float(cfg["embedding"]["scale"])
        else:
            t = rng.standard_normal(shape) / np.sqrt(shape[-1])
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
