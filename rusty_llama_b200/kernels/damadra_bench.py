"""Damadra beside Vezatar (the library's closest model in its feed-forwards: routed experts, results normed behind their sublayer, a
reader of an earlier layer's cache) and beside Llama (the closest in its attention: grouped-query softmax attention) at equal
sizes: prompt-step and decode-step throughput through the engine, and every kernel in which Damadra differs timed alone beside the
library's kernel that does the like work.

    python bench.py --design damadra [--design-sizes small,lite,wide]

Sizes resemble real models' layers (random weights, four layers: full attention + dense, windowed attention + experts, windowed
attention + dense, a reader of the first layer's keys and values + experts; the whole vocabulary).  Vezatar and Llama beside it have
the same width, layer count, dense feed-forward and vocabulary; Vezatar the same experts, Llama the same heads.  Every kernel's
fraction is what it must move (bytes, against the measured copy rate) or compute (flops, against the measured bfloat16 matrix rate),
whichever bound is the tighter one, divided by the time it took; a kernel and the like kernel beside it are timed the same way on
inputs of the same size.
"""

from __future__ import annotations

import math
from types import SimpleNamespace
from typing import Dict

import torch

from . import microbench as mb
from . import ops
from .design_bench import SIZES as VEZATAR_SIZES
from .design_bench import _frac, llama_config, step_times, vezatar_config
from .linear import linear

# Vezatar's sizes, and beside them: query heads, kv heads and their size, the window, the identities among the router's choices
SIZES = {
    "small": dict(VEZATAR_SIZES["small"], q_heads=16, kv_heads=4, hd=64, window=512, identity=8),
    "lite": dict(VEZATAR_SIZES["lite"], q_heads=16, kv_heads=4, hd=128, window=1024, identity=32),
    "wide": dict(VEZATAR_SIZES["wide"], q_heads=32, kv_heads=8, hd=128, window=1024, identity=16),
}
LAYERS = 4
BUCKETS = 32


def damadra_config(z: dict) -> dict:
    sizes = {"heads": z["q_heads"], "kv_heads": z["kv_heads"], "dim": z["hd"], "vdim": z["hd"], "scale": 1.0 / math.sqrt(z["hd"]), "bias_max": z["window"]}
    win = dict(sizes, mask={"size": z["window"]})
    full = dict(sizes, q_temp={"coef": 0.1, "every": 512})
    dense = {"kind": "dense", "ff": z["ff"]}
    moe = {"kind": "moe", "router": {"experts": z["experts"], "identity": z["identity"], "top": z["top"]}, "expert": {"ff": z["eff"]}}
    layers = [{"type": "attention_2", "mixer": full, "mlp": dense}, {"type": "attention", "mixer": win, "mlp": moe},
              {"type": "attention", "mixer": win, "mlp": dense}, {"type": "attention_2", "mixer": dict(full, kv_from=0), "mlp": moe}]
    return {"architecture": "Damadra", "vocab": z["vocab"], "width": z["width"], "norm": {"eps": 1e-5}, "embedding": {"scale": 1.0}, "residual_mult": 0.5,
            "layers": layers}


def like_llama(z: dict) -> dict:
    return dict(llama_config(z), num_attention_heads=z["q_heads"], num_key_value_heads=z["kv_heads"], head_dim=z["hd"])


def kernel_table(z: dict, T: int, batch: int, ctx: int, peaks: dict) -> Dict[str, dict]:
    """Each kernel alone, at a prompt step of T tokens (one sequence) and a decode step of `batch` sequences at `ctx`."""
    from ..parts.attention import chunked_attention_runner
    from ..parts.position import distance_buckets

    dev, bf = "cuda:0", torch.bfloat16
    d, H, K, hd, W = z["width"], z["q_heads"], z["kv_heads"], z["hd"], z["window"]
    out: Dict[str, dict] = {}
    it = dict(iters=10, warmup=2)

    def note(name, us, nbytes, flops, like=None):
        out[name] = {"us": round(us, 1), "frac": _frac(us, nbytes, flops, peaks)}
        if like:
            lname, lus, lbytes, lflops = like
            out[name]["like"] = {"kernel": lname, "us": round(lus, 1), "frac": _frac(lus, lbytes, lflops, peaks)}

    def timed(fn):
        return mb._time(lambda i: fn(), 1, **it)

    n_distances = len(distance_buckets(BUCKETS, W))
    bias = 0.5 * torch.randn(H, n_distances, device=dev)
    scale = 1.0 / math.sqrt(hd)
    for rows, n_seqs, pos0, tag in ((T, 1, 0, "prefill"), (batch, batch, ctx - 1, "decode")):
        per = rows // n_seqs
        prompt = rows > batch
        i32 = dict(dtype=torch.int32, device=dev)
        step = SimpleNamespace(tok_seq=torch.arange(n_seqs, **i32).repeat_interleave(per), tok_pos=(pos0 + torch.arange(per, **i32)).repeat(n_seqs),
                               seq_start=torch.arange(n_seqs + 1, **i32) * per, seq_pos0=torch.full((n_seqs,), pos0, **i32), max_q_len=per, n_seqs=n_seqs,
                               decode_only=not prompt)
        pages = (pos0 + per + 63) // 64
        # ---- a result's norm, the residual sum and the stream as it is
        nbytes = rows * d * (4 + 4 + 2 + 2)
        nv = min(mb._copies(nbytes), 8) if prompt else 1  # (several sets of rows, together larger than the L2)
        sets = [(torch.randn(rows, d, device=dev), torch.randn(rows, d, device=dev, dtype=bf)) for _ in range(nv)]
        w = torch.ones(d, device=dev)
        us_like = mb._time(lambda i: ops.normed_add_rmsnorm(sets[i][0], sets[i][1], w, 1e-5, w, 1e-5, bf), nv, **it)
        us = mb._time(lambda i: ops.normed_add_rmsnorm(sets[i][0], sets[i][1], w, 1e-5, None, 0.0, bf, plain_out=True), nv, **it)
        us_plain = mb._time(lambda i: ops.add_rmsnorm(sets[i][0], sets[i][1], w, 1e-5, bf), nv, **it)
        note(f"{tag}_norm_result_add", us, nbytes, 0, ("normed_add_rmsnorm of Vezatar", us_like, nbytes, 0))
        out[f"{tag}_norm_result_add"]["add_rmsnorm"] = {"us": round(us_plain, 1), "frac": _frac(us_plain, nbytes, 0, peaks)}
        del sets
        # ---- norms of queries and keys, temperature, cache write
        kp, vp = (torch.randn(n_seqs * pages, K, 64, hd, device=dev, dtype=bf) for _ in range(2))
        table = torch.randperm(n_seqs * pages, device=dev).to(torch.int32).view(n_seqs, pages).contiguous()
        args = (None, step.tok_pos, step.tok_seq, table, kp, vp, None, 1.0)
        wq, wk, wh = torch.ones(H * hd, device=dev), torch.ones(K * hd, device=dev), torch.ones(hd, device=dev)
        kv_rows, full_rows = torch.randn(rows, (H + K) * hd, device=dev, dtype=bf), torch.randn(rows, (H + 2 * K) * hd, device=dev, dtype=bf)
        q_rows = torch.randn(rows, H * hd, device=dev, dtype=bf)
        moved = rows * (2 * H + 4 * K) * hd * 2
        us_like = timed(lambda: ops.qkv_prep(full_rows, *args, H, K, hd, hd, 0, False, q_norm=wh, k_norm=wh, norm_eps=1e-5))
        us = timed(lambda: ops.qkv_prep(kv_rows, *args, H, K, hd, hd, 0, False, q_norm=wq, k_norm=wk, norm_eps=1e-5, norm_whole=True, v_from_k=True))
        note(f"{tag}_norm_all_heads_store", us, rows * (2 * H + 3 * K) * hd * 2, 0, ("qkv_prep of Tefavik", us_like, moved, 0))
        us = timed(lambda: ops.qkv_prep(full_rows, *args, H, K, hd, hd, 0, False, q_norm=wh, k_norm=wh, norm_eps=1e-5, temperature=(0.1, 512)))
        note(f"{tag}_norm_temperature_store", us, moved, 0, ("qkv_prep of Tefavik", us_like, moved, 0))
        us = timed(lambda: ops.qkv_prep(q_rows, None, step.tok_pos, step.tok_seq, None, None, None, None, 1.0, H, 0, hd, hd, 0, False, q_norm=wh, norm_eps=1e-5, temperature=(0.1, 512)))
        note(f"{tag}_reader_norm_temperature", us, rows * 2 * H * hd * 2, 0, ("qkv_prep of Tefavik", us_like, moved, 0))
        # ---- attention with a bias by distance, beside the same kernel without
        for window, what in ((W, "windowed"), (0, "full")):
            keys = sum(min(p + 1, window or p + 1) for p in range(pos0, pos0 + per)) * n_seqs
            seen = min(window or ctx, ctx) * n_seqs
            us = {}
            for b in (bias, None):
                us[b is not None] = timed(chunked_attention_runner(full_rows, kp, vp, table, step, H, K, hd, hd, scale, 0, 0.0, None, window=window, bias=b))
            nb, fl = (0, 4.0 * keys * H * hd) if prompt else (seen * K * 2 * hd * 2, 0)
            note(f"{tag}_{what}_attention", us[True], nb, fl, ("the same without a bias", us[False], nb, fl))
        # ---- keys half as long again as the values (sizes that the kernels pad)
        kd, vd = hd * 3 // 4, hd // 2
        kp2, vp2 = torch.randn(n_seqs * pages, K, 64, kd, device=dev, dtype=bf), torch.randn(n_seqs * pages, K, 64, vd, device=dev, dtype=bf)
        rows2 = torch.randn(rows, H * kd + K * (kd + vd), device=dev, dtype=bf)
        us = {}
        for b in (bias, None):
            us[b is not None] = timed(chunked_attention_runner(rows2, kp2, vp2, table, step, H, K, kd, vd, scale, 0, 0.0, None, bias=b))
        keys = sum(p + 1 for p in range(pos0, pos0 + per)) * n_seqs
        nb, fl = (0, 2.0 * keys * H * (kd + vd)) if prompt else (ctx * n_seqs * K * (kd + vd) * 2, 0)
        note(f"{tag}_unequal_attention", us[True], nb, fl, ("the same without a bias", us[False], nb, fl))
        # ---- experts
        E, I, top, eff = z["experts"], z["identity"], z["top"], z["eff"]
        x = torch.randn(rows, d, device=dev, dtype=bf)
        wr, corr = torch.randn(E + I, d, device=dev) / math.sqrt(d), torch.zeros(E + I, device=dev)
        wr16 = wr.to(bf)
        us = timed(lambda: ops.moe_choose(linear(x, wr16, out_dtype=torch.float32), corr, E + I, top))
        us_like = timed(lambda: ops.moe_router(x, wr[:E], corr[:E], E, top))
        note(f"{tag}_router", us, (E + I) * d * 2 + rows * d * 2, 0, ("moe_router (32-bit rows)", us_like, E * d * 4 + rows * d * 2, 0))
        tile_rows = 128 if rows * top >= 64 * E else 32
        ids, wts, _ = ops.moe_router(x, wr, corr, E + I, top)
        ids_l, wts_l, _ = ops.moe_router(x, wr[:E], corr[:E], E, top)
        us, us_like = timed(lambda: ops.moe_plan(ids, E, tile_rows)), timed(lambda: ops.moe_plan(ids_l, E, tile_rows))
        note(f"{tag}_plan", us, rows * top * 12, 0, ("moe_plan, experts only", us_like, rows * top * 12, 0))
        (order, place, tiles, mt), (order_l, place_l, tiles_l, mt_l) = ops.moe_plan(ids, E, tile_rows), ops.moe_plan(ids_l, E, tile_rows)
        n, n_l = int((ids < E).sum()), rows * top
        used, used_l = int(torch.unique(ids[ids < E]).numel()), int(torch.unique(ids_l).numel())
        wu, wg = (torch.randn(E, eff, d, device=dev, dtype=bf) * 0.02 for _ in range(2))
        wd = torch.randn(E, d, eff, device=dev, dtype=bf) * 0.02
        kw = dict(gather_div=top, tile_rows=tile_rows)
        up = lambda: ops.moe_gemm(x, wu, tiles, mt, rows * top, order=order, act="relu2", **kw)  # noqa: E731
        us = timed(up)
        us_like = timed(lambda: ops.moe_gemm(x, wg, tiles_l, mt_l, rows * top, order=order_l, w2=wu, **kw))
        note(f"{tag}_experts_up_relu2", us, (used * eff * d + rows * d + n * eff) * 2, 2.0 * n * eff * d,
             ("experts' gate and up of Vezatar", us_like, (2 * used_l * eff * d + rows * d + n_l * eff) * 2, 4.0 * n_l * eff * d))
        h, h_l = up(), torch.randn(n_l, eff, device=dev, dtype=bf)
        down = lambda: ops.moe_gemm(h, wd, tiles, mt, rows * top, out_dtype=torch.float32, tile_rows=tile_rows)  # noqa: E731
        us = timed(down)
        us_like = timed(lambda: ops.moe_gemm(h_l, wd, tiles_l, mt_l, rows * top, out_dtype=torch.float32, tile_rows=tile_rows))
        note(f"{tag}_experts_down", us, (used * eff * d + n * eff) * 2 + n * d * 4, 2.0 * n * eff * d,
             ("experts' down of Vezatar", us_like, (used_l * eff * d + n_l * eff) * 2 + n_l * d * 4, 2.0 * n_l * eff * d))
        y, y_l = down(), torch.randn(n_l, d, device=dev)
        us = timed(lambda: ops.moe_combine(y, place, wts, None, None, x=x))
        us_like = timed(lambda: ops.moe_combine(y_l, place_l, wts_l, None, None))
        note(f"{tag}_experts_sum", us, n * d * 4 + rows * d * 6, 0, ("moe_combine, experts only", us_like, n_l * d * 4 + rows * d * 4, 0))
    ops.tc_status_check()
    return out


def run(sizes, T: int, batch: int, ctx: int, steps: int, warmup: int, peaks: dict, kernels: bool = True) -> dict:
    result = {"design": "Damadra", "beside": "Vezatar (same experts) and Llama (same heads) at equal width, dense feed-forward, layers and vocabulary", "layers": LAYERS,
              "dtype": "bf16", "prompt_tokens": T, "decode_batch": batch, "decode_context": ctx, "peaks": peaks, "sizes": {}}
    for name in sizes:
        z = SIZES[name]
        row = {"config": z}
        for who, cfg in (("damadra", damadra_config(z)), ("vezatar", vezatar_config(z)), ("llama", like_llama(z))):
            t = step_times(cfg, T, batch, ctx, steps, warmup)
            row[who] = {
                "prefill_ms": round(t["prefill_ms"], 3), "prefill_tokens_per_s": round(T / t["prefill_ms"] * 1e3, 1),
                "decode_ms": round(t["decode_ms"], 4), "decode_tokens_per_s": round(batch / t["decode_ms"] * 1e3, 1),
            }
        if kernels:
            row["kernels"] = kernel_table(z, T, batch, ctx, peaks)
        result["sizes"][name] = row
    return result
