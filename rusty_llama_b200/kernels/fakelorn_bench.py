"""Fakelorn beside Vezatar (the library's closest model: its latent attention with readers of an earlier layer's latents, its dense
and routed feed-forwards with a shared expert are two of Fakelorn's layer kinds) at equal sizes: prompt-step and decode-step
throughput through the engine, and every kernel that only Fakelorn uses timed alone beside the library's kernel that does the
like work.

    python bench.py --design fakelorn [--design-sizes small,lite,wide]

Sizes resemble real models' layers (random weights, four layers: latent attention + dense, differential attention in a window +
experts, state-space + dense, a reader of the first layer's latents + experts; the whole vocabulary).  Vezatar beside it has the same
width, latent attention (in all of its four layers), feed-forwards, layer count and vocabulary.  Every kernel's fraction is what it
must move (bytes, against the measured copy rate) or compute (flops, against the measured bfloat16 matrix rate), whichever bound is
the tighter one, divided by the time it took; a kernel and the like kernel beside it are timed the same way on inputs of the
same size (repeated calls, so inputs below the L2's size stay in it for both).
"""

from __future__ import annotations

import math
from types import SimpleNamespace
from typing import Dict

import torch

from . import microbench as mb
from . import ops
from .design_bench import SIZES as VEZATAR_SIZES
from .design_bench import _frac, step_times, vezatar_config

# Vezatar's sizes, and beside them: the differential attention's heads (two maps of 64 over values of 128) and window, the
# state-space layer's heads (64 values each: twice the width in all), state and groups, the queries' latent, the norms' parts
SIZES = {
    "small": dict(VEZATAR_SIZES["small"], a_heads=8, a_kv=2, window=512, s_heads=32, state=128, s_groups=2, q_rank=512, norm_groups=4),
    "lite": dict(VEZATAR_SIZES["lite"], a_heads=16, a_kv=4, window=1024, s_heads=64, state=128, s_groups=4, q_rank=1024, norm_groups=8),
    "wide": dict(VEZATAR_SIZES["wide"], a_heads=32, a_kv=8, window=1024, s_heads=128, state=128, s_groups=8, q_rank=1536, norm_groups=16),
}
LAYERS = 4
MAP_DIM, A_VDIM, S_VDIM, TAPS = 64, 128, 64, 4


def fakelorn_config(z: dict) -> dict:
    def latent(kv_from=None):
        m = {"heads": z["heads"], "dim": z["dim"], "rot_dim": z["rot"], "vdim": z["vdim"], "q_rank": z["q_rank"], "kv_rank": z["rank"],
             "rot": {"base": 10000.0, "dims": z["rot"]}, "scale": 1.0 / math.sqrt(z["dim"] + z["rot"])}
        if kv_from is not None:
            m["kv_from"] = kv_from
        return m

    attn = {"heads": z["a_heads"], "kv_heads": z["a_kv"], "dim": MAP_DIM, "vdim": A_VDIM, "scale": 1.0 / math.sqrt(MAP_DIM), "diff": 0.4, "mask": {"size": z["window"]}}
    ssm = {"heads": z["s_heads"], "vdim": S_VDIM, "state": z["state"], "groups": z["s_groups"], "conv": TAPS, "norm_groups": z["s_groups"]}
    dense = {"kind": "dense", "ff": z["ff"]}
    moe = {"kind": "moe", "router": {"experts": z["experts"], "top": z["top"]}, "expert": {"ff": z["eff"]}, "shared": {"ff": z["sff"]}}
    layers = [{"type": "latent_attention", "mixer": latent(), "mlp": dense}, {"type": "attention", "mixer": attn, "mlp": moe},
              {"type": "mamba2", "mixer": ssm, "mlp": dense}, {"type": "latent_attention", "mixer": latent(0), "mlp": moe}]
    return {"architecture": "Fakelorn", "vocab": z["vocab"], "width": z["width"], "norm": {"eps": 1e-6, "groups": z["norm_groups"]}, "logit_scale": 1.0,
            "logit_softcap": 30.0, "layers": layers}


def kernel_table(z: dict, T: int, batch: int, ctx: int, peaks: dict) -> Dict[str, dict]:
    """Each kernel of the design alone, at a prompt step of T tokens (one sequence) and a decode step of `batch` sequences at `ctx`."""
    from ..parts.attention import decode_splits

    dev, bf = "cuda:0", torch.bfloat16
    d, AH, AK, W = z["width"], z["a_heads"], z["a_kv"], z["window"]
    out: Dict[str, dict] = {}
    it = dict(iters=10, warmup=2)

    def note(name, us, nbytes, flops, like=None):
        out[name] = {"us": round(us, 1), "frac": _frac(us, nbytes, flops, peaks)}
        if like:
            lname, lus, lbytes, lflops = like
            out[name]["like"] = {"kernel": lname, "us": round(lus, 1), "frac": _frac(lus, lbytes, lflops, peaks)}

    def timed(fn):
        return mb._time(lambda i: fn(), 1, **it)

    for rows, n_seqs, pos0, tag in ((T, 1, 0, "prefill"), (batch, batch, ctx - 1, "decode")):
        per = rows // n_seqs
        prompt = rows > batch
        i32 = dict(dtype=torch.int32, device=dev)
        tok_seq = torch.arange(n_seqs, **i32).repeat_interleave(per)
        tok_pos = (pos0 + torch.arange(per, **i32)).repeat(n_seqs)
        seq_start = torch.arange(n_seqs + 1, **i32) * per
        seq_pos0 = torch.full((n_seqs,), pos0, **i32)
        seq_len = seq_pos0 + per
        slots = torch.arange(n_seqs, **i32)
        # ---- the gated result, the residual sum and the norm in parts
        nbytes = rows * d * (4 + 4 + 2 + 2)
        nv = min(mb._copies(nbytes), 8) if prompt else 1  # (several sets of rows, together larger than the L2)
        sets = [(torch.randn(rows, d, device=dev), torch.randn(rows, d, device=dev, dtype=bf), torch.randn(rows, d, device=dev, dtype=bf)) for _ in range(nv)]
        w, bias = torch.ones(d, device=dev), torch.zeros(d, device=dev)
        us_like = mb._time(lambda i: ops.add_rmsnorm(sets[i][0], sets[i][1], w, 1e-5, bf), nv, **it)
        us = mb._time(lambda i: ops.gated_add_rmsnorm(sets[i][0], sets[i][1], (sets[i][2], bias), w, 1e-5, z["norm_groups"], bf), nv, **it)
        del sets
        note(f"{tag}_gated_add_norm", us, nbytes + rows * d * 2, 0, ("add_rmsnorm", us_like, nbytes, 0))
        # ---- differential attention: store, the two maps' attention, their difference and its norm
        hd = 2 * MAP_DIM
        pages = (pos0 + per + 63) // 64
        kp, vp = (torch.randn(n_seqs * pages, AK, 64, hd, device=dev, dtype=bf) for _ in range(2))
        table = torch.randperm(n_seqs * pages, device=dev).to(torch.int32).view(n_seqs, pages).contiguous()
        qkv = torch.randn(rows, AH * hd + 2 * AK * hd, device=dev, dtype=bf)
        plain = torch.randn(rows, (AH + 2 * AK) * hd, device=dev, dtype=bf)  # as many heads of 128 with one map each
        keys = sum(min(p + 1, W) for p in range(pos0, pos0 + per)) * n_seqs
        seen = min(W, pos0 + per) * n_seqs
        scale = 1.0 / math.sqrt(MAP_DIM)
        if prompt:
            us = timed(lambda: ops.qkv_prep(qkv[:, AH * hd:], None, tok_pos, tok_seq, table, kp, vp, None, 1.0, 0, AK, hd, hd, 0, False))
            us_like = timed(lambda: ops.rope_kv_write(plain, tok_pos, tok_seq, table, kp, vp, None, AH, AK, hd, 0, False))
            note(f"{tag}_store_keys_values", us, rows * AK * hd * 8, 0, ("rope_kv_write without rotation", us_like, rows * AK * hd * 8, 0))
            us = timed(lambda: ops.flash_prefill_tc(qkv, kp, vp, table, seq_start, seq_pos0, per, 2 * AH, AK, hd, window=W, scale=scale, maps=2))
            us_like = timed(lambda: ops.flash_prefill_tc(plain, kp, vp, table, seq_start, seq_pos0, per, AH, AK, hd, window=W, scale=scale))
            us_full = timed(lambda: ops.flash_prefill_tc(plain, kp, vp, table, seq_start, seq_pos0, per, AH, AK, hd, scale=scale))
            note(f"{tag}_two_maps_attention", us, 0, 2.0 * keys * 2 * AH * (MAP_DIM + A_VDIM), ("flash_prefill_tc, same window", us_like, 0, 4.0 * keys * AH * hd))
            out[f"{tag}_two_maps_attention"]["plain_causal"] = {"us": round(us_full, 1), "frac": _frac(us_full, 0, 4.0 * AH * hd * T * (T + 1) / 2, peaks)}
            a = torch.randn(rows, 2 * AH * A_VDIM, device=dev, dtype=bf)
            us = timed(lambda: ops.map_combine(a, AH, A_VDIM, 0.4, 1e-6, 0.6))
            o32 = torch.randn(rows, AH * A_VDIM, device=dev)
            us_like = timed(lambda: ops.head_norm_gate(o32, AH, A_VDIM, None, 1e-6, plain[:, : AH * A_VDIM], ops.GATE_SIGMOID, bf))
            note(f"{tag}_combine_maps", us, rows * AH * A_VDIM * 6, 0, ("head_norm_gate", us_like, rows * AH * A_VDIM * 8, 0))
        else:
            n1, n2 = decode_splits(n_seqs, 2 * AH, AK, min(W, ctx), hd), decode_splits(n_seqs, AH, AK, min(W, ctx), hd)
            sc = torch.empty(max(ops.attn_decode_scratch_floats(n_seqs, 2 * AH, hd, n1), ops.attn_decode_scratch_floats(n_seqs, AH, hd, n2)), device=dev)
            us = timed(lambda: ops.attn_decode(qkv, kp, vp, table, seq_len, 2 * AH, AK, hd, n1, sc, window=W, scale=scale, impl="tma", fuse=2, pair=(0.4, 1e-6, 0.6)))
            us_like = timed(lambda: ops.attn_decode(plain, kp, vp, table, seq_len, AH, AK, hd, n2, sc, window=W, scale=scale, impl="tma", fuse=2))
            note(f"{tag}_two_maps_attention", us, seen * AK * 2 * hd * 2, 4.0 * keys * 2 * AH * hd, ("attn_decode, same window", us_like, seen * AK * 2 * hd * 2, 0))
        # ---- latent attention: what is new is the queries' latent; the attention kernels are Vezatar's
        H, dim, rot, vdim, rank, qr = z["heads"], z["dim"], z["rot"], z["vdim"], z["rank"], z["q_rank"]
        Dk = rank + rot
        lp = torch.randn(rows, qr + H * vdim + Dk, device=dev, dtype=bf)
        lpages = torch.zeros(n_seqs * pages, 1, 64, Dk, device=dev, dtype=bf)
        freq, wn, wq = torch.rand(rot // 2, device=dev), torch.ones(rank, device=dev), torch.ones(qr, device=dev)
        q = torch.randn(rows, H * (dim + rot), device=dev, dtype=bf)
        q_cat = torch.empty(rows, H, Dk, device=dev, dtype=bf)
        turn = (freq, rot // 2, 1.0, tok_pos, tok_seq, table, lpages)
        us1 = timed(lambda: ops.latent_prep(None, lp[:, qr + H * vdim:], wn, 1e-6, *turn, None, H, dim, rot, rank, False, q_latent=lp[:, :qr], q_norm=wq))
        us2 = timed(lambda: ops.latent_prep(q, None, None, 1e-6, *turn, q_cat, H, dim, rot, rank, False))
        us_like = timed(lambda: ops.latent_prep(q, lp[:, qr + H * vdim:], wn, 1e-6, *turn, q_cat, H, dim, rot, rank, True))
        b1, b2 = rows * (2 * qr + 2 * Dk) * 2, rows * 2 * H * rot * 2
        note(f"{tag}_latents_norm_rotate_store", us1, b1, 0, ("latent_prep of Vezatar (latent and queries in one)", us_like, rows * (2 * H * rot + 2 * Dk) * 2, 0))
        note(f"{tag}_queries_rotate", us2, b2, 0, ("latent_prep of Vezatar (latent and queries in one)", us_like, rows * (2 * H * rot + 2 * Dk) * 2, 0))
        # ---- state-space layer: convolution, step sizes and decays, recurrence, gate and norm
        SH, N, G, P = z["s_heads"], z["state"], z["s_groups"], S_VDIM
        inner, C = SH * P, SH * P + 2 * G * N
        proj = torch.randn(rows, inner + C + SH, device=dev, dtype=bf)
        wc, bc = torch.randn(TAPS, C, device=dev), torch.zeros(C, device=dev)
        rec = torch.zeros(n_seqs, TAPS - 1, C, device=dev)
        us = timed(lambda: ops.short_conv(proj[:, inner: inner + C], wc, rec, slots, seq_start, tok_seq, bias=bc, single=not prompt))
        us_like = timed(lambda: ops.short_conv(proj[:, inner: inner + C], wc, rec, slots, seq_start, tok_seq))
        note(f"{tag}_ssm_short_conv", us, rows * C * 4, 0, ("short_conv of Namalix", us_like, rows * C * 4, 0))
        conv = ops.short_conv(proj[:, inner: inner + C], wc, rec, slots, seq_start, tok_seq, bias=bc)
        a_log, dtb = torch.zeros(SH, device=dev), torch.zeros(SH, device=dev)
        us = timed(lambda: ops.ssm_gates(proj[:, inner + C:], a_log, dtb))
        us_like = timed(lambda: ops.gla_log_decay(proj[:, inner + C:], dtb, 8.0))
        note(f"{tag}_ssm_gates", us, rows * SH * 10, 0, ("gla_log_decay", us_like, rows * SH * 6, 0))
        log_a, dt = ops.ssm_gates(proj[:, inner + C:], a_log, dtb)
        xs, B, Cq = conv[:, :inner], conv[:, inner: inner + G * N], conv[:, inner + G * N:]
        st = torch.zeros(n_seqs, SH, N, P, device=dev)
        nbytes, flops = rows * (C * 2 + inner * 4) + 2 * st.numel() * 4, 4.0 * rows * SH * N * P
        # the like recurrences with as many heads, key and value sizes: keys of their own per head
        lq = torch.randn(rows, 2 * SH * N + SH * P, device=dev, dtype=bf)
        q1, k1, v1 = lq[:, : SH * N], lq[:, SH * N: 2 * SH * N], lq[:, 2 * SH * N:]
        lbytes = rows * (lq.shape[1] * 2 + inner * 4) + 2 * st.numel() * 4
        decay = torch.full((SH,), 0.99, device=dev)
        if prompt:
            scr = torch.empty(ops.scalar_decay_chunked_scratch_floats(n_seqs, per, SH, N, P), device=dev)
            us = timed(lambda: ops.scalar_decay_chunked(Cq, B, xs, log_a, dt, st, slots, seq_start, SH, N, P, per, scr, qk_heads=G))
            scr2 = torch.empty(max(ops.gated_attn_chunked_scratch_floats(n_seqs, per, SH, N, P), ops.decay_attn_chunked_scratch_floats(n_seqs, per, SH, N, P)), device=dev)
            us_like = timed(lambda: ops.decay_attn(q1, k1, v1, decay, st, slots, seq_start, SH, N, P, max_q_len=per, scratch=scr2))
            us_gated = timed(lambda: ops.gated_attn_chunked(q1, k1, v1, log_a, dt, st, slots, seq_start, SH, N, P, per, scr2))
        else:
            us = timed(lambda: ops.gated_attn(Cq, B, xs, log_a, dt, st, slots, seq_start, SH, N, P, qk_heads=G))
            us_like = timed(lambda: ops.decay_attn(q1, k1, v1, decay, st, slots, seq_start, SH, N, P))
            us_gated = timed(lambda: ops.gated_attn(q1, k1, v1, log_a, dt, st, slots, seq_start, SH, N, P))
        note(f"{tag}_ssm_recurrence", us, nbytes, flops, ("decay_attn", us_like, lbytes, flops))
        out[f"{tag}_ssm_recurrence"]["gated_attn"] = {"us": round(us_gated, 1), "frac": _frac(us_gated, lbytes, flops, peaks)}
        y, wi, D = torch.randn(rows, inner, device=dev), torch.ones(inner, device=dev), torch.ones(SH, device=dev)
        us = timed(lambda: ops.ssm_gate_norm(y, xs, D, proj[:, :inner], wi, 1e-6, G, bf))
        us_like = timed(lambda: ops.rms_gate(y, wi, 1e-6, proj[:, :inner], bf))
        note(f"{tag}_ssm_gate_norm", us, rows * inner * (4 + 2 + 2 + 2), 0, ("rms_gate", us_like, rows * inner * 8, 0))
        # ---- logits
        n_rows = 1 if prompt else rows
        lg = torch.randn(n_rows, z["vocab"], device=dev)
        us = timed(lambda: ops.scale_softcap(lg, 1.0, 30.0))
        note(f"{tag}_scale_cap_logits", us, lg.numel() * 8, 0)
    ops.tc_status_check()
    return out


def run(sizes, T: int, batch: int, ctx: int, steps: int, warmup: int, peaks: dict, kernels: bool = True) -> dict:
    result = {"design": "Fakelorn", "beside": "Vezatar at equal width, latent attention, feed-forwards, layers and vocabulary", "layers": LAYERS, "dtype": "bf16",
              "prompt_tokens": T, "decode_batch": batch, "decode_context": ctx, "peaks": peaks, "sizes": {}}
    for name in sizes:
        z = SIZES[name]
        row = {"config": z}
        for who, cfg in (("fakelorn", fakelorn_config(z)), ("vezatar", vezatar_config(z))):
            t = step_times(cfg, T, batch, ctx, steps, warmup)
            row[who] = {
                "prefill_ms": round(t["prefill_ms"], 3), "prefill_tokens_per_s": round(T / t["prefill_ms"] * 1e3, 1),
                "decode_ms": round(t["decode_ms"], 4), "decode_tokens_per_s": round(batch / t["decode_ms"] * 1e3, 1),
            }
        if kernels:
            row["kernels"] = kernel_table(z, T, batch, ctx, peaks)
        result["sizes"][name] = row
    return result
