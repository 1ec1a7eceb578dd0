"""Attention whose heads are the difference of two softmax maps over the same values."""

from __future__ import annotations

import math
from typing import Dict, Mapping

import torch

from ..errors import ConfigError
from ..kernels import ops
from ..kernels.linear import linear, linear_to_stream
from ..spec import PartSpec
from .attention import _NAMES, _QKV_PARTIALS_MAX_ROWS, Attention, decode_splits
from .base import MIXERS, ParamInfo

_DIFF_NAMES = dict(_NAMES, lambda_q1="lq1", lambda_k1="lk1", lambda_q2="lq2", lambda_k2="lk2")


@MIXERS.register("differential_attention")
class DifferentialAttention(Attention):
    """Every query head has two queries and every kv head two keys of `map_dim` numbers, side by side as [map 1 | map 2], and one
    value of `value_dim` numbers:

        a1 = softmax(q1 . k1 * scale) v,   a2 = softmax(q2 . k2 * scale) v              (over the keys the window shows)
        lambda = exp(sum(lq1 lk1)) - exp(sum(lq2 lk2)) + diff                             (one number for the layer)
        o = a1 - lambda a2;   head = o / sqrt(mean(o^2) + eps) * (1 - diff)
        result = W_o concat_h(head)

    No position signal.  Query head h reads kv head h // (H / K).

    The two maps are 2 H query heads over K kv heads for the attention kernels (`maps`): the cache holds a kv head's two keys as one
    row of 2 map_dim numbers and its value once, and query heads 2h and 2h + 1 use a half each of head h's query row and of the
    keys.  In bfloat16 at 2 map_dim = value_dim = 64 or 128 a decode step runs on the TMA-fed decode kernel, which stores the new key
    and value itself, with the difference, the norm and the factor in the kernel that adds its key ranges up; prompts (and every
    other size and 32-bit runs) run the attention for the 2 H heads and `map_combine` behind it.

    params: hidden_size, num_heads, num_kv_heads, map_dim, value_dim, scale (default map_dim^-1/2), window (0 = all keys), diff, eps,
            names (tensor names after the prefix, keys q k v o lambda_q1 lambda_k1 lambda_q2 lambda_k2).
    tensors: <prefix>q [H 2 map_dim, d], k [K 2 map_dim, d], v [K value_dim, d], o [d, H value_dim], lq1, lk1, lq2, lk2 [map_dim]."""

    takes_out = False
    maps = 2

    def __init__(self, spec, runtime):
        dim = int(spec.params.get("map_dim", 0))
        if dim <= 0:
            raise ConfigError(f"differential_attention: map_dim {dim}")
        self.map_dim = dim
        self.out_heads = int(spec.params.get("num_heads", 0))
        params = {
            "hidden_size": spec.params.get("hidden_size"), "num_heads": 2 * self.out_heads, "num_kv_heads": spec.params.get("num_kv_heads"), "head_dim": 2 * dim,
            "value_dim": spec.params.get("value_dim"), "scale": float(spec.params.get("scale") or 1.0 / math.sqrt(dim)),
            "window": spec.params.get("window", 0), "position": PartSpec("none"),
        }
        if self.out_heads <= 0 or not params["num_kv_heads"] or self.out_heads % int(params["num_kv_heads"]):
            raise ConfigError(f"differential_attention: {self.out_heads} heads are not a multiple of {params['num_kv_heads']} kv heads")
        super().__init__(PartSpec(spec.kind, params, spec.prefix), runtime)
        self.names = dict(_DIFF_NAMES, **dict(spec.params.get("names", {})))
        self.diff, self.eps = float(spec.params.get("diff", 0.0)), float(spec.params.get("eps", 0.0))
        self.extended = True
        self.qd, self.od = self.out_heads * self.hd, self.out_heads * self.vd  # rows of W_q; numbers of a token's result
        self.lam = None
        # the decode kernel that stores the new key and value itself and combines the maps where it adds its key ranges up
        self.fused_decode = runtime.dtype == torch.bfloat16 and self.hd == self.vd and self.hd in ops.ATTN_DECODE_TMA_HEAD_DIMS

    def param_infos(self) -> Dict[str, ParamInfo]:
        p, n = self.prefix, self.names
        infos = {
            p + n["q"]: ParamInfo((self.qd, self.d)),
            p + n["k"]: ParamInfo((self.kvd, self.d)),
            p + n["v"]: ParamInfo((self.vvd, self.d)),
            p + n["o"]: ParamInfo((self.d, self.od)),
        }
        for key in ("lambda_q1", "lambda_k1", "lambda_q2", "lambda_k2"):
            infos[p + n[key]] = ParamInfo((self.map_dim,), "scalars", centre=0.0)
        return infos

    def load(self, tensors: Mapping[str, torch.Tensor]) -> None:
        p, n = self.prefix, self.names
        self.w_qkv = torch.cat([tensors[p + n["q"]], tensors[p + n["k"]], tensors[p + n["v"]]], dim=0).contiguous()
        self.w_o = tensors[p + n["o"]].contiguous()
        q1, k1, q2, k2 = (tensors[p + n[key]].to("cpu", torch.float64) for key in ("lambda_q1", "lambda_k1", "lambda_q2", "lambda_k2"))
        self.lam = float(torch.exp((q1 * k1).sum()) - torch.exp((q2 * k2).sum())) + self.diff

    def forward_unprojected(self, xn: torch.Tensor, step, cache, shared_cache: bool = False, out=None):
        if shared_cache:
            raise ConfigError("differential_attention: a layer that reads another layer's cache is not built")
        factor = 1.0 - self.diff
        if step.decode_only and self.fused_decode:
            qkv = linear_to_stream(xn, self.w_qkv) if xn.shape[0] <= _QKV_PARTIALS_MAX_ROWS else linear(xn, self.w_qkv)
            keys = min(self.window, step.plan_kv_len) if self.window else step.plan_kv_len
            n_splits = decode_splits(step.n_seqs, self.H, self.K, keys, self.hd)
            scratch = self.rt.workspace.get("attn_decode", ops.attn_decode_scratch_floats(step.n_seqs, self.H, self.hd, n_splits), torch.float32)
            a = ops.attn_decode(
                qkv, cache.k_pages, cache.v_pages, cache.block_table, step.seq_len, self.H, self.K, self.hd, n_splits, scratch,
                window=self.window, scale=self.scale, impl="tma", fuse=2, pair=(self.lam, self.eps, factor),
            )
            return a, self.w_o
        proj = linear(xn, self.w_qkv)
        ops.qkv_prep(proj[:, self.qd :], None, step.tok_pos, step.tok_seq, cache.block_table, cache.k_pages, cache.v_pages, None, 1.0, 0, self.K,
                     self.hd, self.vd, 0, False)
        a = self._attend(proj, None, step, cache, None)
        return ops.map_combine(a, self.out_heads, self.vd, self.lam, self.eps, factor), self.w_o
