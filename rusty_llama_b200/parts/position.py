"""Position encodings that an attention mixer can own."""

from __future__ import annotations

import math
from typing import Dict, List, Mapping

import torch

from ..config.rope_scaling import RopeScaling, inverse_frequencies, magnitude
from ..errors import ConfigError
from ..kernels import ops
from .base import POSITIONS, ParamInfo, PositionEncoding


@POSITIONS.register("rotary")
class Rotary(PositionEncoding):
    """Rotary embedding: pair j of every q and k head is turned by pos * inv_freq[j]
    (src/backend/cpu.rs:306-361), the table computed once at load
    (src/config.rs:243-316).  Fused with the cache write in one kernel.

    params: rotary_dim, theta, scaling (RopeScaling), interleaved."""

    def __init__(self, spec, runtime):
        super().__init__(spec, runtime)
        self.rotary_dim = int(self._param("rotary_dim"))
        self.interleaved = bool(self._param("interleaved"))
        scaling = self._param("scaling")
        if not isinstance(scaling, RopeScaling):
            scaling = RopeScaling.from_json(scaling)
        table = inverse_frequencies(self.rotary_dim, float(self._param("theta")), scaling)
        self.inv_freq = torch.from_numpy(table).to(runtime.device)
        # what cosines and sines are multiplied by (other than 1 only with "yarn" scaling); a mixer that rotates with
        # kernels of its own reads it here
        self.magnitude = magnitude(scaling)

    def write_qk(self, qkv, step, kv, num_heads, num_kv_heads, head_dim, write_kv):
        if self.magnitude != 1.0:
            raise ConfigError("rotary: the fused rotation and cache write of grouped-query attention has no magnitude factor")
        ops.rope_kv_write(
            qkv, step.tok_pos, step.tok_seq,
            kv.block_table if write_kv else None, kv.k_pages if write_kv else None, kv.v_pages if write_kv else None,
            self.inv_freq, num_heads, num_kv_heads, head_dim, self.rotary_dim, self.interleaved, write_kv=write_kv,
        )

    def rotate(self, q, k, step):
        raise NotImplementedError("Rotary encodes positions inside write_qk")

    def decode_fusion(self):
        if self.magnitude != 1.0:
            return None
        if self.rotary_dim % 8:  # the fused kernel moves a pair's halves between lanes in steps of four values
            return None
        return self.inv_freq, self.rotary_dim, self.interleaved


@POSITIONS.register("none")
class NoPosition(PositionEncoding):
    """No position signal: keys and values are stored as they are."""

    def rotate(self, q, k, step):
        return None

    def decode_fusion(self):
        return None, 0, False


def distance_buckets(rows: int, max_distance: float) -> List[int]:
    """The table row of every distance 0, 1, ... up to the first that belongs to the last row (which then serves all larger ones):
    half of the rows have a distance each, the others m = rows - half have borders that grow geometrically from `half` to
    `max_distance`: row half + floor(m ln(n / half) / ln(max_distance / half)), at most rows - 1."""
    half = rows // 2
    if rows < 2 or max_distance <= half:
        raise ConfigError(f"distance bias: a table of {rows} rows cannot reach to a distance of {max_distance}")
    out = list(range(half))
    while out[-1:] != [rows - 1]:
        # (a border that is a whole number counts as reached although the quotient of two logarithms may round to just below it)
        at = math.log(len(out) / half) / math.log(max_distance / half) * (rows - half)
        out.append(min(rows - 1, half + math.floor(at + 1e-9)))
    return out


@POSITIONS.register("distance_bias")
class DistanceBias(PositionEncoding):
    """Queries and keys stay as they are; a learned number per head and bucket of the distance i - j is added to the score of query
    i and key j.  The checkpoint's table has a row per bucket (`distance_buckets`); it is laid out by distance at load.

    params: num_heads, max_distance (the distance from which on the last row holds), name (optional: the tensor's name after the
    prefix, "rel").  tensor: <prefix>rel [rows, H]."""

    def __init__(self, spec, runtime):
        super().__init__(spec, runtime)
        self.H = int(self._param("num_heads"))
        self.max_distance = float(self._param("max_distance"))
        self.tensor_name = self.prefix + str(spec.params.get("name", "rel"))
        self.table = None

    def param_infos(self) -> Dict[str, ParamInfo]:
        return {self.tensor_name: ParamInfo((-1, self.H), "scalars", centre=0.0, free=32)}

    def load(self, tensors: Mapping[str, torch.Tensor]) -> None:
        rel = tensors[self.tensor_name]
        buckets = torch.tensor(distance_buckets(rel.shape[0], self.max_distance), dtype=torch.long, device=rel.device)
        self.table = rel[buckets].t().contiguous()  # [H, distances]

    def score_bias(self):
        return self.table

    def rotate(self, q, k, step):
        return None
