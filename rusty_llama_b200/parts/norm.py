"""RMSNorm, fused with the residual sum that precedes it, and the arrangement's way to have no norm there."""

from __future__ import annotations

from typing import Dict, Mapping, Optional

import torch

from ..errors import ConfigError
from ..kernels import ops
from .base import NORMS, Norm, ParamInfo, ResidualStream


@NORMS.register("rmsnorm")
class RMSNorm(Norm):
    """y = x / sqrt(mean(x^2) + eps) * weight (src/backend/cpu.rs:96-105).

    params: size, eps, name (optional: the tensor's name after the prefix, "weight" if absent), offset (optional, default 0:
    the stored tensor is the weight's distance from `offset`, y = ... * (offset + w); such a weight is kept in 32-bit whatever
    the run's type, since offset + w has more digits than w), float32 (optional bool: the weight is kept in 32-bit in every run,
    for designs whose norms are 32-bit arithmetic throughout), groups (optional, default 1: the row is cut into that many equal
    consecutive parts and each is divided by its own root mean square), factor (optional, default 1: a constant that the weight is
    multiplied by at load; such a weight is kept in 32-bit too).  tensor: <prefix>weight [size]."""

    def __init__(self, spec, runtime):
        super().__init__(spec, runtime)
        self.size = int(self._param("size"))
        self.eps = float(self._param("eps"))
        self.offset = float(spec.params.get("offset", 0.0))
        self.factor = float(spec.params.get("factor", 1.0))
        self.keep32 = bool(spec.params.get("float32", False)) or self.factor != 1.0
        self.tensor_name = self.prefix + str(spec.params.get("name", "weight"))
        self.groups = int(spec.params.get("groups", 1))
        if self.groups < 1 or self.size % self.groups:
            raise ConfigError(f"rmsnorm: {self.groups} groups do not divide a row of {self.size}")
        self.weight: Optional[torch.Tensor] = None

    def param_infos(self) -> Dict[str, ParamInfo]:
        if self.offset:
            return {self.tensor_name: ParamInfo((self.size,), "scalars", centre=0.0)}
        if self.keep32:
            return {self.tensor_name: ParamInfo((self.size,), "scalars", centre=1.0)}
        return {self.tensor_name: ParamInfo((self.size,), "vector")}

    def load(self, tensors: Mapping[str, torch.Tensor]) -> None:
        self.weight = tensors[self.tensor_name]
        if self.offset:
            self.weight = (self.weight.to(torch.float32) + self.offset).contiguous()
        if self.factor != 1.0:
            self.weight = self.weight * self.factor

    def rms_weight(self):
        return (self.weight, self.eps) if self.groups == 1 else None

    def forward(self, stream: ResidualStream, rows: Optional[torch.Tensor] = None) -> torch.Tensor:
        if self.groups > 1 and stream.pending_norm is not None:
            stream.flush()  # (the kernel that norms a result before it adds it norms whole rows)
        delta, delta_norm, gate = stream.take_pending()
        if gate is not None or self.groups > 1:
            return ops.gated_add_rmsnorm(stream.x, delta, gate, self.weight, self.eps, self.groups, stream.act_dtype, rows=rows, write_x=rows is None)
        if delta_norm is not None:
            return ops.normed_add_rmsnorm(
                stream.x, delta, delta_norm[0], delta_norm[1], self.weight, self.eps, stream.act_dtype, rows=rows, write_x=rows is None,
                delta_bias=delta_norm[2],
            )
        return ops.add_rmsnorm(
            stream.x, delta, self.weight, self.eps, stream.act_dtype, rows=rows, write_x=rows is None
        )


@NORMS.register("identity")
class NoNorm(Norm):
    """y = x in the activation type: for sublayers that read the stream as it is.  What is pending on the stream is added (through its
    own norm, if it has one) in the same pass.  No params, no tensors."""

    def forward(self, stream: ResidualStream, rows: Optional[torch.Tensor] = None) -> torch.Tensor:
        delta, delta_norm, gate = stream.take_pending()
        if gate is not None:
            stream.add(delta, gate=gate)
            stream.flush()
            delta = None
        if delta_norm is not None:
            return ops.normed_add_rmsnorm(stream.x, delta, delta_norm[0], delta_norm[1], None, 0.0, stream.act_dtype, rows=rows,
                                          write_x=rows is None, delta_bias=delta_norm[2], plain_out=True)
        return ops.add_rmsnorm(stream.x, delta, None, 0.0, stream.act_dtype, rows=rows, write_x=rows is None and delta is not None, plain_out=True)
