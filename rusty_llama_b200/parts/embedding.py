"""Token embedding and the classifier."""

from __future__ import annotations

from typing import Dict, Mapping, Optional

import torch

from ..kernels import ops
from ..kernels.linear import linear
from .base import EMBEDDINGS, HEADS, ParamInfo, Part, ResidualStream


@EMBEDDINGS.register("token_embedding")
class TokenEmbedding(Part):
    """x = E[token], a row copy (src/model.rs:1237-1242), widened to the 32-bit stream; times `scale` there if one is named.

    params: vocab_size, hidden_size, name (optional: the tensor's name after the prefix, "weight" if absent), scale (optional,
    default 1: a constant that the rows are multiplied by, in 32-bit).
    tensor: <prefix>weight [V, d]."""

    def __init__(self, spec, runtime):
        super().__init__(spec, runtime)
        self.vocab_size = int(self._param("vocab_size"))
        self.d = int(self._param("hidden_size"))
        self.tensor_name = self.prefix + str(spec.params.get("name", "weight"))
        self.scale = float(spec.params.get("scale", 1.0))
        self.weight: Optional[torch.Tensor] = None

    def param_infos(self) -> Dict[str, ParamInfo]:
        return {self.tensor_name: ParamInfo((self.vocab_size, self.d))}

    def load(self, tensors: Mapping[str, torch.Tensor]) -> None:
        self.weight = tensors[self.tensor_name]

    def forward(self, tokens: torch.Tensor) -> ResidualStream:
        return ResidualStream(ops.embed_gather(tokens, self.weight, scale=self.scale), self.rt.dtype)


@HEADS.register("linear_head")
class LinearHead(Part):
    """logits = W xn in 32-bit (src/model.rs:1366); `tied_to` names the embedding
    tensor that serves as W when the model has no classifier of its own (src/model.rs:469-473).

    params: vocab_size, hidden_size, tied_to (a tensor name or None), name (optional, as for the embedding), scale (optional,
    default 1: a constant factor on the logits), softcap (optional, 0: the cap c of z <- c tanh(z / c) on the scaled logits)."""

    def __init__(self, spec, runtime):
        super().__init__(spec, runtime)
        self.vocab_size = int(self._param("vocab_size"))
        self.d = int(self._param("hidden_size"))
        self.tied_to = self._param("tied_to")
        self.scale = float(spec.params.get("scale", 1.0))
        self.softcap = float(spec.params.get("softcap", 0.0) or 0.0)
        self.weight: Optional[torch.Tensor] = None

    def weight_name(self) -> str:
        return self.tied_to or (self.prefix + str(self.spec.params.get("name", "weight")))

    def param_infos(self) -> Dict[str, ParamInfo]:
        return {self.weight_name(): ParamInfo((self.vocab_size, self.d))}

    def load(self, tensors: Mapping[str, torch.Tensor]) -> None:
        self.weight = tensors[self.weight_name()]

    def forward(self, xn: torch.Tensor) -> torch.Tensor:
        logits = linear(xn, self.weight, out_dtype=torch.float32)
        if self.scale != 1.0 or self.softcap:
            ops.scale_softcap(logits, self.scale, self.softcap)
        return logits
