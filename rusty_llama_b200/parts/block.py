"""Arrangements of a layer's parts."""

from __future__ import annotations

import os

import torch

from ..kernels import ops
from ..kernels.linear import STREAM_MAX_ROWS, linear, linear_to_stream
from ..errors import ConfigError
from ..spec import PartSpec
from .base import BLOCKS, NORMS, Block, ParamInfo, ResidualStream


def _fold_enabled() -> bool:
    return os.environ.get("RL_FOLD_NORM", "1") != "0"


@BLOCKS.register("prenorm")
class PreNormBlock(Block):
    """x += mixer(norm_m(x)); x += feed_forward(norm_f(x)) (src/model.rs:1244-1357).

    Each sum is left pending on the stream and performed by the next norm's
    kernel, the following layer's or the model's final one.

    A decode step of up to 8 sequences in bfloat16 folds the second norm into the products around it where
    the parts allow it: if the mixer ends in a projection that it can leave to the caller, the norm is an RMSNorm
    and the feed-forward a gated one with fused weights, then the projection's kernel adds its sums to the stream
    itself, writes x * w beside it and leaves the rows' sums of squares, and the gate/up kernel multiplies its sums
    by the rows' 1 / sqrt(mean(x^2) + eps) before the activation: the norm's own kernel, with its pass over the
    stream, is not launched.  The parts are asked, not named: any mixer, norm or feed-forward that answers
    `forward_unprojected`, `rms_weight` and `gated_weights` takes part.  RL_FOLD_NORM=0 in the environment turns
    this off."""

    def forward(self, stream: ResidualStream, step, cache, shared_cache: bool = False) -> None:
        xn = self.norms["mixer"].forward(stream)
        if self._folded(stream, xn, step, cache, shared_cache):
            return
        stream.add_result(self.mixer.forward(xn, step, cache, shared_cache), bias=self.mixer.output_bias())
        if self.feed_forward is None:  # a layer may consist of its mixer alone
            return
        xn = self.norms["feed_forward"].forward(stream)
        stream.add(self.feed_forward.forward(xn, step))

    def _folded(self, stream: ResidualStream, xn, step, cache, shared_cache: bool) -> bool:
        if not (step.decode_only and self.rt.dtype == torch.bfloat16 and xn.shape[0] <= STREAM_MAX_ROWS and xn.is_cuda and _fold_enabled()):
            return False
        if self.feed_forward is None:
            return False
        norm, gated = self.norms["feed_forward"].rms_weight(), self.feed_forward.gated_weights()
        if norm is None or gated is None or self.mixer.output_bias() is not None:
            return False
        (w_norm, eps), (w_gate_up, w_down) = norm, gated
        d = stream.x.shape[1]
        if w_gate_up.dtype != torch.bfloat16 or w_gate_up.shape[1] != d or w_norm.shape[0] != d:
            return False
        unprojected = self.mixer.forward_unprojected(xn, step, cache, shared_cache)
        if unprojected is None:
            return False
        a, w_o = unprojected
        M, k = a.shape
        ok = (a.dtype == torch.bfloat16 and w_o.dtype == torch.bfloat16 and tuple(w_o.shape) == (d, k)
              and ops.gemv_stream_slices(M, k, 1) == 1 and ops.gemv_stream_slices(M, d, 1) == 1
              and not (a.stride(0) % 8 or w_o.stride(0) % 8 or w_gate_up.stride(0) % 8 or a.data_ptr() % 16))
        if not ok:
            # the attention has run; finish the layer the plain way
            stream.add(linear_to_stream(a, w_o))
            xn = self.norms["feed_forward"].forward(stream)
            stream.add(self.feed_forward.forward(xn, step))
            return True
        ws = self.rt.workspace
        xw = ws.get("fold_xw", M * d, torch.bfloat16)[: M * d].view(M, d)
        sumsq = ws.get("fold_sumsq", 8 * 1024, torch.float32)
        xw, sumsq, blocks = ops.gemv_stream_into_stream(a, w_o, stream.x, w_norm, xw=xw, sumsq=sumsq)
        h = ops.gemv_stream(xw, w_gate_up, torch.bfloat16, swiglu=True, row_scale=(sumsq, blocks, d, eps))
        stream.add(linear_to_stream(h, w_down))
        return True


@BLOCKS.register("sandwich")
class SandwichBlock(Block):
    """x += norm_mo(mixer(norm_m(x))); x += norm_fo(feed_forward(norm_f(x))): every sublayer has a norm before it and a
    norm of its own result.  norms: "mixer", "mixer_out", and with a feed-forward "feed_forward", "feed_forward_out".

    A sublayer's result stays pending on the stream together with the norm it has to go through; the kernel of the next
    norm (the next sublayer's, the next layer's or the model's final one) norms it, adds it and norms the sum, all in
    32-bit and in one pass.  The result norms must be RMS norms (`Norm.rms_weight`)."""

    def __init__(self, spec, runtime, mixer, feed_forward, norms):
        super().__init__(spec, runtime, mixer, feed_forward, norms)
        need = ["mixer", "mixer_out"] + (["feed_forward", "feed_forward_out"] if feed_forward is not None else [])
        for name in need:
            if name not in self.norms:
                raise ConfigError(f"sandwich block: no norm '{name}'")
        for name in need[1::2]:
            if self.norms[name].rms_weight() is None:
                raise ConfigError(f"sandwich block: norm '{name}' is not an RMS norm")

    def forward(self, stream: ResidualStream, step, cache, shared_cache: bool = False) -> None:
        xn = self.norms["mixer"].forward(stream)
        stream.add_result(self.mixer.forward(xn, step, cache, shared_cache), norm=self.norms["mixer_out"].rms_weight(), bias=self.mixer.output_bias())
        if self.feed_forward is None:
            return
        xn = self.norms["feed_forward"].forward(stream)
        stream.add(self.feed_forward.forward(xn, step), norm=self.norms["feed_forward_out"].rms_weight())


@BLOCKS.register("postnorm")
class PostNormBlock(Block):
    """x += norm_m(mixer(x)); x += norm_f(feed_forward(x)): the sublayers read the stream as it is and only their results are normed
    (a constant factor on a result is part of its norm's weight: `factor`).  norms: "mixer_out", and with a feed-forward
    "feed_forward_out", both RMS norms.

    A sublayer's result stays pending on the stream together with its norm; one pass then norms it, adds it and hands the sum on
    in the activation type."""

    def __init__(self, spec, runtime, mixer, feed_forward, norms):
        super().__init__(spec, runtime, mixer, feed_forward, norms)
        for name in ["mixer_out"] + (["feed_forward_out"] if feed_forward is not None else []):
            if name not in self.norms or self.norms[name].rms_weight() is None:
                raise ConfigError(f"postnorm block: no RMS norm '{name}'")
        self.read = NORMS.build(PartSpec("identity"), runtime)

    def forward(self, stream: ResidualStream, step, cache, shared_cache: bool = False) -> None:
        x = self.read.forward(stream)
        stream.add_result(self.mixer.forward(x, step, cache, shared_cache), norm=self.norms["mixer_out"].rms_weight(), bias=self.mixer.output_bias())
        if self.feed_forward is None:
            return
        x = self.read.forward(stream)
        stream.add(self.feed_forward.forward(x, step), norm=self.norms["feed_forward_out"].rms_weight())


@BLOCKS.register("shared_norm")
class SharedNormBlock(Block):
    """x += mixer(norm(x)) + feed_forward(norm(x)): one norm, and both sublayers read its output (the feed-forward may be absent).
    norms: "mixer".

    The mixer's result and the feed-forward's are two terms of the residual sum; both are 32-bit additions to the stream, the
    first by a pass of its own when the second is handed over, the second inside the next norm's kernel."""

    def forward(self, stream: ResidualStream, step, cache, shared_cache: bool = False) -> None:
        xn = self.norms["mixer"].forward(stream)
        stream.add_result(self.mixer.forward(xn, step, cache, shared_cache), bias=self.mixer.output_bias())
        if self.feed_forward is not None:
            stream.add(self.feed_forward.forward(xn, step))


@BLOCKS.register("gated_prenorm")
class GatedPreNormBlock(Block):
    """x += s(W_m h + b_m) * mixer(h), h = norm_m(x);  x += s(W_f h + b_f) * feed_forward(h), h = norm_f(x): every sublayer's result
    is multiplied element by element by the logistic function s of a linear map of the sublayer's input.  norms: "mixer", and with a
    feed-forward "feed_forward".

    A result stays pending on the stream together with its gate's pre-activation; the kernel of the next norm applies bias and
    logistic function, multiplies, adds and norms the sum, all in 32-bit and in one pass.

    params: hidden_size, names (the gates' tensors after the block's prefix, keys mixer feed_forward; a bias is its name + ".b").
    tensors: <prefix><name> [d, d], <prefix><name>.b [d]."""

    def __init__(self, spec, runtime, mixer, feed_forward, norms):
        super().__init__(spec, runtime, mixer, feed_forward, norms)
        self.d = int(self._param("hidden_size"))
        names = dict({"mixer": "gate_mixer", "feed_forward": "gate_feed_forward"}, **dict(spec.params.get("names", {})))
        self.gate_names = {k: self.prefix + names[k] for k in (["mixer"] + (["feed_forward"] if feed_forward is not None else []))}
        for k in self.gate_names:
            if k not in self.norms:
                raise ConfigError(f"gated_prenorm block: no norm '{k}'")
        self.gates = {}

    def param_infos(self):
        infos = {}
        for name in self.gate_names.values():
            infos[name] = ParamInfo((self.d, self.d))
            infos[name + ".b"] = ParamInfo((self.d,), "scalars", centre=0.0)
        return infos

    def load(self, tensors):
        self.gates = {k: (tensors[name].contiguous(), tensors[name + ".b"].contiguous()) for k, name in self.gate_names.items()}

    def _gate(self, which: str, h: torch.Tensor):
        w, b = self.gates[which]
        return linear(h, w), b

    def forward(self, stream: ResidualStream, step, cache, shared_cache: bool = False) -> None:
        h = self.norms["mixer"].forward(stream)
        gate = self._gate("mixer", h)
        if self.mixer.output_bias() is not None:
            raise ConfigError("gated_prenorm block: a mixer with an output bias is not built")
        stream.add_result(self.mixer.forward(h, step, cache, shared_cache), gate=gate)
        if self.feed_forward is None:
            return
        h = self.norms["feed_forward"].forward(stream)
        gate = self._gate("feed_forward", h)
        stream.add(self.feed_forward.forward(h, step), gate=gate)
