"""The interfaces every part implements, and the registries that name them.

A model is put together from five families of parts:

  mixer          what mixes information across positions (attention here);
                 it may need cache storage and says so with `cache_need()`
  feed-forward   what acts on each position alone (a gated MLP here)
  norm           normalisation applied to the residual stream
  position       how positions reach the mixer (rotary here); owned by a mixer
  block          the arrangement of the above inside one layer (pre-norm here)

A part gets its sizes and constants from its `PartSpec.params` and nothing
else; no part knows which model it is in.  A new part is a subclass registered
under a new kind name; nothing in the library's files has to change for it.
The reference keeps the same seams as `Backend` trait methods
(src/backend/mod.rs:32-279) chosen by per-architecture predicates
(src/arch.rs:163-206).
"""

from __future__ import annotations

from dataclasses import dataclass
from typing import List, Callable, Dict, Mapping, Optional, Tuple

import torch

from ..errors import ConfigError
from ..spec import PartSpec


# --------------------------------------------------------------------------- runtime
class Workspace:
    """Scratch tensors that live across steps and grow on demand.

    Kernels that need global memory beyond their inputs and outputs (the split
    partials of decode attention, the probabilities of the sampler) take it
    from here, so that a replayed CUDA graph always sees the same addresses.  A tensor that
    has to grow is replaced, but the old one is kept for good: graphs captured while it was
    current still write to its address when they are replayed."""

    def __init__(self, device: torch.device):
        self.device = device
        self._bufs: Dict[str, torch.Tensor] = {}
        self._retired: List[torch.Tensor] = []

    def get(self, name: str, numel: int, dtype: torch.dtype, zeroed: bool = False) -> torch.Tensor:
        """zeroed: the tensor starts as zeros and its users leave it as zeros (counters that the
        kernels reset themselves); such a name must always be asked for with zeroed=True."""
        buf = self._bufs.get(name)
        if buf is None or buf.numel() < numel or buf.dtype != dtype:
            if self.device.type == "cuda" and torch.cuda.is_current_stream_capturing():
                raise RuntimeError(f"workspace '{name}' would have to grow during graph capture")
            if buf is not None:
                self._retired.append(buf)
            make = torch.zeros if zeroed else torch.empty
            buf = make(max(numel, 1), dtype=dtype, device=self.device)
            self._bufs[name] = buf
        return buf


@dataclass
class Runtime:
    """Where and in which precision a model runs.

    dtype: torch.bfloat16 (the serving path) or torch.float32 (everything in
    true 32-bit: no tensor-core product, no reduced-precision matrix mode)."""

    device: torch.device
    dtype: torch.dtype
    workspace: Workspace

    @classmethod
    def create(cls, device, dtype) -> "Runtime":
        device = torch.device(device)
        if isinstance(dtype, str):
            try:
                dtype = {"bfloat16": torch.bfloat16, "bf16": torch.bfloat16, "float32": torch.float32, "fp32": torch.float32}[dtype]
            except KeyError:
                raise ConfigError(f"dtype '{dtype}' is neither bfloat16 nor float32") from None
        if dtype not in (torch.bfloat16, torch.float32):
            raise ConfigError(f"dtype {dtype} is neither bfloat16 nor float32")
        return cls(device, dtype, Workspace(device))


# --------------------------------------------------------------------------- parameters
@dataclass(frozen=True)
class ParamInfo:
    """One tensor a part expects in the checkpoint.

    kind "matrix": stored in the run's matrix type (bfloat16, or float32 on the
    32-bit path).  kind "vector": a tensor stored in 32-bit stays so; otherwise
    it follows the run.  kind "scalars": a few learned numbers that enter 32-bit
    arithmetic directly (a softmax sink, a router's bias, a router's rows): always
    float32 at run time.  kind "table": integers, kept as int32.

    centre: what random weights of a "vector" are drawn around when a model is made from a seed (None: 1, the
    neutral value of a norm's weight; a norm that stores its weight's distance from one names 0)."""

    shape: Tuple[int, ...]
    kind: str = "matrix"
    centre: Optional[float] = None
    upper: Optional[int] = None  # of a "table" whose rows name different members of 0 .. upper - 1 (random models draw such rows)
    free: int = 0  # a -1 in `shape` is a size that only the checkpoint names (the part reads it at load); random models use `free`


def runtime_dtype(info: ParamInfo, stored: torch.dtype, run: torch.dtype) -> torch.dtype:
    if info.kind == "table":
        return torch.int32
    if info.kind == "scalars":
        return torch.float32
    if info.kind == "vector":
        return torch.float32 if (stored == torch.float32 or run == torch.float32) else run
    return run


# --------------------------------------------------------------------------- cache needs
@dataclass(frozen=True)
class KVNeed:
    """Keys and values of every position (window 0) or of the last `window` positions.

    values=False: the mixer keeps one row per position and head only (a latent from which it
    makes keys and values itself); the group then has no value pages.
    value_dim: the size of a value row where it differs from a key row's `head_dim` (None: the same).
    chunk: 0, or the size of the chunks (counted from position 0) outside of which no query reads: the pages that lie wholly before
    the chunk of the next position are given back."""

    num_kv_heads: int
    head_dim: int
    window: int = 0
    dtype: Optional[torch.dtype] = None  # None: the run's activation type
    values: bool = True
    value_dim: Optional[int] = None
    chunk: int = 0


@dataclass(frozen=True)
class StateNeed:
    """A record of fixed shape per sequence, zero when the sequence starts."""

    shape: Tuple[int, ...]
    dtype: torch.dtype = torch.float32


# --------------------------------------------------------------------------- part base classes
class Part:
    def __init__(self, spec: PartSpec, runtime: Runtime):
        self.spec = spec
        self.rt = runtime
        self.prefix = spec.prefix

    def param_infos(self) -> Dict[str, ParamInfo]:
        """Full checkpoint names of this part's tensors and what they must look like."""
        return {}

    def load(self, tensors: Mapping[str, torch.Tensor]) -> None:
        """Receive the tensors named by `param_infos`, already on the device in their run types."""

    def children(self) -> Tuple["Part", ...]:
        """Parts that this part owns (an attention mixer's position encoding, extra norms): the model
        asks them for their tensors and loads them like its own parts."""
        return ()

    def _param(self, key: str):
        try:
            return self.spec.params[key]
        except KeyError:
            raise ConfigError(f"part '{self.spec.kind}' (prefix '{self.prefix}') lacks parameter '{key}'") from None


class NormedTerms(list):
    """What a mixer returns when its result is a sum of terms that each go through an RMS norm of their own:
    a list of (delta, (weight, eps)), delta as `Mixer.forward` describes it; the result is sum_i rmsnorm(delta_i) * weight_i.
    Constant factors of the terms are part of their weights."""


class ResidualStream:
    """The 32-bit residual stream x[T, d] plus what was returned last and not yet added.

    A mixer or feed-forward hands back `delta` ([T, d] or [parts, T, d] partial
    sums, in the activation type).  It is added when the next norm runs, inside
    the norm's kernel, or by `flush()`."""

    def __init__(self, x: torch.Tensor, act_dtype: torch.dtype):
        self.x = x
        self.act_dtype = act_dtype
        self.pending: Optional[torch.Tensor] = None
        # (weight, eps, bias) of an RMSNorm that what is pending goes through before it is added (a layer that
        # norms its sublayers' results); None: it is added as it is
        self.pending_norm = None
        # (z [T, d], bias float32 [d]): what is pending is multiplied by the logistic function of z + bias before it is added
        self.pending_gate = None

    def add(self, delta: torch.Tensor, norm=None, bias: Optional[torch.Tensor] = None, gate=None) -> None:
        """norm: None, or (weight, eps): the stream receives rmsnorm(delta) * weight instead of delta.
        gate: None, or (z, gate_bias): the stream receives delta * logistic(z + gate_bias), element by element.
        bias: None, or a float32 row [d] that belongs to every row of delta (the bias of the projection that made it); the
        kernel that norms delta adds it first, so it needs a norm."""
        if self.pending is not None:
            self.flush()
        if bias is not None and norm is None:
            raise ConfigError("a sublayer's result with a bias row can only be added through a norm of that result")
        if gate is not None and norm is not None:
            raise ConfigError("a sublayer's result goes through a norm of its own or through a gate, not both")
        self.pending = delta
        self.pending_norm = None if norm is None else (norm[0], norm[1], bias)
        self.pending_gate = gate

    def add_result(self, result, norm=None, bias: Optional[torch.Tensor] = None, gate=None) -> None:
        """`add` for what a sublayer returned: a tensor, or `NormedTerms`, whose terms are added one after the other (each but the
        last by a pass of its own; the last stays pending for the next norm's kernel)."""
        if isinstance(result, NormedTerms):
            if norm is not None or bias is not None or gate is not None:
                raise ConfigError("a sublayer's result that is a sum of normed terms takes no further norm, gate or bias row")
            for delta, term_norm in result:
                self.add(delta, norm=term_norm)
        else:
            self.add(result, norm=norm, bias=bias, gate=gate)

    def take_pending(self):
        """(delta, norm, gate) of what is pending, which is the caller's to add from now on."""
        out = (self.pending, self.pending_norm, self.pending_gate)
        self.pending = self.pending_norm = self.pending_gate = None
        return out

    def flush(self) -> None:
        from ..kernels import ops

        if self.pending is not None:
            if self.pending_norm is not None:
                ops.normed_add_rmsnorm(self.x, self.pending, self.pending_norm[0], self.pending_norm[1], None, 0.0, self.act_dtype,
                                       delta_bias=self.pending_norm[2])
            elif self.pending_gate is not None:
                ops.gated_add_rmsnorm(self.x, self.pending, self.pending_gate, None, 0.0, 1, self.act_dtype)
            else:
                ops.add_rmsnorm(self.x, self.pending, None, 0.0, self.act_dtype)
            self.pending = self.pending_norm = self.pending_gate = None


class Norm(Part):
    def forward(self, stream: ResidualStream, rows: Optional[torch.Tensor] = None) -> torch.Tensor:
        """Add what is pending to the stream and return the normalised rows
        (all, or those named by `rows`) in the activation type."""
        raise NotImplementedError

    def rms_weight(self):
        """(weight, eps) if this norm is y = x / sqrt(mean(x^2) + eps) * weight, else None: an arrangement
        may then fold the norm into the products around it (the weight where the product before it stores its
        result, the row's scale where the product after it stores its own)."""
        return None


class PositionEncoding(Part):
    """How a mixer's queries and keys learn their positions.

    `write_qk` is what the attention mixer calls; the default does it in two
    steps from `rotate`, a fused implementation overrides it."""

    def rotate(self, q: torch.Tensor, k: torch.Tensor, step) -> None:
        """Encode positions into q[T, H, hd] and k[T, K, hd] in place."""
        raise NotImplementedError

    def decode_fusion(self):
        """None, or (inv_freq, rotary_dim, interleaved) if this encoding is a rotation by angles
        position * inv_freq[j] of `rotary_dim` leading dimensions (0 = none at all): a mixer may then
        leave `write_qk` out of a decode step and have its attention kernel do the same work."""
        return None

    def score_bias(self) -> Optional[torch.Tensor]:
        """None, or float32 [H, L]: the score of head h for a key n positions behind its query is raised by
        table[h, min(n, L - 1)].  Only a mixer that knows how to add it takes such an encoding."""
        return None

    def write_qk(self, qkv: torch.Tensor, step, kv, num_heads: int, num_kv_heads: int, head_dim: int, write_kv: bool) -> None:
        from ..kernels import ops

        T = qkv.shape[0]
        q = qkv[:, : num_heads * head_dim].view(T, num_heads, head_dim)
        k = qkv[:, num_heads * head_dim : (num_heads + num_kv_heads) * head_dim].view(T, num_kv_heads, head_dim)
        self.rotate(q, k, step)
        if write_kv:
            ops.rope_kv_write(
                qkv, step.tok_pos, step.tok_seq, kv.block_table, kv.k_pages, kv.v_pages, None,
                num_heads, num_kv_heads, head_dim, 0, False, write_kv=True,
            )


class Mixer(Part):
    def cache_need(self):
        """KVNeed, StateNeed, None, or a tuple of needs (a mixer made of several): `forward` then gets a tuple of views
        in the same order."""
        return None

    def output_bias(self) -> Optional[torch.Tensor]:
        """None, or a float32 row [d] that belongs to every row of what `forward` returns (the bias of a last projection,
        left to the kernel that takes the result next)."""
        return None

    def forward(self, xn: torch.Tensor, step, cache, shared_cache: bool = False) -> torch.Tensor:
        """xn[T, d] -> delta [T, d] (or partial sums [parts, T, d]), or `NormedTerms`.

        cache: this run's view of the cache (a KVView or StateView, or None).
        shared_cache: the view belongs to an earlier run of the schedule; read it, do not write it."""
        raise NotImplementedError

    def forward_unprojected(self, xn: torch.Tensor, step, cache, shared_cache: bool = False):
        """None, or (a[T, k], w[d, k]) such that forward(...) == a . w^T: a mixer whose last operation is a
        projection may leave it to the caller, who can then fuse it with what follows."""
        return None


class FeedForward(Part):
    def forward(self, xn: torch.Tensor, step) -> torch.Tensor:
        raise NotImplementedError

    def gated_weights(self):
        """None, or (w_gate_up[2 ff, d] with gate and up rows alternating, w_down[d, ff]) if this feed-forward
        is down(silu(gate(x)) * up(x)) with its weights in that form."""
        return None


class Block(Part):
    """The arrangement of one layer's parts.  Built by the model from a LayerSpec."""

    def __init__(self, spec: PartSpec, runtime: Runtime, mixer: Mixer, feed_forward: FeedForward, norms: Mapping[str, Norm]):
        super().__init__(spec, runtime)
        self.mixer = mixer
        self.feed_forward = feed_forward
        self.norms = dict(norms)

    def forward(self, stream: ResidualStream, step, cache, shared_cache: bool = False) -> None:
        raise NotImplementedError


# --------------------------------------------------------------------------- registries
class Registry:
    def __init__(self, family: str):
        self.family = family
        self._kinds: Dict[str, Callable] = {}

    def register(self, kind: str, cls=None, replace: bool = False):
        """`register("name", Class)` or `@register("name")` above the class."""

        def put(c):
            if kind in self._kinds and not replace:
                raise ConfigError(f"{self.family} '{kind}' is already registered")
            self._kinds[kind] = c
            return c

        return put(cls) if cls is not None else put

    def unregister(self, kind: str) -> None:
        self._kinds.pop(kind, None)

    def get(self, kind: str):
        try:
            return self._kinds[kind]
        except KeyError:
            raise ConfigError(f"unknown {self.family} '{kind}' (known: {', '.join(sorted(self._kinds)) or 'none'})") from None

    def build(self, spec: PartSpec, runtime: Runtime, *args, **kwargs):
        return self.get(spec.kind)(spec, runtime, *args, **kwargs)

    def kinds(self):
        return sorted(self._kinds)


MIXERS = Registry("mixer")
FEED_FORWARDS = Registry("feed-forward")
NORMS = Registry("norm")
POSITIONS = Registry("position encoding")
BLOCKS = Registry("block")
EMBEDDINGS = Registry("embedding")
HEADS = Registry("head")
