"""Damadra, as a description made of the library's parts.

A decoder whose sublayers read the residual stream as it is and whose results are normed before they are added,
    x += m norm_1(mixer(x));   x += m norm_2(ff(x))          (m a constant; a layer may have no ff)
No rotation anywhere: positions enter through a learned bias on the scores by head and distance (a table of buckets per layer),
through windows and through the queries' temperature.  Per layer one of two mixers:

  attention     grouped-query attention in a sliding window; queries and keys normed over all their heads at once; the values are
                the keys as projected, before that norm
  attention_2   grouped-query attention over every earlier token; queries and keys normed head by head, queries times a temperature
                that grows with the logarithm of the position; a layer may read an earlier layer's keys and values

and a dense gated feed-forward or experts W_down relu(W_up x)^2 chosen by score plus correction and weighted by their softmax
scores as they are, among them choices that hand the input on.

Tensor names: embed, head, final.norm, and per layer i: l<i>.norm1 / norm2, l<i>.mix.q / k / v / o / q.norm / k.norm / rel,
l<i>.mlp.gate / up / down or l<i>.mlp.e<j>.up / down, l<i>.mlp.router, l<i>.mlp.correction.
"""

from __future__ import annotations

from ..config.damadra import (
    ARCHITECTURE, MAX_POSITIONS, DamadraConfig, DenseConfig, ExpertsConfig, FullMixerConfig, WindowedMixerConfig,
)
from ..registry import Architecture, register_architecture
from ..spec import LayerSpec, ModelSpec, PartSpec, ScheduleEntry

_ATTENTION_NAMES = {"q": "q", "k": "k", "v": "v", "o": "o", "q_norm": "q.norm", "k_norm": "k.norm"}


def describe_damadra(cfg: DamadraConfig) -> ModelSpec:
    def norm(prefix: str, factor: float = 1.0) -> PartSpec:
        return PartSpec("rmsnorm", {"size": cfg.width, "eps": cfg.eps, "name": "", "float32": True, "factor": factor}, prefix)

    def attention(m, prefix: str, **options) -> PartSpec:
        position = PartSpec("distance_bias", {"num_heads": m.heads, "max_distance": m.bias_max}, prefix)
        params = {"hidden_size": cfg.width, "num_heads": m.heads, "num_kv_heads": m.kv_heads, "head_dim": m.dim, "scale": m.scale,
                  "qk_norm": cfg.eps, "position": position, "names": _ATTENTION_NAMES}
        return PartSpec("attention", dict(params, **options), prefix)

    layers, schedule = [], []
    for i, layer in enumerate(cfg.layers):
        p, m = f"l{i}.", layer.mixer
        cache_from = None
        if isinstance(m, WindowedMixerConfig):
            mixer = attention(m, p + "mix.", window=m.window, values="keys", qk_norm_span="all")
        elif isinstance(m, FullMixerConfig):
            mixer = attention(m, p + "mix.", window=0, value_dim=m.vdim, own_kv=m.kv_from is None,
                              q_temperature=(m.temp_coef, m.temp_every) if m.temp_every else None)
            cache_from = m.kv_from
        else:
            raise TypeError(f"layer {i}: {type(m).__name__} is not a mixer configuration of this architecture")
        norms = {"mixer_out": norm(p + "norm1", cfg.residual_mult)}
        ff = None
        if isinstance(layer.mlp, DenseConfig):
            ff = PartSpec(
                "gated_mlp",
                {"hidden_size": cfg.width, "intermediate_size": layer.mlp.ff, "activation": "silu", "names": {"gate": "gate", "up": "up", "down": "down"}},
                p + "mlp.",
            )
        elif isinstance(layer.mlp, ExpertsConfig):
            e = layer.mlp
            ff = PartSpec(
                "routed_experts",
                {"hidden_size": cfg.width, "n_experts": e.experts, "identity": e.identity, "top": e.top, "expert_ff": e.ff, "bias": True,
                 "renormalize": False, "activation": "relu2"},
                p + "mlp.",
            )
        if ff is not None:
            norms["feed_forward_out"] = norm(p + "norm2", cfg.residual_mult)
        layers.append(LayerSpec(block="postnorm", mixer=mixer, feed_forward=ff, norms=norms))
        schedule.append(ScheduleEntry(i, cache_from=cache_from))
    return ModelSpec(
        architecture=cfg.architecture,
        hidden_size=cfg.width,
        vocab_size=cfg.vocab,
        max_positions=MAX_POSITIONS,
        embedding=PartSpec("token_embedding", {"vocab_size": cfg.vocab, "hidden_size": cfg.width, "name": "", "scale": cfg.embedding_scale}, "embed"),
        layers=tuple(layers),
        schedule=tuple(schedule),
        final_norm=norm("final.norm"),
        head=PartSpec("linear_head", {"vocab_size": cfg.vocab, "hidden_size": cfg.width, "tied_to": None, "name": ""}, "head"),
        stored_dtype="bfloat16",
    )


register_architecture(Architecture(ARCHITECTURE, DamadraConfig.from_json, describe_damadra), replace=True)
