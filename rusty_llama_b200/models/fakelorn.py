"""Fakelorn, as a description made of the library's parts.

A pre-norm decoder whose two results per layer are gated element by element by the sublayer's own input,
    x += s(W_1 h + b_1) * mixer(h), h = norm_1(x);   x += s(W_2 h + b_2) * ff(h), h = norm_2(x)       (s the logistic function)
every norm an RMS norm over equal consecutive parts of the row, the classifier tied to the embedding table, its logits scaled
and capped.  Per layer one of three mixers:

  attention         differential attention in a sliding window: two softmax maps per head over the same values, their difference
                    normed per head; no position signal
  mamba2            a state-space layer: one decay number per head and token, state keys and queries shared by groups of heads,
                    behind a short causal convolution; the output gate comes before the norm
  latent_attention  attention over one cached latent and one shared rotated key part per position (halves paired), the queries
                    through a latent of their own, an output gate; a layer may read an earlier layer's latents

and a dense gated feed-forward or experts weighted by a softmax over the chosen ones' logits, beside a shared expert.

Tensor names: embed, final.norm, and per layer i: l<i>.norm1 / norm2, l<i>.rg1 / rg1.b / rg2 / rg2.b (the result gates),
l<i>.mix.<name>, l<i>.mlp.gate / up / down or l<i>.mlp.e<j>.gate / up / down, l<i>.mlp.router, l<i>.mlp.shared.<name>.
"""

from __future__ import annotations

from ..config.fakelorn import (
    ARCHITECTURE, MAX_POSITIONS, AttentionMixerConfig, DenseConfig, FakelornConfig, LatentMixerConfig, Mamba2MixerConfig,
)
from ..registry import Architecture, register_architecture
from ..spec import LayerSpec, ModelSpec, PartSpec, ScheduleEntry

_DIFFERENTIAL_NAMES = {"q": "q", "k": "k", "v": "v", "o": "o"}


def describe_fakelorn(cfg: FakelornConfig) -> ModelSpec:
    def norm(prefix: str) -> PartSpec:
        return PartSpec("rmsnorm", {"size": cfg.width, "eps": cfg.eps, "name": "", "groups": cfg.norm_groups, "float32": True}, prefix)

    layers, schedule = [], []
    for i, layer in enumerate(cfg.layers):
        p, m = f"l{i}.", layer.mixer
        cache_from = None
        if isinstance(m, AttentionMixerConfig):
            mixer = PartSpec(
                "differential_attention",
                {"hidden_size": cfg.width, "num_heads": m.heads, "num_kv_heads": m.kv_heads, "map_dim": m.dim, "value_dim": m.vdim,
                 "scale": m.scale, "window": m.window, "diff": m.diff, "eps": cfg.eps, "names": _DIFFERENTIAL_NAMES},
                p + "mix.",
            )
        elif isinstance(m, Mamba2MixerConfig):
            mixer = PartSpec(
                "mamba2",
                {"hidden_size": cfg.width, "num_heads": m.heads, "vdim": m.vdim, "state": m.state, "groups": m.groups, "taps": m.conv,
                 "norm_groups": m.norm_groups, "eps": cfg.eps},
                p + "mix.",
            )
        elif isinstance(m, LatentMixerConfig):
            position = PartSpec("rotary", {"rotary_dim": m.rot_dims, "theta": m.rot_base, "scaling": None, "interleaved": False}) \
                if m.rot_dims else PartSpec("none")
            mixer = PartSpec(
                "latent_attention",
                {"hidden_size": cfg.width, "num_heads": m.heads, "dim": m.dim, "rot_dim": m.rot_dim, "vdim": m.vdim, "q_rank": m.q_rank,
                 "kv_rank": m.kv_rank, "scale": m.scale, "eps": cfg.eps, "sink": False, "gate": True, "own_kv": m.kv_from is None,
                 "window": 0, "position": position},
                p + "mix.",
            )
            cache_from = m.kv_from
        else:
            raise TypeError(f"layer {i}: {type(m).__name__} is not a mixer configuration of this architecture")
        norms = {"mixer": norm(p + "norm1")}
        ff = None
        if isinstance(layer.mlp, DenseConfig):
            ff = PartSpec(
                "gated_mlp",
                {"hidden_size": cfg.width, "intermediate_size": layer.mlp.ff, "activation": "silu", "names": {"gate": "gate", "up": "up", "down": "down"}},
                p + "mlp.",
            )
        elif layer.mlp is not None:
            e = layer.mlp
            ff = PartSpec(
                "routed_experts",  # (softmax over all experts, divided by the chosen ones' sum: the softmax over the chosen logits)
                {"hidden_size": cfg.width, "n_experts": e.experts, "top": e.top, "expert_ff": e.ff, "bias": False, "renormalize": True,
                 "shared_ff": e.shared_ff, "shared_gate": False},
                p + "mlp.",
            )
        if ff is not None:
            norms["feed_forward"] = norm(p + "norm2")
        layers.append(LayerSpec(block="gated_prenorm", mixer=mixer, feed_forward=ff, norms=norms,
                                block_params={"hidden_size": cfg.width, "names": {"mixer": "rg1", "feed_forward": "rg2"}}, block_prefix=p))
        schedule.append(ScheduleEntry(i, cache_from=cache_from))
    return ModelSpec(
        architecture=cfg.architecture,
        hidden_size=cfg.width,
        vocab_size=cfg.vocab,
        max_positions=MAX_POSITIONS,
        embedding=PartSpec("token_embedding", {"vocab_size": cfg.vocab, "hidden_size": cfg.width, "name": ""}, "embed"),
        layers=tuple(layers),
        schedule=tuple(schedule),
        final_norm=norm("final.norm"),
        head=PartSpec("linear_head", {"vocab_size": cfg.vocab, "hidden_size": cfg.width, "tied_to": "embed", "name": "",
                                      "scale": cfg.logit_scale, "softcap": cfg.logit_softcap}, "head"),
        stored_dtype="bfloat16",
    )


register_architecture(Architecture(ARCHITECTURE, FakelornConfig.from_json, describe_fakelorn), replace=True)
