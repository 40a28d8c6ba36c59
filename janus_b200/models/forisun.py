"""The Forisun decoder as data: a `ModelSpec` made from a `ForisunConfig`.

Every layer is latent attention with a rotated key part and an output gate (`parts.latent_attention`; a layer with
`kv_from` is a place of the schedule that reads the rows an earlier place cached), then a dense feed-forward with the
exact GELU and no gate (`parts.feedforward`), experts chosen by corrected sigmoid scores, weighted on their outputs
(`parts.routed`), or none.  Dynamic tanh stands in the place of every norm: on the scaled embedding, before and after
each sublayer (arrangement `sandwich_norm`) and before the head.  Tensor names: `embed`, `embed.norm`, `l<i>.norm1`,
`l<i>.norm1b`, `l<i>.norm2`, `l<i>.norm2b`, `l<i>.mix.*`, `l<i>.mlp.*`, `final.norm`, `head`; a norm has `.b` and
`.alpha` beside its weight.
"""
from __future__ import annotations

from typing import Dict, List

from ..config.forisun import DenseConfig, ForisunConfig
from ..config.registry import register_architecture
from ..parts.base import LayerSpec, ModelSpec, PartSpec, ScheduleEntry


def _norm_weights(name: str) -> Dict[str, str]:
    return dict(gamma=name, beta=name + ".b", alpha=name + ".alpha")


def _mixer_spec(config: ForisunConfig, i: int) -> PartSpec:
    m, p = config.layers[i].mixer, f"l{i}.mix."
    own = m.kv_from is None
    weights = dict(q=p + "q", uk=p + "uk", uv=p + "uv", g=p + "g", o=p + "o")
    if own:
        weights.update(dkv=p + "dkv", dkv_norm=p + "dkv.norm")
    position = None
    if m.rot is not None:
        scaling = None if m.rot.scaling is None else dict(zip(("factor", "original", "fast", "slow"), m.rot.scaling))
        position = PartSpec("ramped_rotary", dict(dims=m.rot.dims, theta=m.rot.base, max_positions=config.max_positions,
                                                  scaling=scaling))
    return PartSpec("rotary_latent_attention",
                    dict(hidden_size=config.width, num_heads=m.heads, dim=m.dim, rot_dim=m.rot_dim, vdim=m.vdim,
                         rank=m.kv_rank, scale=m.scale, eps=config.eps, position=position, gate=True, own_latent=own),
                    weights=weights)


def _feed_forward_spec(config: ForisunConfig, i: int) -> PartSpec:
    mlp, p = config.layers[i].mlp, f"l{i}.mlp."
    if isinstance(mlp, DenseConfig):
        return PartSpec("gelu_mlp", dict(hidden_size=config.width, intermediate_size=mlp.ff),
                        weights=dict(up=p + "up", down=p + "down"))
    weights = {"router": p + "router", "correction": p + "correction"}
    for e in range(mlp.experts):
        weights.update({f"e{e}_{n}": p + f"e{e}.{n}" for n in ("gate", "up", "down")})
    return PartSpec("routed_experts",
                    dict(hidden_size=config.width, intermediate_size=mlp.ff, experts=mlp.experts, top=mlp.top,
                         weight_on="output", correction=True, scale=mlp.scale), weights=weights)


def forisun_spec(config: ForisunConfig) -> ModelSpec:
    layers: List[LayerSpec] = []
    schedule: List[ScheduleEntry] = []
    unused: List[str] = []
    norm_of = lambda name: PartSpec("dynamic_tanh", dict(width=config.width), weights=_norm_weights(name))   # noqa: E731
    for i, layer in enumerate(config.layers):
        p = f"l{i}."
        feed_forward = feed_forward_norm = None
        extra = (("mixer_out_norm", "norm", norm_of(p + "norm1b")),)
        if layer.mlp is not None:
            feed_forward, feed_forward_norm = _feed_forward_spec(config, i), norm_of(p + "norm2")
            extra += (("feed_forward_out_norm", "norm", norm_of(p + "norm2b")),)
        else:       # a layer without a feed-forward leaves its norms unread if the file has them
            unused += [*_norm_weights(p + "norm2").values(), *_norm_weights(p + "norm2b").values()]
        layers.append(LayerSpec(mixer=_mixer_spec(config, i), feed_forward=feed_forward, mixer_norm=norm_of(p + "norm1"),
                                feed_forward_norm=feed_forward_norm, arrangement="sandwich_norm", extra=extra))
        schedule.append(ScheduleEntry(i, reads_cache_of=layer.mixer.kv_from))    # layers and places have the same numbers
    return ModelSpec(
        hidden_size=config.width, vocab_size=config.vocab, layers=tuple(layers), schedule=tuple(schedule),
        final_norm=norm_of("final.norm"), embedding_weight="embed", head_weight="head",
        max_positions=config.max_positions, ignorable_weights=tuple(unused),
        embedding_transforms=(PartSpec("scale_soft_cap", dict(scale=config.embedding_scale)),
                              PartSpec("dynamic_tanh", dict(width=config.width), weights=_norm_weights("embed.norm"))),
        pad_head_width=True)


def build_forisun(config: ForisunConfig, dtype, device):
    from ..engine.model import DecoderModel
    return DecoderModel(forisun_spec(config), dtype, device)


def forisun_weight_specs(config: ForisunConfig):
    from ..engine.model import model_weight_specs
    return model_weight_specs(forisun_spec(config))


register_architecture(ForisunConfig.ARCHITECTURE, ForisunConfig, build_forisun, forisun_weight_specs)
