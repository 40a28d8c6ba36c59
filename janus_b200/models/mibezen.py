"""The Mibezen decoder as data: a `ModelSpec` made from a `MibezenConfig`.

A layer mixes by latent attention whose queries have a latent of their own, with a rotated key part (pairs of neighbours,
ramped frequencies) and an output gate per head (`parts.latent_attention`), or by grouped-query attention without positions
of its own: a bias that is linear in the distance, chunks, a learned sink per head, values that take a share of those of
the first such layer, the same gate (`parts.capped_attention`).  Then a dense feed-forward with the square of relu
(`parts.feedforward`), experts chosen by softmax scores whose weights are shares of their sum (`parts.routed`), or none.
Pre-norm, RMS norms whose weights are stored around zero, a soft cap on the logits.  Tensor names: `embed`, `l<i>.norm1`,
`l<i>.norm2`, `l<i>.mix.*`, `l<i>.mlp.*`, `final.norm`, `head`.
"""
from __future__ import annotations

from typing import List

from ..config.mibezen import DenseConfig, LatentMixerConfig, MibezenConfig
from ..config.registry import register_architecture
from ..parts.base import LayerSpec, ModelSpec, PartSpec, ScheduleEntry


def distance_slopes(heads: int):
    """Slope of the distance bias of every head: a geometric row from 2^(-8 / heads) to 2^-8."""
    return tuple(2.0 ** (-8.0 * (h + 1) / heads) for h in range(heads))


def _latent_spec(config: MibezenConfig, m: LatentMixerConfig, p: str) -> PartSpec:
    position = None
    if m.rot is not None:
        scaling = None if m.rot.scaling is None else dict(zip(("factor", "original", "fast", "slow"), m.rot.scaling))
        position = PartSpec("ramped_rotary", dict(dims=m.rot.dims, theta=m.rot.base, max_positions=config.max_positions,
                                                  scaling=scaling))
    return PartSpec("rotary_latent_attention",
                    dict(hidden_size=config.width, num_heads=m.heads, dim=m.dim, rot_dim=m.rot_dim, vdim=m.vdim,
                         rank=m.kv_rank, q_rank=m.q_rank, scale=m.scale, eps=config.eps, position=position, gate="head",
                         pairs="neighbours"),
                    weights=dict(dq=p + "dq", dq_norm=p + "dq.norm", uq=p + "uq", dkv=p + "dkv", dkv_norm=p + "dkv.norm",
                                 uk=p + "uk", uv=p + "uv", g=p + "g", o=p + "o"))


def _mixer_spec(config: MibezenConfig, i: int) -> PartSpec:
    m, p = config.layers[i].mixer, f"l{i}.mix."
    if isinstance(m, LatentMixerConfig):
        return _latent_spec(config, m, p)
    mix = None if not m.v_mix else "first" if i == config.first_mixed else "mix"
    weights = {n: p + n for n in ("q", "k", "v", "g", "o", "sink")}
    if mix == "mix":
        weights["vmix"] = p + "vmix"
    return PartSpec("capped_attention",
                    dict(hidden_size=config.width, num_heads=m.heads, num_kv_heads=m.kv_heads, dim=m.dim, vdim=m.vdim,
                         scale=m.scale, eps=config.eps, chunk=m.chunk, qk_norm=False, gate="head", sink="learned",
                         slopes=distance_slopes(m.heads), value_mix=mix), weights=weights)


def _feed_forward_spec(config: MibezenConfig, i: int) -> PartSpec:
    mlp, p = config.layers[i].mlp, f"l{i}.mlp."
    if isinstance(mlp, DenseConfig):
        return PartSpec("relu2_mlp", dict(hidden_size=config.width, intermediate_size=mlp.ff),
                        weights=dict(up=p + "up", down=p + "down"))
    weights = {"router": p + "router"}
    for e in range(mlp.experts):
        weights.update({f"e{e}_{n}": p + f"e{e}.{n}" for n in ("gate", "up", "down")})
    return PartSpec("routed_experts",
                    dict(hidden_size=config.width, intermediate_size=mlp.ff, experts=mlp.experts, top=mlp.top,
                         score="softmax", weight_on="output", shares=True), weights=weights)


def mibezen_spec(config: MibezenConfig) -> ModelSpec:
    layers: List[LayerSpec] = []
    # tensors a file may have that nothing reads: shares of layers that mix no values in, norms of feed-forwards that are
    # not there
    unused = [f"l{i}.mix.vmix" for i, layer in enumerate(config.layers)
              if i == config.first_mixed or not getattr(layer.mixer, "v_mix", False)]
    norm_of = lambda name: PartSpec("rms_norm", dict(width=config.width, eps=config.eps, weight_offset=1.0),   # noqa: E731
                                    weights=dict(gamma=name))
    for i, layer in enumerate(config.layers):
        p = f"l{i}."
        feed_forward = feed_forward_norm = None
        if layer.mlp is not None:
            feed_forward, feed_forward_norm = _feed_forward_spec(config, i), norm_of(p + "norm2")
        else:
            unused.append(p + "norm2")
        layers.append(LayerSpec(mixer=_mixer_spec(config, i), feed_forward=feed_forward, mixer_norm=norm_of(p + "norm1"),
                                feed_forward_norm=feed_forward_norm))
    cap = () if config.logit_softcap is None else (PartSpec("scale_soft_cap", dict(cap=config.logit_softcap)),)
    return ModelSpec(
        hidden_size=config.width, vocab_size=config.vocab, layers=tuple(layers),
        schedule=tuple(ScheduleEntry(i) for i in range(len(layers))), final_norm=norm_of("final.norm"),
        embedding_weight="embed", head_weight="head", max_positions=config.max_positions,
        ignorable_weights=tuple(unused), logit_transforms=cap, pad_head_width=True)


def build_mibezen(config: MibezenConfig, dtype, device):
    from ..engine.model import DecoderModel
    return DecoderModel(mibezen_spec(config), dtype, device)


def mibezen_weight_specs(config: MibezenConfig):
    from ..engine.model import model_weight_specs
    return model_weight_specs(mibezen_spec(config))


register_architecture(MibezenConfig.ARCHITECTURE, MibezenConfig, build_mibezen, mibezen_weight_specs)
