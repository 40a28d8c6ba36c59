"""Typed configuration of the Mibezen decoder, read from its config.json.

Keys: `architecture` ("Mibezen"), `vocab`, `width`, `norm.eps`, optional `logit_softcap` (the logits are capped at it),
and `layers`: a list whose entries give `type` ("latent_attention" or "attention"), the mixer's sizes and constants under
`mixer` and the feed-forward under `mlp` (null: none).

mixer of a latent_attention layer: `heads`, `dim` (unrotated query/key numbers per head), `rot_dim` (rotated ones),
`vdim`, `q_rank` (size of the queries' latent), `kv_rank`, `scale`, `rot` (`dims`, equal to `rot_dim`, `base`, optional
`scaling` with `factor`, `original`, `fast`, `slow`).
mixer of an attention layer: `heads`, `kv_heads`, `dim`, `vdim`, `scale`, optional `mask.size` (positions per chunk; none:
one chunk), optional `v_mix` (the values take a share of those of the first layer that has it).
mlp: `kind` "dense" with `ff`, or "moe" with `expert.ff`, `router.experts`, `router.top`.
"""
from __future__ import annotations

from dataclasses import dataclass
from typing import Any, Dict, Optional, Tuple, Union

from .base import ConfigError, KeyReader

ARCHITECTURE = "Mibezen"
MAX_POSITIONS = 131072      # the design names no longest sequence; rotation tables are made for as many positions as an engine allows, at most this


def _object(data: Any, where: str) -> Dict[str, Any]:
    if not isinstance(data, dict):
        raise ConfigError(f"key '{where}' must be an object, got {data!r}")
    return data


@dataclass(frozen=True)
class RampedRotaryConfig:
    dims: int
    base: float
    scaling: Optional[Tuple[float, float, float, float]] = None     # factor, original, fast, slow

    def to_dict(self):
        d: Dict[str, Any] = {"base": self.base, "dims": self.dims}
        if self.scaling is not None:
            d["scaling"] = dict(zip(("factor", "original", "fast", "slow"), self.scaling))
        return d


@dataclass(frozen=True)
class LatentMixerConfig:
    heads: int
    dim: int
    rot_dim: int
    vdim: int
    q_rank: int
    kv_rank: int
    scale: float
    rot: Optional[RampedRotaryConfig] = None

    TYPE = "latent_attention"

    def to_dict(self):
        d: Dict[str, Any] = {"dim": self.dim, "heads": self.heads, "kv_rank": self.kv_rank, "q_rank": self.q_rank,
                             "rot_dim": self.rot_dim, "scale": self.scale, "vdim": self.vdim}
        if self.rot is not None:
            d["rot"] = self.rot.to_dict()
        return d


@dataclass(frozen=True)
class ChunkedMixerConfig:
    heads: int
    kv_heads: int
    dim: int
    vdim: int
    scale: float
    chunk: int = 0              # 0: one chunk
    v_mix: bool = False

    TYPE = "attention"

    def to_dict(self):
        return {"dim": self.dim, "heads": self.heads, "kv_heads": self.kv_heads,
                "mask": {"size": self.chunk} if self.chunk else None, "scale": self.scale, "v_mix": self.v_mix,
                "vdim": self.vdim}


@dataclass(frozen=True)
class DenseConfig:
    ff: int

    def to_dict(self):
        return {"ff": self.ff, "kind": "dense"}


@dataclass(frozen=True)
class ExpertsConfig:
    ff: int
    experts: int
    top: int

    def to_dict(self):
        return {"expert": {"ff": self.ff}, "kind": "moe", "router": {"experts": self.experts, "top": self.top}}


@dataclass(frozen=True)
class MibezenLayer:
    mixer: Union[LatentMixerConfig, ChunkedMixerConfig]
    mlp: Union[DenseConfig, ExpertsConfig, None]

    def to_dict(self):
        return {"mixer": self.mixer.to_dict(), "mlp": None if self.mlp is None else self.mlp.to_dict(),
                "type": self.mixer.TYPE}


def _read_latent_mixer(raw: Dict[str, Any], where: str) -> LatentMixerConfig:
    r = KeyReader(raw)
    rot_dim = r.integer("rot_dim", minimum=0)
    rot = None
    if raw.get("rot") is not None:
        rraw = _object(raw["rot"], where + ".rot")
        k = KeyReader(rraw)
        dims = k.integer("dims")
        if dims != rot_dim or dims % 2:
            raise ConfigError(f"key '{where}.rot.dims' ({dims}) must be even and equal 'rot_dim' ({rot_dim})")
        scaling = None
        if rraw.get("scaling") is not None:
            s = KeyReader(_object(rraw["scaling"], where + ".rot.scaling"))
            scaling = (s.number("factor"), s.number("original"), s.number("fast"), s.number("slow"))
        rot = RampedRotaryConfig(dims, k.number("base"), scaling)
    elif rot_dim:
        raise ConfigError(f"missing required key '{where}.rot' ({rot_dim} rotated numbers)")
    return LatentMixerConfig(r.integer("heads"), r.integer("dim"), rot_dim, r.integer("vdim"), r.integer("q_rank"),
                             r.integer("kv_rank"), r.number("scale"), rot)


def _read_chunked_mixer(raw: Dict[str, Any], where: str) -> ChunkedMixerConfig:
    r = KeyReader(raw)
    heads, kv_heads = r.integer("heads"), r.integer("kv_heads")
    if heads % kv_heads:
        raise ConfigError(f"key '{where}.heads' ({heads}) must be a multiple of 'kv_heads' ({kv_heads})")
    chunk = 0
    if raw.get("mask") is not None:
        chunk = KeyReader(_object(raw["mask"], where + ".mask")).integer("size", 0)
    return ChunkedMixerConfig(heads, kv_heads, r.integer("dim"), r.integer("vdim"), r.number("scale"), chunk,
                              r.boolean("v_mix", False))


def _read_mlp(raw: Any, where: str):
    if raw is None:
        return None
    m = _object(raw, where)
    kind = m.get("kind")
    if kind == "dense":
        return DenseConfig(KeyReader(m).integer("ff"))
    if kind != "moe":
        raise ConfigError(f"key '{where}.kind': unsupported value {kind!r} (supported: 'dense', 'moe')")
    router = KeyReader(_object(m.get("router"), where + ".router"))
    experts, top = router.integer("experts"), router.integer("top")
    if top > experts:
        raise ConfigError(f"key '{where}.router.top' ({top}) exceeds 'experts' ({experts})")
    return ExpertsConfig(KeyReader(_object(m.get("expert"), where + ".expert")).integer("ff"), experts, top)


@dataclass(frozen=True)
class MibezenConfig:
    vocab: int
    width: int
    eps: float
    logit_softcap: Optional[float]
    layers: Tuple[MibezenLayer, ...]

    ARCHITECTURE = ARCHITECTURE

    @property
    def max_positions(self) -> int:
        return MAX_POSITIONS

    def stop_token_ids(self) -> Tuple[int, ...]:
        return ()

    @property
    def first_mixed(self) -> Optional[int]:
        """The first layer with `v_mix`, whose values the later ones take a share of."""
        return next((i for i, layer in enumerate(self.layers) if getattr(layer.mixer, "v_mix", False)), None)

    @classmethod
    def from_dict(cls, d: Dict[str, Any]) -> "MibezenConfig":
        r = KeyReader(d)
        norm = KeyReader(_object(d.get("norm"), "norm"))
        raw_layers = d.get("layers")
        if not isinstance(raw_layers, list) or not raw_layers:
            raise ConfigError(f"key 'layers' must be a non-empty list, got {type(raw_layers).__name__}")
        readers = {"latent_attention": _read_latent_mixer, "attention": _read_chunked_mixer}
        layers = []
        for i, raw in enumerate(raw_layers):
            where = f"layers[{i}]"
            raw = _object(raw, where)
            read = readers.get(raw.get("type"))
            if read is None:
                raise ConfigError(f"key '{where}.type': unsupported value {raw.get('type')!r} (supported: {sorted(readers)})")
            mixer = read(_object(raw.get("mixer"), where + ".mixer"), where + ".mixer")
            layers.append(MibezenLayer(mixer, _read_mlp(raw.get("mlp"), where + ".mlp")))
        config = cls(vocab=r.integer("vocab"), width=r.integer("width"), eps=norm.number("eps"),
                     logit_softcap=r.number("logit_softcap", None), layers=tuple(layers))
        first = config.first_mixed
        for i, layer in enumerate(layers):
            if i != first and getattr(layer.mixer, "v_mix", False):
                a, b = layers[first].mixer, layer.mixer
                if (a.kv_heads, a.vdim) != (b.kv_heads, b.vdim):
                    raise ConfigError(f"key 'layers[{i}].mixer.v_mix': the values of layer {first} have another 'kv_heads' or "
                                      f"'vdim' than this layer's")
        return config

    def to_dict(self) -> Dict[str, Any]:
        return {"architecture": ARCHITECTURE, "layers": [layer.to_dict() for layer in self.layers],
                "logit_softcap": self.logit_softcap, "norm": {"eps": self.eps}, "vocab": self.vocab, "width": self.width}
