"""Typed configuration of the Forisun decoder, read from its config.json.

Keys: `architecture` ("Forisun"), `vocab`, `width`, `norm.eps`, `embedding.scale` (the embedding is multiplied by it),
and `layers`: a list whose entries give `type` ("latent_attention"), the mixer's sizes and constants under `mixer` and
the feed-forward under `mlp` (null: none).

mixer: `heads`, `dim` (unrotated query/key numbers per head), `rot_dim` (rotated ones), `vdim`, `kv_rank`, `scale`,
`rot` (`dims`, equal to `rot_dim`, `base`, optional `scaling` with `factor`, `original`, `fast`, `slow`), optional
`kv_from` (the index of the earlier layer whose cached rows this layer attends over; it then has no latent projection of
its own).
mlp: `kind` "dense" with `ff`, or "moe" with `expert.ff`, `router.experts`, `router.top`, `router.scale`.
"""
from __future__ import annotations

from dataclasses import dataclass
from typing import Any, Dict, Optional, Tuple, Union

from .base import ConfigError, KeyReader

ARCHITECTURE = "Forisun"
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
    kv_rank: int
    scale: float
    rot: Optional[RampedRotaryConfig] = None
    kv_from: Optional[int] = None

    def to_dict(self):
        d: Dict[str, Any] = {"dim": self.dim, "heads": self.heads, "kv_rank": self.kv_rank, "rot_dim": self.rot_dim,
                             "scale": self.scale, "vdim": self.vdim}
        if self.rot is not None:
            d["rot"] = self.rot.to_dict()
        if self.kv_from is not None:
            d["kv_from"] = self.kv_from
        return d


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
    scale: float

    def to_dict(self):
        return {"expert": {"ff": self.ff}, "kind": "moe",
                "router": {"experts": self.experts, "scale": self.scale, "top": self.top}}


@dataclass(frozen=True)
class ForisunLayer:
    mixer: LatentMixerConfig
    mlp: Union[DenseConfig, ExpertsConfig, None]

    def to_dict(self):
        return {"mixer": self.mixer.to_dict(), "mlp": None if self.mlp is None else self.mlp.to_dict(),
                "type": "latent_attention"}


def _read_mixer(raw: Dict[str, Any], where: str) -> LatentMixerConfig:
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
    return LatentMixerConfig(r.integer("heads"), r.integer("dim"), rot_dim, r.integer("vdim"), r.integer("kv_rank"),
                             r.number("scale"), rot, r.integer("kv_from", None, minimum=0))


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
    return ExpertsConfig(KeyReader(_object(m.get("expert"), where + ".expert")).integer("ff"), experts, top,
                         router.number("scale", 1.0))


@dataclass(frozen=True)
class ForisunConfig:
    vocab: int
    width: int
    eps: float
    embedding_scale: float
    layers: Tuple[ForisunLayer, ...]

    ARCHITECTURE = ARCHITECTURE

    @property
    def max_positions(self) -> int:
        return MAX_POSITIONS

    def stop_token_ids(self) -> Tuple[int, ...]:
        return ()

    @classmethod
    def from_dict(cls, d: Dict[str, Any]) -> "ForisunConfig":
        r = KeyReader(d)
        norm = KeyReader(_object(d.get("norm"), "norm"))
        embedding = KeyReader(_object(d.get("embedding"), "embedding"))
        raw_layers = d.get("layers")
        if not isinstance(raw_layers, list) or not raw_layers:
            raise ConfigError(f"key 'layers' must be a non-empty list, got {type(raw_layers).__name__}")
        layers = []
        for i, raw in enumerate(raw_layers):
            where = f"layers[{i}]"
            raw = _object(raw, where)
            if raw.get("type") != "latent_attention":
                raise ConfigError(f"key '{where}.type': unsupported value {raw.get('type')!r} (supported: 'latent_attention')")
            mixer = _read_mixer(_object(raw.get("mixer"), where + ".mixer"), where + ".mixer")
            layers.append(ForisunLayer(mixer, _read_mlp(raw.get("mlp"), where + ".mlp")))
        for i, layer in enumerate(layers):
            j = layer.mixer.kv_from
            if j is None:
                continue
            where = f"layers[{i}].mixer.kv_from"
            if j >= i or layers[j].mixer.kv_from is not None:
                raise ConfigError(f"key '{where}' must name an earlier layer with a latent of its own, got {j}")
            a, b = layers[j].mixer, layer.mixer
            if (a.kv_rank, a.rot_dim, a.rot) != (b.kv_rank, b.rot_dim, b.rot):
                raise ConfigError(f"key '{where}': layer {j}'s rows have another kv_rank, rot_dim or rotation than this layer's")
        return cls(vocab=r.integer("vocab"), width=r.integer("width"), eps=norm.number("eps"),
                   embedding_scale=embedding.number("scale"), layers=tuple(layers))

    def to_dict(self) -> Dict[str, Any]:
        return {"architecture": ARCHITECTURE, "embedding": {"scale": self.embedding_scale},
                "layers": [layer.to_dict() for layer in self.layers], "norm": {"eps": self.eps}, "vocab": self.vocab,
                "width": self.width}
