"""`ZosuraxConfig`: the config.json of a Zosurax decoder, typed and validated.

The file is nested: `layers` lists the layers, each with its `type` (which mixer: "hgrn2", "attention" or "attention_2"), the
mixer's sizes under `mixer` and its feed-forward under `mlp` (null: none; `kind` "dense"); `loop` (absent: none) names the
range of layers that runs several times; `norm.eps`, `vocab` and `width` are the model's.  A key the design always has is
required and every error names its key; an attention's `rot` may be absent (nothing is rotated).
"""
from __future__ import annotations

from dataclasses import dataclass

from .base import ConfigError, ConfigReader


@dataclass(frozen=True)
class Rotation:
    base: float
    dims: int


@dataclass(frozen=True)
class AttentionSizes:
    heads: int
    kv_heads: int
    dim: int
    vdim: int
    scale: float
    rot: Rotation | None


@dataclass(frozen=True)
class HGRN2Sizes:
    heads: int
    dim: int
    vdim: int


@dataclass(frozen=True)
class DenseSizes:
    ff: int


@dataclass(frozen=True)
class Loop:
    start: int
    stop: int
    times: int


@dataclass(frozen=True)
class ZosuraxLayer:
    type: str
    mixer: object
    mlp: DenseSizes | None


def _rotation(raw, where, most) -> Rotation | None:
    if raw is None:
        return None
    r = ConfigReader(raw, where)
    rot = Rotation(r.float("base", positive=True), r.int("dims", min=0))
    if rot.dims % 2 or rot.dims > most:
        raise ConfigError(f"{where}: 'dims' {rot.dims} must be even and at most {most}")
    return rot


def _mixer(kind: str, raw, where: str):
    if not isinstance(raw, dict):
        raise ConfigError(f"{where}: 'mixer' must be an object")
    r = ConfigReader(raw, where)
    if kind == "hgrn2":
        return HGRN2Sizes(r.int("heads", min=1), r.int("dim", min=1), r.int("vdim", min=1))
    if kind in ("attention", "attention_2"):
        heads, kv = r.int("heads", min=1), r.int("kv_heads", min=1)
        if heads % kv:
            raise ConfigError(f"{where}: 'heads' {heads} is not a multiple of 'kv_heads' {kv}")
        dim = r.int("dim", min=1)
        return AttentionSizes(heads, kv, dim, r.int("vdim", min=1), r.float("scale", positive=True), _rotation(r.any("rot"), f"{where}.rot", dim))
    raise ConfigError(f"{where}: layer type {kind!r} is not one of 'hgrn2', 'attention', 'attention_2'")


def _mlp(raw, where: str):
    if raw is None:
        return None
    r = ConfigReader(raw, where)
    kind = r.str("kind")
    if kind != "dense":
        raise ConfigError(f"{where}: feed-forward kind {kind!r} is not 'dense'")
    return DenseSizes(r.int("ff", min=1))


@dataclass(frozen=True)
class ZosuraxConfig:
    architecture: str
    vocab: int
    width: int
    norm_eps: float
    layers: tuple
    loop: Loop | None

    @classmethod
    def from_dict(cls, raw: dict, where: str = "config.json") -> "ZosuraxConfig":
        r = ConfigReader(raw, where)
        layers_raw = r.any("layers")
        if not (isinstance(layers_raw, list) and layers_raw):
            raise ConfigError(f"{where}: 'layers' must be a non-empty list")
        layers = []
        for i, lr in enumerate(layers_raw):
            w = f"{where}: layers[{i}]"
            l = ConfigReader(lr, w)
            kind = l.str("type")
            layers.append(ZosuraxLayer(kind, _mixer(kind, l.any("mixer"), f"{w}.mixer"), _mlp(l.any("mlp"), f"{w}.mlp")))
        loop = None
        if r.any("loop") is not None:
            lp = ConfigReader(r.any("loop"), f"{where}: loop")
            loop = Loop(lp.int("start", min=0), lp.int("stop", min=0), lp.int("times", min=1))
            if not loop.start <= loop.stop <= len(layers):
                raise ConfigError(f"{where}: loop: 0 <= start <= stop <= {len(layers)} layers, got {loop.start}, {loop.stop}")
        norm = ConfigReader(r.any("norm"), f"{where}: norm")
        return cls(architecture=r.str("architecture", "Zosurax"), vocab=r.int("vocab", min=1), width=r.int("width", min=1),
                   norm_eps=norm.float("eps", positive=True), layers=tuple(layers), loop=loop)

    def run_order(self) -> list:
        """[(layer, pass)]: the layers in the order they run; `pass` is the number of the loop's pass in front of whose
        first layer the entry stands, else None."""
        L, lp = len(self.layers), self.loop
        if lp is None or lp.stop == lp.start:
            return [(i, None) for i in range(L)]
        order = [(i, None) for i in range(lp.start)]
        for p in range(lp.times):
            order += [(i, p if i == lp.start else None) for i in range(lp.start, lp.stop)]
        return order + [(i, None) for i in range(lp.stop, L)]

    # what every engine front end asks of a configuration
    @property
    def vocab_size(self) -> int:
        return self.vocab

    @property
    def hidden_size(self) -> int:
        return self.width

    eos_token_id = None
    max_position_embeddings = None

    def to_json_dict(self) -> dict:
        layers = []
        for l in self.layers:
            m = l.mixer
            mixer = {"dim": m.dim, "heads": m.heads, "vdim": m.vdim}
            if l.type != "hgrn2":
                mixer.update(kv_heads=m.kv_heads, scale=m.scale)
                if m.rot is not None:
                    mixer["rot"] = {"base": m.rot.base, "dims": m.rot.dims}
            layers.append({"mixer": mixer, "mlp": None if l.mlp is None else {"ff": l.mlp.ff, "kind": "dense"}, "type": l.type})
        out = {"architecture": self.architecture, "layers": layers, "norm": {"eps": self.norm_eps}, "vocab": self.vocab,
               "width": self.width}
        if self.loop is not None:
            out["loop"] = {"start": self.loop.start, "stop": self.loop.stop, "times": self.loop.times}
        return out

    def num_parameters(self) -> int:
        from ..models.registry import expected_tensors
        n = 0
        for spec in expected_tensors(self).values():
            if spec.optional:
                continue
            k = 1
            for s in spec.shape:
                k *= s
            n += k
        return n
