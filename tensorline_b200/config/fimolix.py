"""`FimolixConfig`: the config.json of a Fimolix decoder, typed and validated.

The file is nested: `layers` lists the layers, each with its `type` (which mixer: "attention", two maps a head whose difference
is taken, or "latent_attention"), the mixer's sizes under `mixer` and its feed-forward under `mlp` (null: none; `kind` "dense");
`norm.eps`, `vocab` and `width` are the model's.  A latent attention with `kv_from` reads the latents that layer `kv_from` keeps.
A key the design always has is required and every error names its key.
"""
from __future__ import annotations

from dataclasses import dataclass

from .base import ConfigError, ConfigReader


@dataclass(frozen=True)
class Rotation:
    base: float
    dims: int


@dataclass(frozen=True)
class DifferentialSizes:
    heads: int
    kv_heads: int
    dim: int
    vdim: int
    conv: int
    scale: float
    softcap: float
    diff: float


@dataclass(frozen=True)
class LatentSizes:
    heads: int
    dim: int
    rot_dim: int
    vdim: int
    kv_rank: int
    scale: float
    window: int
    rot: Rotation
    kv_from: int | None


@dataclass(frozen=True)
class DenseSizes:
    ff: int


@dataclass(frozen=True)
class FimolixLayer:
    type: str
    mixer: object
    mlp: DenseSizes | None


def _mixer(kind: str, raw, where: str):
    if not isinstance(raw, dict):
        raise ConfigError(f"{where}: 'mixer' must be an object")
    r = ConfigReader(raw, where)
    if kind == "attention":
        heads, kv = r.int("heads", min=1), r.int("kv_heads", min=1)
        if heads % kv:
            raise ConfigError(f"{where}: 'heads' {heads} is not a multiple of 'kv_heads' {kv}")
        return DifferentialSizes(heads, kv, r.int("dim", min=1), r.int("vdim", min=1), r.int("conv", min=1), r.float("scale", positive=True),
                                 r.float("softcap", positive=True), r.float("diff"))
    if kind == "latent_attention":
        rot_dim = r.int("rot_dim", min=0)
        rr = ConfigReader(r.any("rot"), f"{where}.rot")
        rot = Rotation(rr.float("base", positive=True), rr.int("dims", min=0))
        if rot.dims % 2 or rot.dims > rot_dim:
            raise ConfigError(f"{where}.rot: 'dims' {rot.dims} must be even and at most 'rot_dim' {rot_dim}")
        mask = ConfigReader(r.any("mask"), f"{where}.mask")
        return LatentSizes(r.int("heads", min=1), r.int("dim", min=1), rot_dim, r.int("vdim", min=1), r.int("kv_rank", min=1),
                           r.float("scale", positive=True), mask.int("size", min=1), rot, r.int("kv_from", None, min=0))
    raise ConfigError(f"{where}: layer type {kind!r} is not one of 'attention', 'latent_attention'")


def _mlp(raw, where: str):
    if raw is None:
        return None
    r = ConfigReader(raw, where)
    kind = r.str("kind")
    if kind != "dense":
        raise ConfigError(f"{where}: feed-forward kind {kind!r} is not 'dense'")
    return DenseSizes(r.int("ff", min=1))


def _check_sharing(layers, where: str) -> None:
    for i, l in enumerate(layers):
        m = l.mixer
        if l.type != "latent_attention" or m.kv_from is None:
            continue
        w = f"{where}: layers[{i}].mixer"
        if m.kv_from >= i:
            raise ConfigError(f"{w}: 'kv_from' {m.kv_from} must name an earlier layer")
        src = layers[m.kv_from]
        if src.type != "latent_attention" or src.mixer.kv_from is not None:
            raise ConfigError(f"{w}: 'kv_from' {m.kv_from} must name a latent attention with a latent of its own")
        if (src.mixer.kv_rank, src.mixer.rot_dim, src.mixer.rot) != (m.kv_rank, m.rot_dim, m.rot):
            raise ConfigError(f"{w}: 'kv_rank', 'rot_dim' and 'rot' must be those of layer {m.kv_from}, whose latents it reads")


@dataclass(frozen=True)
class FimolixConfig:
    architecture: str
    vocab: int
    width: int
    norm_eps: float
    layers: tuple

    @classmethod
    def from_dict(cls, raw: dict, where: str = "config.json") -> "FimolixConfig":
        r = ConfigReader(raw, where)
        layers_raw = r.any("layers")
        if not (isinstance(layers_raw, list) and layers_raw):
            raise ConfigError(f"{where}: 'layers' must be a non-empty list")
        layers = []
        for i, lr in enumerate(layers_raw):
            w = f"{where}: layers[{i}]"
            l = ConfigReader(lr, w)
            kind = l.str("type")
            layers.append(FimolixLayer(kind, _mixer(kind, l.any("mixer"), f"{w}.mixer"), _mlp(l.any("mlp"), f"{w}.mlp")))
        _check_sharing(layers, where)
        norm = ConfigReader(r.any("norm"), f"{where}: norm")
        return cls(architecture=r.str("architecture", "Fimolix"), vocab=r.int("vocab", min=1), width=r.int("width", min=1),
                   norm_eps=norm.float("eps", positive=True), layers=tuple(layers))

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
            if l.type == "attention":
                mixer = {"conv": m.conv, "diff": m.diff, "dim": m.dim, "heads": m.heads, "kv_heads": m.kv_heads, "scale": m.scale,
                         "softcap": m.softcap, "vdim": m.vdim}
            else:
                mixer = {"dim": m.dim, "heads": m.heads, "kv_rank": m.kv_rank, "mask": {"size": m.window},
                         "rot": {"base": m.rot.base, "dims": m.rot.dims}, "rot_dim": m.rot_dim, "scale": m.scale, "vdim": m.vdim}
                if m.kv_from is not None:
                    mixer["kv_from"] = m.kv_from
            layers.append({"mixer": mixer, "mlp": None if l.mlp is None else {"ff": l.mlp.ff, "kind": "dense"}, "type": l.type})
        return {"architecture": self.architecture, "layers": layers, "norm": {"eps": self.norm_eps}, "vocab": self.vocab,
                "width": self.width}

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
