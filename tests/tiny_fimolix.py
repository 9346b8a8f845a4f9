"""Tiny Fimolix configurations of the tests and a helper that writes their model folders.

F1 to F6 differ in every size and option: a layer that reads another's latents through a wider window than the owner's, through a
narrower one, several readers of one layer, owners that nobody reads; grouped and ungrouped heads, value heads wider and narrower
than two maps, convolutions of one to six taps, lambdas of either sign, caps that most scores stay far below and caps that they
reach; layers without a feed-forward; head sizes that are no multiples of 16, odd ones, a single head; widths that are multiples
of nothing; latents wider than the tensor-core kernels take.  The attention scores are spread so that a softmax is decided by few
keys, so that a wrong key shows.
"""
from __future__ import annotations

import tempfile
from pathlib import Path

import torch

from tensorline_b200.config.fimolix import FimolixConfig
from tensorline_b200.models import expected_tensors
from tensorline_b200.weights import write_random_model
from tensorline_b200.weights.safetensors_io import SafetensorsFile, write_safetensors


def _mlp(ff):
    return None if ff is None else {"ff": ff, "kind": "dense"}


def _dif(heads, kv, dim, vdim, scale, cap, diff, conv, ff=None):
    return {"type": "attention", "mlp": _mlp(ff), "mixer": {"conv": conv, "diff": diff, "dim": dim, "heads": heads, "kv_heads": kv,
                                                             "scale": scale, "softcap": cap, "vdim": vdim}}


def _lat(heads, dim, rot, vdim, rank, window, scale, ff=None, kv_from=None):
    m = {"dim": dim, "heads": heads, "kv_rank": rank, "mask": {"size": window}, "rot": {"base": rot[0], "dims": rot[1]},
         "rot_dim": rot[1], "scale": scale, "vdim": vdim}
    if kv_from is not None:
        m["kv_from"] = kv_from
    return {"type": "latent_attention", "mlp": _mlp(ff), "mixer": m}


def _model(vocab, width, eps, layers):
    return {"architecture": "Fimolix", "layers": layers, "norm": {"eps": eps}, "vocab": vocab, "width": width}


# the reader's window is wider than the owner's: the owner's pages must stay for it
F1 = _model(131, 48, 1e-6, [
    _lat(3, 8, (1000.0, 4), 12, 20, 9, 0.5, 40), _dif(6, 2, 8, 24, 0.6, 3.0, 0.3, 3, 56), _lat(5, 12, (1000.0, 4), 8, 20, 37, 0.4, None, 0),
    _dif(4, 1, 12, 16, 0.5, 30.0, -0.2, 4), _lat(2, 6, (50.0, 6), 10, 26, 5, 0.6, 24),
])
# narrower readers, two of them, the first layer a pair of maps behind a convolution of one tap
F2 = _model(90, 72, 1e-5, [
    _dif(3, 3, 16, 40, 0.4, 2.0, 0.8, 1, 48), _lat(4, 16, (10000.0, 8), 24, 40, 50, 0.35, 56), _lat(7, 5, (10000.0, 8), 9, 40, 11, 0.5, 24, 1),
    _dif(2, 1, 8, 8, 0.7, 50.0, 0.5, 6, None), _lat(4, 16, (10000.0, 8), 16, 40, 50, 0.3, None, 1),
])
# odd head sizes, single heads, a width that is a multiple of nothing
F3 = _model(64, 33, 1e-6, [_dif(1, 1, 5, 7, 0.8, 4.0, 0.1, 2, 20), _lat(1, 7, (30.0, 2), 5, 11, 3, 0.7), _dif(3, 1, 7, 21, 0.6, 1.5, 0.9, 5, 18),
                           _lat(3, 3, (30.0, 2), 9, 11, 1, 0.9, 30, 1)])
# sizes that the tensor-core kernels take, for prompts of hundreds of tokens; more than sixteen rows a key/value head
F4 = _model(300, 160, 1e-5, [
    _dif(18, 2, 32, 64, 0.25, 12.0, 0.6, 4, 96), _lat(6, 32, (5000.0, 16), 32, 48, 96, 0.2, 128), _dif(4, 2, 64, 128, 0.18, 8.0, 0.4, 3, 64),
    _lat(20, 24, (5000.0, 16), 16, 48, 130, 0.25, None, 1), _dif(2, 2, 128, 64, 0.12, 20.0, 0.5, 2),
])
# latents wider than the tensor-core attention takes, and wider than 512
F5 = _model(77, 40, 1e-5, [_lat(2, 16, (100.0, 16), 12, 260, 21, 0.12, 24), _dif(2, 2, 4, 8, 0.9, 6.0, 0.2, 3), _lat(3, 8, (100.0, 24), 8, 516, 12, 0.12),
                           _lat(1, 9, (100.0, 16), 6, 260, 30, 0.15, 16, 0)])
# no latent at all, every layer without a feed-forward
F6 = _model(101, 52, 1e-5, [_dif(5, 5, 8, 16, 0.7, 5.0, 0.0, 4), _dif(5, 1, 24, 12, 0.5, 9.0, 0.7, 2)])
CONFIGS = {"F1": F1, "F2": F2, "F3": F3, "F4": F4, "F5": F5, "F6": F6}
PAGE_SIZE = {"F1": 8, "F2": 16, "F3": 4, "F4": 16, "F5": 16, "F6": 32}


def write_tiny_fimolix(name: str, folder=None, seed: int = 0, config: dict | None = None, std: float = 0.12) -> Path:
    cfg = FimolixConfig.from_dict(config or CONFIGS[name])
    folder = Path(folder) if folder is not None else Path(tempfile.mkdtemp(prefix=f"tiny_{name}_"))
    write_random_model(folder, cfg, expected_tensors(cfg), seed=seed, std=std, norm_std=0.2)
    f = SafetensorsFile(folder / "model.safetensors")
    tensors = {n: f.tensor(n).clone() for n in f.names()}
    f.close()
    g = torch.Generator().manual_seed(seed + 31)
    for n, t in tensors.items():
        if n.endswith((".q.norm", ".k.norm", ".dkv.norm")):
            tensors[n] = (0.9 + 0.5 * torch.rand(t.shape, generator=g)).to(t.dtype)
        elif n.endswith((".norm1", ".norm2", "final.norm")):   # stored around zero
            tensors[n] = (0.3 * torch.randn(t.shape, generator=g)).to(t.dtype)
        elif n.endswith(".conv"):                              # every tap counts, the current token most
            w = 0.5 * torch.randn(t.shape, generator=g)
            w[:, -1] += 1.0
            tensors[n] = w.to(t.dtype)
        elif n.endswith((".lq1", ".lk1", ".lq2", ".lk2")):
            tensors[n] = (0.9 * t.shape[0] ** -0.25 * torch.randn(t.shape, generator=g)).to(t.dtype)
        elif n.endswith(".sink"):
            tensors[n] = (1.0 + torch.randn(t.shape, generator=g)).to(t.dtype)
        elif n.endswith(".mix.g"):
            tensors[n] = (t.float() * 3.0).to(t.dtype)
        elif n == "embed":
            tensors[n] = (t.float() * 8.0).to(t.dtype)
    write_safetensors(folder / "model.safetensors", tensors, {"format": "pt"})
    return folder
