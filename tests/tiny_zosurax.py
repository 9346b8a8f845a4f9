"""Tiny Zosurax configurations of the tests and a helper that writes their model folders.

Z1 to Z6 differ in every size and option: loops of one to four passes over the first, middle or last layers, over layers
without a feed-forward only, and no loop; grouped and ungrouped heads, value heads wider and narrower than query heads, head
sizes that are no multiples of 16, odd ones, seventeen heads (one more than a group of sixteen in the mix) and a single one;
rotations over all, part or none of a head; recurrent heads of 5 to 128 dimensions; widths that are multiples of nothing.  The
attention scores are spread so that a softmax is decided by few keys, the forget gates lie near one so that a lost or stale
state shows many tokens later, the shift, the layer scales and the heads' mix are of order one.
"""
from __future__ import annotations

import tempfile
from pathlib import Path

import torch

from tensorline_b200.config.zosurax import ZosuraxConfig
from tensorline_b200.models import expected_tensors
from tensorline_b200.weights import write_random_model
from tensorline_b200.weights.safetensors_io import SafetensorsFile, write_safetensors


def _rec(heads, dim, vdim, ff=None):
    return {"type": "hgrn2", "mixer": {"dim": dim, "heads": heads, "vdim": vdim}, "mlp": _mlp(ff)}


def _att(kind, heads, kv, dim, vdim, scale, rot=None, ff=None):
    m = {"dim": dim, "heads": heads, "kv_heads": kv, "scale": scale, "vdim": vdim}
    if rot is not None:
        m["rot"] = {"base": rot[0], "dims": rot[1]}
    return {"type": "attention" if kind == 1 else "attention_2", "mixer": m, "mlp": _mlp(ff)}


def _mlp(ff):
    return None if ff is None else {"ff": ff, "kind": "dense"}


def _model(vocab, width, eps, layers, loop=None):
    out = {"architecture": "Zosurax", "layers": layers, "norm": {"eps": eps}, "vocab": vocab, "width": width}
    if loop is not None:
        out["loop"] = dict(zip(("start", "stop", "times"), loop))
    return out


Z1 = _model(131, 48, 1e-6, [
    _rec(3, 8, 16), _att(1, 6, 2, 16, 24, 0.5, (100.0, 8), 40), _att(2, 4, 2, 8, 8, 1.1, (500.0, 8), 56), _rec(2, 16, 8, 24),
], (1, 3, 2))
Z2 = _model(90, 72, 1e-5, [
    _att(2, 5, 1, 24, 40, 0.5, (10000.0, 12), 48), _rec(2, 24, 12, 56), _att(1, 3, 3, 32, 16, 0.3, (1000.0, 32)),
], (0, 3, 3))
# no loop, nothing rotated, one head each, a recurrence of more than 32 and of more than 64 rows
Z3 = _model(77, 40, 1e-5, [_rec(1, 40, 24, 24), _att(1, 1, 1, 12, 12, 0.9), _att(2, 1, 1, 20, 8, 0.8), _rec(1, 72, 40)])
# a loop over layers without a feed-forward only (every pass piles up addends), odd head sizes, a width that is a multiple of nothing
Z4 = _model(64, 33, 1e-6, [_att(1, 2, 1, 7, 9, 0.9, (30.0, 6), 20), _rec(3, 5, 7), _att(2, 3, 3, 9, 7, 1.0, (50.0, 4)), _rec(2, 11, 3)], (1, 4, 4))
# seventeen heads in the mix, a loop of one pass at the end
Z5 = _model(101, 52, 1e-5, [_rec(5, 6, 10, 18), _att(1, 4, 1, 12, 6, 0.7, (1e6, 10)), _att(2, 17, 1, 8, 12, 1.2, (200.0, 6), 30)], (2, 3, 1))
# sizes that the tensor-core kernels take, for prompts of hundreds of tokens
Z6 = _model(300, 160, 1e-5, [
    _att(2, 20, 4, 128, 64, 0.12, (10000.0, 64), 96), _rec(4, 128, 64, 128), _att(1, 8, 2, 128, 128, 0.08, (50000.0, 128), 64),
    _att(2, 6, 6, 64, 128, 0.15, (5000.0, 64)),
], (0, 2, 2))
CONFIGS = {"Z1": Z1, "Z2": Z2, "Z3": Z3, "Z4": Z4, "Z5": Z5, "Z6": Z6}
PAGE_SIZE = {"Z1": 8, "Z2": 16, "Z3": 4, "Z4": 16, "Z5": 16, "Z6": 32}


def write_tiny_zosurax(name: str, folder=None, seed: int = 0, config: dict | None = None, std: float = 0.12) -> Path:
    cfg = ZosuraxConfig.from_dict(config or CONFIGS[name])
    folder = Path(folder) if folder is not None else Path(tempfile.mkdtemp(prefix=f"tiny_{name}_"))
    write_random_model(folder, cfg, expected_tensors(cfg), seed=seed, std=std, norm_std=0.2)
    f = SafetensorsFile(folder / "model.safetensors")
    tensors = {n: f.tensor(n).clone() for n in f.names()}
    f.close()
    g = torch.Generator().manual_seed(seed + 31)
    for n, t in tensors.items():
        if n.endswith(".talk"):                                # every head mostly keeps its own weights and takes of the others'
            tensors[n] = (torch.eye(t.shape[0]) + 0.4 * torch.randn(t.shape, generator=g)).to(t.dtype)
        elif n.endswith(".lower"):
            tensors[n] = (torch.rand(t.shape, generator=g) * 0.9).to(t.dtype)
        elif n.endswith(".f.b"):                               # forget gates near one: a far token still counts
            tensors[n] = (torch.rand(t.shape, generator=g) * 4.0 + 1.0).to(t.dtype)
        elif n.endswith(".f"):                                 # gates that move from token to token
            tensors[n] = (t.float() * 3.0).to(t.dtype)
        elif n.endswith(".shift"):
            tensors[n] = torch.rand(t.shape, generator=g).to(t.dtype)
        elif n.endswith((".q.norm", ".k.norm")):
            tensors[n] = (1.0 + 0.5 * torch.rand(t.shape, generator=g)).to(t.dtype)
        elif n.endswith((".up", ".mix.v")):
            tensors[n] = (t.float() * 2.0).to(t.dtype)
        elif n == "loop.step":
            tensors[n] = (t.float() * 3.0).to(t.dtype)
        elif n == "embed":
            tensors[n] = (t.float() * 4.0).to(t.dtype)
    write_safetensors(folder / "model.safetensors", tensors, {"format": "pt"})
    return folder
