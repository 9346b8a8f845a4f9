"""Differential attention (Ye et al., "Differential Transformer"): every head is two attention maps over the same values.

    q, k, v = Wq h, Wk h, Wv h              a head of q and k is [map 1 | map 2], `dim` each; query head a reads KV head a // (H / G)
    conv (optional): y[t, c] = sum_j w[c, j] u[t - taps + 1 + j, c] on every channel of q, k and v, zeros before the request's start
    RMS norm of every map of q and k over its dim, one weight for all heads and maps (optional)
    s_m = scale q_m . k_m, with `score_cap`: cap * tanh(s_m / cap);   a_m = softmax(s_m) v
    o = a_1 - lambda a_2,  lambda = exp(lq1 . lk1) - exp(lq2 . lk2) + init;   y = Wo [o / rms(o) * (1 - init)]

One run of the paged attention kernels serves both maps.  A key's two maps lie side by side in its page row, and map m of a query
is a row of its own that is zero outside the columns of map m: the kernels then see 2 H query heads over G key/value heads of one
size, so a key and a value are read once for both maps of all the heads that share them, and every option of those kernels
(window, sink, cap) is there.  The row is as wide as the wider of two maps and a value (`d`, padded to what the kernels take);
with 2 dim = vdim, the usual choice, nothing in the pages is padding.

`csrc/differential.cu` has the steps around it: convolution, norms, the query rows and the page write in one kernel in front (the
last taps - 1 projected rows of a request are its state, in the activation type), the difference and its norm in one behind.
Norms, scores, softmax, lambda and the difference are float32 in both engines.
"""
from __future__ import annotations

import torch

from .. import ops
from ..cache import PagedKV, SlotState
from .base import Part, Runtime, TensorSpec, register_mixer
from .linear import matmul, resolve

_NAMES = {"q": "q", "k": "k", "v": "v", "o": "o", "q_norm": "q.norm", "k_norm": "k.norm", "q_conv": "q.conv", "k_conv": "k.conv",
          "v_conv": "v.conv", "lq1": "lq1", "lk1": "lk1", "lq2": "lq2", "lk2": "lk2"}
MAPS = 2


@register_mixer("differential_attention")
class DifferentialAttention(Part):
    graph_capturable = True

    def __init__(self, rt: Runtime, hidden: int, num_heads: int, num_kv_heads: int, head_dim: int, v_head_dim: int, scale: float,
                 init: float, norm_eps: float, taps: int | None = None, qk_norm: bool = True, score_cap: float | None = None,
                 window: int | None = None, names: dict | None = None):
        """`taps` None: no convolution (one tap is a factor a channel, without state).  `init`: the constant part of lambda, also 1 - the outputs' factor.  `norm_eps`: of the q/k
        norms and of the outputs' norm."""
        super().__init__(rt)
        if num_heads % num_kv_heads:
            raise ValueError(f"{num_heads} query heads are not a multiple of {num_kv_heads} KV heads")
        if taps is not None and taps < 1:
            raise ValueError(f"a convolution of {taps} taps")
        d = max(MAPS * head_dim, v_head_dim)
        if not rt.exact:
            d = -(-d // 16) * 16                          # the bfloat16 attention kernels take multiples of 16
        self.hidden, self.H, self.G, self.dk, self.dv, self.d = hidden, num_heads, num_kv_heads, head_dim, v_head_dim, d
        self.has_conv, self.taps, self.init, self.eps, self.qk_norm = taps is not None, taps or 1, float(init), float(norm_eps), bool(qk_norm)
        self.C = (num_heads + num_kv_heads) * MAPS * head_dim + num_kv_heads * v_head_dim
        self.names = {**_NAMES, **(names or {})}
        # what `attention_kernels.attend` reads of a mixer
        self.nq, self.nkv, self.scale, self.window, self.score_cap, self.sink = MAPS * num_heads, num_kv_heads, float(scale), window, score_cap, None
        self.w_qkv = self.w_o = self.taps_w = self.q_norm = self.k_norm = None
        self.weight = 0.0                                 # lambda

    def cache_need(self):
        need = {"kv": PagedKV(self.G, self.d, self.window)}
        if self.taps > 1:
            need["rows"] = SlotState((self.taps - 1, self.C), "float32" if self.rt.exact else "bfloat16")
        return need

    def _heads(self):
        return (("q", self.H * MAPS * self.dk), ("k", self.G * MAPS * self.dk), ("v", self.G * self.dv))

    def expected_tensors(self, prefix):
        n = {k: f"{prefix}.{v}" for k, v in self.names.items()}
        out = {n[k]: TensorSpec((rows, self.hidden)) for k, rows in self._heads()}
        out[n["o"]] = TensorSpec((self.hidden, self.H * self.dv))
        if self.has_conv:
            out.update({n[k + "_conv"]: TensorSpec((rows, self.taps)) for k, rows in self._heads()})
        if self.qk_norm:
            out.update({n["q_norm"]: TensorSpec((self.dk,), init="ones"), n["k_norm"]: TensorSpec((self.dk,), init="ones")})
        out.update({n[k]: TensorSpec((self.dk,)) for k in ("lq1", "lk1", "lq2", "lk2")})
        return out

    def bind(self, weights, prefix):
        n = {k: f"{prefix}.{v}" for k, v in self.names.items()}
        self.w_qkv = self._compute_copy(torch.cat([weights[n[k]] for k, _ in self._heads()], dim=0))
        self.w_o = self._compute_copy(weights[n["o"]])
        if self.has_conv:
            self.taps_w = torch.cat([weights[n[k + "_conv"]] for k, _ in self._heads()], dim=0).contiguous()
        else:
            self.taps_w = torch.ones((self.C, 1), dtype=torch.bfloat16, device=self.w_o.device)
        if self.taps_w.dtype not in (torch.float32, torch.bfloat16):
            self.taps_w = self.taps_w.float()
        if self.qk_norm:
            self.q_norm, self.k_norm = weights[n["q_norm"]].float().contiguous(), weights[n["k_norm"]].float().contiguous()
        a, b = ((weights[n[q]].double() * weights[n[k]].double()).sum().exp() for q, k in (("lq1", "lk1"), ("lq2", "lk2")))
        self.weight = float(a - b) + self.init            # one number for the layer, made once

    def forward(self, h, ctx, cache):
        H, d = self.H, self.d
        h = resolve(h)
        T = h.shape[0]
        kv = cache["kv"]
        table = ctx.tables[kv.group]
        proj = resolve(matmul(h, self.w_qkv))
        q = torch.empty((T, H * MAPS * d), dtype=proj.dtype, device=proj.device)
        ops.conv_heads(proj, self.taps_w, cache["rows"].state if self.taps > 1 else None, ctx, table, ctx.page_size, q, kv.k, kv.v, nq=H,
                       nkv=self.G, maps=MAPS, dim=self.dk, dv=self.dv, q_norm=self.q_norm, k_norm=self.k_norm, eps=self.eps)
        a = torch.empty((T, H * MAPS * d), dtype=proj.dtype, device=proj.device)
        from . import attention_kernels
        attention_kernels.attend(self, q, a, ctx, kv, table)
        o = torch.empty((T, H * self.dv), dtype=proj.dtype, device=proj.device)
        ops.map_difference(a, o, H, self.dv, self.weight, self.eps, 1.0 - self.init)
        return matmul(o, self.w_o)
