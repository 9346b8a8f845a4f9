"""A plain, slow implementation of the Fimolix decoder, used only as the oracle of the tests.

Whole sequences, no cache, no batching, one function per mechanism, float64 on the CPU, written from the design's
equations in the notation below; it shares no code with the package under test.

Notation.  Tokens t = 0, 1, ... of one sequence; W: matrices stored [out, in], applied as W h; sig = the logistic function;
u(v) = v / sqrt(mean(v^2) + eps) with the model's eps.

  start      x_t = embed[tok_t]
  layer      x <- x + u(mixer(x)) (1 + norm1);   x <- x + u(ff(x)) (1 + norm2)   (the second only where the layer has an ff)
  ff         Wdown act(Wup h),  act(z) = z (1 + tanh(sqrt(2 / pi) (z + 0.044715 z^3))) / 2
  pair of maps ("attention")
             P = Wq h, Wk h, Wv h, each channel c through y_t = sum_j w[c, j] P_(t - taps + 1 + j), zeros before the start;
             a head of q is [map 1 | map 2] of dim each, so is a head of k; every map of q and k: u(.) * norm;
             query head a reads KV head a // (heads / kv_heads);  s = cap tanh(scale q . k / cap), every j <= t, softmax,
             a1 and a2 the two maps' sums over the same v;  lambda = exp(lq1 . lk1) - exp(lq2 . lk2) + diff;
             o = u(a1 - lambda a2) (1 - diff);  y = Wo (heads side by side)
  latent     q = Wq h, per head [dim plain | rot_dim turned];  Wdkv h = [kv_rank | rot_dim]: c = u(first) * dkv.norm, r = the rest,
             turned, one for all heads, or both from layer kv_from;  k_a = Wuk_a c, v_a = Wuv_a c;
             s_tj = scale (q_plain . k_a(j) + q_turned . r(j)), 0 <= t - j < size;
             o_t = sum_j exp(s_tj) v_a(j) / (sum_j exp(s_tj) + exp(sink_a));  head a times sig(Wg h)_a;  y = Wo (heads side by side)
  turning    pairs (2i, 2i + 1), i < dims / 2, angle t * base^(-2i / dims):  (u, v) -> (u cos - v sin, v cos + u sin)
  output     logits = embed (u(x) (1 + final.norm))
"""
from __future__ import annotations

import json
import math
from pathlib import Path

import torch

from tests.plain.qwen2_plain import read_safetensors

F64 = torch.float64


def unit(v, eps):
    return v / torch.sqrt((v * v).mean(-1, keepdim=True) + eps)


def one_plus_norm(v, w, eps):
    return unit(v, eps) * (1.0 + w)


def sig(z):
    return 1.0 / (1.0 + torch.exp(-z))


def gelu(z):
    return 0.5 * z * (1.0 + torch.tanh(math.sqrt(2.0 / math.pi) * (z + 0.044715 * z ** 3)))


def feed_forward(h, w):
    return gelu(h @ w["up"].T) @ w["down"].T


def short_conv(x, taps_w):
    """x [T, C], taps_w [C, taps]: the last tap meets the current token."""
    taps = taps_w.shape[1]
    padded = torch.cat([torch.zeros(taps - 1, x.shape[1], dtype=x.dtype), x])
    return sum(taps_w[:, j] * padded[j:j + x.shape[0]] for j in range(taps))


def capped(s, cap):
    return cap * torch.tanh(s / cap)


def causal(T):
    return torch.ones(T, T, dtype=torch.bool).tril()


def head_norm(o, eps):
    return unit(o, eps)


def mix_weight(w, diff):
    return float(torch.exp((w["lq1"] * w["lk1"]).sum()) - torch.exp((w["lq2"] * w["lk2"]).sum()) + diff)


def differential_attention(h, w, c, eps):
    T = h.shape[0]
    H, G, d, dv = c["heads"], c["kv_heads"], c["dim"], c["vdim"]
    q, k, v = (short_conv(h @ w[n].T, w[n + ".conv"]) for n in ("q", "k", "v"))
    q = unit(q.view(T, H, 2, d), eps) * w["q.norm"]
    k = unit(k.view(T, G, 2, d), eps) * w["k.norm"]
    v = v.view(T, G, dv)
    lam = mix_weight(w, c["diff"])
    o = torch.zeros(T, H, dv, dtype=F64)
    for a in range(H):
        kv = a // (H // G)
        maps = []
        for m in range(2):
            s = capped((q[:, a, m] @ k[:, kv, m].T) * c["scale"], c["softcap"])
            maps.append(torch.softmax(s.masked_fill(~causal(T), float("-inf")), -1) @ v[:, kv])
        o[:, a] = head_norm(maps[0] - lam * maps[1], eps) * (1.0 - c["diff"])
    return o.reshape(T, H * dv) @ w["o"].T


def turn_pairs(x, rot):
    """x [T, ..., d]: dimensions (2i, 2i + 1) below rot.dims turned by the token's position."""
    x, T, dims = x.clone(), x.shape[0], rot["dims"]
    where = torch.arange(T, dtype=F64).view(T, *([1] * (x.dim() - 2)))
    for i in range(dims // 2):
        a = where * float(rot["base"]) ** (-2.0 * i / dims)
        p, q = x[..., 2 * i].clone(), x[..., 2 * i + 1].clone()
        x[..., 2 * i] = p * torch.cos(a) - q * torch.sin(a)
        x[..., 2 * i + 1] = q * torch.cos(a) + p * torch.sin(a)
    return x


def latent_of(h, w, c, eps):
    """What a layer caches of every token: the latent and the turned key part."""
    down = h @ w["dkv"].T
    return unit(down[:, :c["kv_rank"]], eps) * w["dkv.norm"], turn_pairs(down[:, c["kv_rank"]:], c["rot"])


def window(T, size):
    t = torch.arange(T)
    back = t[:, None] - t[None]
    return (back >= 0) & (back < size)


def softmax_with_sink(s, sink):
    top = torch.clamp(s.max(-1, keepdim=True).values, min=float(sink))
    e = torch.exp(s - top)
    return e / (e.sum(-1, keepdim=True) + torch.exp(sink - top))


def head_gates(h, w):
    return sig(h @ w["g"].T)


def latent_attention(h, w, c, kept, eps):
    T = h.shape[0]
    H, d, dv = c["heads"], c["dim"], c["vdim"]
    q = (h @ w["q"].T).view(T, H, d + c["rot_dim"])
    turned = turn_pairs(q[..., d:], c["rot"])
    lat, r = kept
    k = (lat @ w["uk"].T).view(T, H, d)
    v = (lat @ w["uv"].T).view(T, H, dv)
    o = torch.zeros(T, H, dv, dtype=F64)
    for a in range(H):
        s = (q[:, a, :d] @ k[:, a].T + turned[:, a] @ r.T) * c["scale"]
        o[:, a] = softmax_with_sink(s.masked_fill(~window(T, c["mask"]["size"]), float("-inf")), w["sink"][a]) @ v[:, a]
    return (o * head_gates(h, w)[..., None]).reshape(T, H * dv) @ w["o"].T


def sub(w, prefix):
    return {k[len(prefix) + 1:]: v for k, v in w.items() if k.startswith(prefix + ".")}


def source_layer(c, i):
    """The layer whose latent layer i reads."""
    return i if c.get("kv_from") is None else c["kv_from"]


def forward(config: dict, weights: dict, tokens, per_layer: bool = False):
    """Logits [T, vocab] of one whole sequence (and the residual stream after every layer)."""
    w = {k: (v.to(F64) if v.is_floating_point() else v) for k, v in weights.items()}
    eps = float(config["norm"]["eps"])
    x = w["embed"][list(tokens)]
    kept, streams = {}, []
    for i, layer in enumerate(config["layers"]):
        lw, c = sub(w, f"l{i}"), layer["mixer"]
        mw = sub(lw, "mix")
        if layer["type"] == "attention":
            y = differential_attention(x, mw, c, eps)
        else:
            j = source_layer(c, i)
            if c.get("kv_from") is None:
                kept[i] = latent_of(x, mw, c, eps)
            y = latent_attention(x, mw, c, kept[j], eps)
        x = x + one_plus_norm(y, lw["norm1"], eps)
        if layer["mlp"] is not None:
            x = x + one_plus_norm(feed_forward(x, sub(lw, "mlp")), lw["norm2"], eps)
        streams.append(x)
    logits = one_plus_norm(x, w["final.norm"], eps) @ w["embed"].T
    return (logits, torch.stack(streams)) if per_layer else logits


def load(folder):
    folder = Path(folder)
    return json.loads((folder / "config.json").read_text()), read_safetensors(folder / "model.safetensors")


class PlainFimolix:
    def __init__(self, folder):
        self.cfg, self.weights = load(folder)


def logits_of(model: PlainFimolix, tokens, layers: list | None = None):
    """Logits [T, vocab]; `layers`, if given, receives the residual stream after every layer."""
    out, streams = forward(model.cfg, model.weights, tokens, per_layer=True)
    if layers is not None:
        layers.extend(streams)
    return out


def greedy_generate(model: PlainFimolix, prompt, n: int) -> list:
    seq, out = list(prompt), []
    for _ in range(n):
        tok = int(torch.argmax(logits_of(model, seq)[-1]))
        out.append(tok)
        seq.append(tok)
    return out
