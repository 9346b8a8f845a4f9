"""A plain, slow implementation of the Zosurax decoder, used only as the oracle of the tests.

Whole sequences, no cache, no batching, one function per mechanism, float64 on the CPU, written from the design's
equations in the notation below; it shares no code with the package under test.

Notation.  Tokens t = 0, 1, ... of one sequence; W: matrices stored [out, in], applied as W h; sig = the logistic function;
u(v) = v / sqrt(mean(v^2) + eps) and n(v; w) = u(v) * w with the model's eps.

  start      e_t = embed[tok_t];  x = e
  passes     layers loop.start .. loop.stop - 1 run loop.times times in a row with the same weights; in front of pass r > 0
             x += e, then in front of every pass x += loop.step[r]
  layer      x += ls1 * mixer(shifted(n(x; norm1)));  x += ls2 * ff(n(x; norm2)), the second only where there is one
  shifted    h_t + (h_(t-1) - h_t) * shift, h_(-1) = 0
  hgrn2      q = silu(Wq h), v = Wv h per head; f = lower + (1 - lower) sig(Wf h + bf) per head and channel;
             S_t = diag(f_t) S_(t-1) + (1 - f_t) v_t^T, S before the start = 0;  o_t = S_t^T q_t;
             y = Wo (n(o; norm) per head, side by side)
  attention  q = Wq h, k = Wk h, v = Wv h; every head of q and k: n(.; q.norm) or n(.; k.norm), then turned (pairs i, i + dims/2);
             query head a reads KV head a // (heads / kv_heads); softmax over j <= t of scale q_t . k_j; y = Wo (heads side by side)
  attention_2  as attention, but q and k are turned first (pairs 2i, 2i + 1) and then through u;
             P_a(t, j) the softmax of head a; P'_a = sum_b talk[a, b] P_b; head a's output sum_j P'_a(t, j) v_j
  turning    angle t * base^(-2i / dims) for pair i < dims / 2: (p, r) -> (p cos - r sin, r cos + p sin)
  ff         Wdown relu(Wup h)^2
  output     logits = embed n(x; final.norm)
"""
from __future__ import annotations

import json
from pathlib import Path

import torch

from tests.plain.qwen2_plain import read_safetensors

F64 = torch.float64


def unit(v, eps):
    return v / torch.sqrt((v * v).mean(-1, keepdim=True) + eps)


def normed(v, w, eps):
    return unit(v, eps) * w


def sig(z):
    return 1.0 / (1.0 + torch.exp(-z))


def silu(z):
    return z * sig(z)


def shifted(h, mu):
    """h [T, W]: every row moved towards the row in front of it (zeros in front of the first)."""
    before = torch.cat([torch.zeros_like(h[:1]), h[:-1]])
    return h + (before - h) * mu


def turn(x, rot, pairing):
    """x [T, heads, d]: the first rot["dims"] dimensions of every head turned by the token's position."""
    x = x.clone()
    dims = int(rot["dims"])
    where = torch.arange(x.shape[0], dtype=F64).view(-1, 1)
    for i in range(dims // 2):
        a = where * float(rot["base"]) ** (-2.0 * i / dims)
        first, second = (i, i + dims // 2) if pairing == "half" else (2 * i, 2 * i + 1)
        p, r = x[..., first].clone(), x[..., second].clone()
        x[..., first] = p * torch.cos(a) - r * torch.sin(a)
        x[..., second] = r * torch.cos(a) + p * torch.sin(a)
    return x


def softmax_weights(q, k, scale):
    """P [H, T, T] of causal attention, q [T, H, d], k [T, G, d]."""
    T, H = q.shape[:2]
    g = H // k.shape[1]
    hidden = torch.ones(T, T, dtype=torch.bool).triu(1)
    return torch.stack([torch.softmax(((q[:, a] @ k[:, a // g].T) * scale).masked_fill(hidden, float("-inf")), -1) for a in range(H)])


def apply_weights(P, v):
    """[T, H * dv]: head a's weights P[a] over the values of its own KV head, v [T, G, dv]."""
    g = P.shape[0] // v.shape[1]
    return torch.cat([P[a] @ v[:, a // g] for a in range(P.shape[0])], dim=-1)


def _qkv(h, w, c):
    T = h.shape[0]
    H, G, d, dv = c["heads"], c["kv_heads"], c["dim"], c["vdim"]
    return (h @ w["q"].T).view(T, H, d), (h @ w["k"].T).view(T, G, d), (h @ w["v"].T).view(T, G, dv)


def attention(h, w, c, eps):
    q, k, v = _qkv(h, w, c)
    q, k = normed(q, w["q.norm"], eps), normed(k, w["k.norm"], eps)
    if c.get("rot"):
        q, k = turn(q, c["rot"], "half"), turn(k, c["rot"], "half")
    return apply_weights(softmax_weights(q, k, c["scale"]), v) @ w["o"].T


def mixed_weights(P, talk):
    return torch.einsum("ab,btj->atj", talk, P)


def attention_2(h, w, c, eps):
    q, k, v = _qkv(h, w, c)
    if c.get("rot"):
        q, k = turn(q, c["rot"], "pairs"), turn(k, c["rot"], "pairs")
    q, k = unit(q, eps), unit(k, eps)
    return apply_weights(mixed_weights(softmax_weights(q, k, c["scale"]), w["talk"]), v) @ w["o"].T


def forget_gates(h, w, c):
    lower = w["lower"]
    return (lower + (1.0 - lower) * sig(h @ w["f"].T + w["f.b"])).view(h.shape[0], c["heads"], c["dim"])


def decayed_memory(q, f, v):
    """o [T, H, dv] of S_t = diag(f_t) S_(t-1) + (1 - f_t) v_t^T, o_t = S_t^T q_t;  q, f [T, H, d], v [T, H, dv]."""
    T, H, d = q.shape
    S = torch.zeros(H, d, v.shape[2], dtype=F64)
    out = []
    for t in range(T):
        S = f[t][:, :, None] * S + (1.0 - f[t])[:, :, None] * v[t][:, None, :]
        out.append(torch.einsum("hde,hd->he", S, q[t]))
    return torch.stack(out)


def hgrn2(h, w, c, eps):
    T = h.shape[0]
    q = silu(h @ w["q"].T).view(T, c["heads"], c["dim"])
    v = (h @ w["v"].T).view(T, c["heads"], c["vdim"])
    o = decayed_memory(q, forget_gates(h, w, c), v)
    return normed(o, w["norm"], eps).reshape(T, -1) @ w["o"].T


def relu_squared_ff(h, w):
    return torch.clamp(h @ w["up"].T, min=0.0) ** 2 @ w["down"].T


MIXERS = {"hgrn2": hgrn2, "attention": attention, "attention_2": attention_2}


def order(config):
    """[(layer, number of the pass that begins in front of it or None)] of one forward run."""
    n, loop = len(config["layers"]), config.get("loop")
    if not loop or loop["stop"] <= loop["start"]:
        return [(i, None) for i in range(n)]
    out = [(i, None) for i in range(loop["start"])]
    for r in range(loop["times"]):
        out += [(i, r if i == loop["start"] else None) for i in range(loop["start"], loop["stop"])]
    return out + [(i, None) for i in range(loop["stop"], n)]


def sub(w, prefix):
    return {k[len(prefix) + 1:]: v for k, v in w.items() if k.startswith(prefix + ".")}


def layer_step(x, w, layer, eps):
    h = shifted(normed(x, w["norm1"], eps), w["shift"])
    x = x + w["ls1"] * MIXERS[layer["type"]](h, sub(w, "mix"), layer["mixer"], eps)
    if layer["mlp"] is not None:
        x = x + w["ls2"] * relu_squared_ff(normed(x, w["norm2"], eps), sub(w, "mlp"))
    return x


def forward(config: dict, weights: dict, tokens, per_layer: bool = False):
    """Logits [T, vocab] of one whole sequence (and the residual stream after every layer run)."""
    w = {k: (v.to(F64) if v.is_floating_point() else v) for k, v in weights.items()}
    eps = float(config["norm"]["eps"])
    start = w["embed"][list(tokens)]
    x = start
    streams = []
    for i, r in order(config):
        if r is not None:
            if r > 0:
                x = x + start
            x = x + w["loop.step"][r]
        x = layer_step(x, sub(w, f"l{i}"), config["layers"][i], eps)
        streams.append(x)
    logits = normed(x, w["final.norm"], eps) @ w["embed"].T
    return (logits, torch.stack(streams)) if per_layer else logits


def load(folder):
    folder = Path(folder)
    return json.loads((folder / "config.json").read_text()), read_safetensors(folder / "model.safetensors")


class PlainZosurax:
    def __init__(self, folder):
        self.cfg, self.weights = load(folder)


def logits_of(model: PlainZosurax, tokens, layers: list | None = None):
    """Logits [T, vocab]; `layers`, if given, receives the residual stream after every layer run."""
    out, streams = forward(model.cfg, model.weights, tokens, per_layer=True)
    if layers is not None:
        layers.extend(streams)
    return out


def greedy_generate(model: PlainZosurax, prompt, n: int) -> list:
    seq, out = list(prompt), []
    for _ in range(n):
        tok = int(torch.argmax(logits_of(model, seq)[-1]))
        out.append(tok)
        seq.append(tok)
    return out
