"""The Zosurax decoder as a `ModelSpec`.

Every layer is a pre-norm block (plain RMS norms in float32) whose mixer reads its input shifted towards the previous token's
by a vector (`shift`) and whose sub-blocks' outputs join the stream times a vector each (`ls1`, `ls2`).  Three mixers: HGRN2
(a matrix memory per head whose forget gate decides what is written), grouped-query attention with weighted q/k norms in front
of a rotation of half pairs, and grouped-query attention with neighbouring pairs, q and k divided by their root mean square and
softmax weights that are mixed across the heads (`talk`) before they meet the values.  The feed-forward, where a layer has
one, is W_down relu(W_up h)^2.  `loop` runs a range of layers several times with the same weights, every pass with caches of
its own, the embedding's output added to the stream in front of every pass but the first and a learned vector
(`loop.step[pass]`) in front of every one.  The output head is the embedding table.  Tensor names: `embed`, `loop.step`,
`l<i>.norm1`, `l<i>.mix.*`, `l<i>.mlp.*`, `final.norm`, each tensor under its own name, biases with `.b`.
"""
from __future__ import annotations

from ..config.zosurax import ZosuraxConfig
from ..parts import PartSpec
from .spec import LayerSpec, ModelSpec, RunEntry

_ATTENTION_NAMES = {"q": "q", "k": "k", "v": "v", "o": "o", "q_norm": "q.norm", "k_norm": "k.norm", "head_mix": "talk"}


def describe_zosurax(cfg: ZosuraxConfig) -> ModelSpec:
    W, eps = cfg.width, cfg.norm_eps
    norm = PartSpec("rms_norm", {"dim": W, "eps": eps, "tensor": "", "cast_first": False})
    layers = []
    for i, layer in enumerate(cfg.layers):
        m = layer.mixer
        if layer.type == "hgrn2":
            mixer = PartSpec("hgrn2", {"hidden": W, "num_heads": m.heads, "head_dim": m.dim, "v_head_dim": m.vdim, "norm_eps": eps})
        else:
            talking = layer.type == "attention_2"
            position = PartSpec("none") if m.rot is None else PartSpec(
                "rotary_interleaved" if talking else "rotary_half", {"theta": m.rot.base, "rotary_dim": m.rot.dims})
            mixer = PartSpec("paged_attention", {
                "hidden": W, "num_heads": m.heads, "num_kv_heads": m.kv_heads, "head_dim": m.dim, "v_head_dim": m.vdim,
                "qkv_bias": False, "scale": m.scale, "qk_norm_eps": eps, "qk_norm_weight": not talking, "qk_norm_cast": False,
                "head_mix": talking, "names": _ATTENTION_NAMES, "position": position})
        ff = None if layer.mlp is None else PartSpec("plain_mlp", {"hidden": W, "intermediate": layer.mlp.ff, "activation": "relu_squared",
                                                                   "names": {"up": "up", "down": "down"}})
        layers.append(LayerSpec(PartSpec("shifted_pre_norm", {
            "mixer": mixer, "feed_forward": ff, "norm1": norm, "norm2": norm, "token_shift": True, "layer_scale": True,
            "names": {"norm1": "norm1", "mixer": "mix", "norm2": "norm2", "feed_forward": "mlp"}}), f"l{i}"))
    run = tuple(RunEntry(i, add_row=p, add_start=p is not None and p > 0) for i, p in cfg.run_order())
    return ModelSpec(
        vocab_size=cfg.vocab, hidden_size=W, layers=tuple(layers), run=run, final_norm=norm, tie_word_embeddings=True,
        embedding_prefix="embed", final_norm_prefix="final.norm", head_prefix="head",
        embedding=PartSpec("token_table", {"tensor": ""}), head=PartSpec("linear", {"tensor": ""}),
        stream_rows=cfg.loop.times if cfg.loop is not None else 0,       # the table exists whenever the file names a loop
        stream_rows_name="loop.step", stream_rows_eps=eps)
