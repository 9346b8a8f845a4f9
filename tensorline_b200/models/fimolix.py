"""The Fimolix decoder as a `ModelSpec`.

Every layer normalises what its sublayers give (RMS norms in float32 whose weights are stored around zero) and nothing else: the
sublayers read the residual stream itself.  Two mixers: differential attention (Ye et al., "Differential Transformer": the
difference of two maps a head over the same values) behind a short causal convolution and weighted q/k norms, without rotation and
with a cap on its scores; and attention through a latent over a window of keys, with a sink in the softmax and a sigmoid gate per
head, some of whose layers read the latents that an earlier layer keeps.  The feed-forward, where a layer has one, is
W_down gelu(W_up h).  The output head is the embedding table.  Tensor names: `embed`, `l<i>.norm1`, `l<i>.mix.*`, `l<i>.norm2`,
`l<i>.mlp.*`, `final.norm`, each tensor under its own name.
"""
from __future__ import annotations

from ..config.fimolix import FimolixConfig
from ..parts import PartSpec
from .spec import LayerSpec, ModelSpec, RunEntry


def describe_fimolix(cfg: FimolixConfig) -> ModelSpec:
    W, eps = cfg.width, cfg.norm_eps
    norm = PartSpec("rms_norm", {"dim": W, "eps": eps, "tensor": "", "cast_first": False, "one_plus": True})
    layers, run = [], []
    for i, layer in enumerate(cfg.layers):
        m = layer.mixer
        if layer.type == "attention":
            mixer = PartSpec("differential_attention", {
                "hidden": W, "num_heads": m.heads, "num_kv_heads": m.kv_heads, "head_dim": m.dim, "v_head_dim": m.vdim, "scale": m.scale,
                "init": m.diff, "norm_eps": eps, "taps": m.conv, "score_cap": m.softcap})
            run.append(RunEntry(i))
        else:
            mixer = PartSpec("latent_attention", {
                "hidden": W, "num_heads": m.heads, "head_dim": m.dim, "rot_dim": m.rot_dim, "v_head_dim": m.vdim, "q_rank": None,
                "kv_rank": m.kv_rank, "scale": m.scale, "norm_eps": eps, "window": m.window, "sink": True, "head_gate": True,
                "reads_latent": m.kv_from is not None, "names": {"uq": "q"},
                "position": PartSpec("rotary_interleaved", {"theta": m.rot.base, "rotary_dim": m.rot.dims})})
            run.append(RunEntry(i, reads_cache_of=m.kv_from))
        ff = None if layer.mlp is None else PartSpec("plain_mlp", {"hidden": W, "intermediate": layer.mlp.ff, "activation": "gelu_tanh",
                                                                   "names": {"up": "up", "down": "down"}})
        layers.append(LayerSpec(PartSpec("post_norm", {
            "mixer": mixer, "feed_forward": ff, "norm1": norm, "norm2": norm,
            "names": {"norm1": "norm1", "mixer": "mix", "norm2": "norm2", "feed_forward": "mlp"}}), f"l{i}"))
    return ModelSpec(
        vocab_size=cfg.vocab, hidden_size=W, layers=tuple(layers), run=tuple(run), final_norm=norm, tie_word_embeddings=True,
        embedding_prefix="embed", final_norm_prefix="final.norm", head_prefix="head",
        embedding=PartSpec("token_table", {"tensor": ""}), head=PartSpec("linear", {"tensor": ""}))
