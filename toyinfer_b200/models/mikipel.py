"""Mikipel: the description of the model in terms of parts.

A decoder over one float32 stream that is averaged over depth: after every layer a learned weighted sum of the embedding
and of all layers' results goes on.  Mixer and feed-forward of a layer read the same norm, the mixer a token-shifted form of
it, and their sum is scaled before it is added; the embedding's rows are scaled.  Mixers are grouped softmax attention
(rotary positions with linearly scaled frequencies, queries and keys over their root mean square per head), latent
attention (low-rank shared key/value rows, rotary positions on neighbouring pairs) or the gated delta rule with one decay
per head; feed-forwards are dense with a gelu, or mixtures of silu-gated experts under a router whose weights are a softmax
over the chosen logits; the head is the embedding table behind the final norm, soft-capped.  Tensor names: ``embed``,
``final.norm``, ``l<i>.norm1``, ``l<i>.shift``, ``l<i>.dwa``, ``l<i>.mix.*``, ``l<i>.mlp.*``.  Nothing here computes: the parts do.
"""
from __future__ import annotations

import json

from ..config.mikipel import MikipelConfig
from ..config.registry import register_architecture
from ..parts.base import PartSpec
from ..parts.model import LayerSpec, ModelSpec


def describe_mikipel(cfg: MikipelConfig) -> ModelSpec:
    eps = cfg.eps
    norm = lambda name: PartSpec("depth_rmsnorm", {"size": cfg.width, "eps": eps, "name": name})
    positions = {}

    def position(rot, pairing):
        """The name of the tables for a rotation; layers with the same one share them."""
        scaling = dict(rot["scaling"], kind="linear") if rot.get("scaling") else None
        name = "rot:" + json.dumps([rot["dims"], rot["base"], scaling, pairing], sort_keys=True)
        positions.setdefault(name, PartSpec("rotary_half", {"dim": rot["dims"], "theta": rot["base"], "max_positions": cfg.max_positions,
                                                            "scaling": scaling, "lazy": True, "pairing": pairing}))
        return name

    layers = []
    for i, L in enumerate(cfg.layers):
        m = L["mixer"]
        if L["type"] == "attention":
            # every earlier key is visible: no window, no kept first positions
            mixer = PartSpec("kept_window_attention", {
                "n_heads": m["heads"], "n_kv_heads": m["kv_heads"], "dim": m["dim"], "vdim": m["vdim"], "scale": m["scale"], "window": 0,
                "eps": eps, "biases": False, "head_norm": "unit", "position": position(m["rot"], "half") if m.get("rot") else None})
        elif L["type"] == "latent_attention":
            mixer = PartSpec("latent_attention", {
                "n_heads": m["heads"], "dim": m["dim"], "rot_dim": m["rot_dim"], "vdim": m["vdim"], "kv_rank": m["kv_rank"],
                "scale": m["scale"], "eps": eps, "position": position(m["rot"], "neighbours") if m["rot_dim"] else None, "sinks": False})
        else:
            mixer = PartSpec("head_delta", {"n_heads": m["heads"], "n_qk_heads": m["kv_heads"], "dim": m["dim"], "vdim": m["vdim"],
                                            "conv": m["conv"], "eps": eps})
        f = L.get("mlp")
        ffn = None
        if f is not None and f["kind"] == "dense":
            ffn = PartSpec("ungated_dense", {"intermediate_size": f["ff"], "act": "gelu"})
        elif f is not None:
            ffn = PartSpec("softmax_moe", {"n_experts": f["router"]["experts"], "top": f["router"]["top"], "intermediate_size": f["expert"]["ff"],
                                           "correction": False, "router_bias": True})
        block = PartSpec("averaged_parallel", {"norm": norm("norm1"), "mixer": mixer, "feed_forward": ffn, "depth": i,
                                               "mult": cfg.residual_mult})
        layers.append(LayerSpec(prefix=f"l{i}.", block=block))
    return ModelSpec(
        vocab_size=cfg.vocab,
        hidden_size=cfg.width,
        max_positions=cfg.max_positions,
        layers=layers,
        final_norm=None,
        positions=positions,
        embedding=PartSpec("token_table", {"vocab_size": cfg.vocab, "name": "embed", "wide": True, "scale": cfg.embedding_scale}),
        head=PartSpec("linear", {"vocab_size": cfg.vocab, "norm": norm("norm"), "tied": True, "name": "head", "norm_prefix": "final.",
                                 "softcap": float(cfg.logit_softcap or 0.0)}),
        stop_token_ids=cfg.stop_token_ids,
    )


register_architecture("Mikipel", MikipelConfig, describe_mikipel)
