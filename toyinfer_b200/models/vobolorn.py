"""Vobolorn: the description of the model in terms of parts.

A decoder over a float32 residual stream whose sublayers read the stream as it is and are normed on their outputs only.
Mixers are grouped softmax attention over all earlier positions, without rotation, with queries and keys normed per head, in
two kinds (one with biases on its projections and an output gate per element, one with a query temperature that grows with
the position), and latent attention whose queries come through a latent of their own, with rotary positions on neighbouring
pairs and a gate per head.  The attention layers blend the values of the first of them into their own.  Feed-forwards are
dense with a silu gate; the head is a matrix of its own behind the final norm, soft-capped.  Tensor names: ``embed``, ``head``,
``final.norm``, ``l<i>.norm1``, ``l<i>.norm2``, ``l<i>.mix.*``, ``l<i>.mlp.*``.  Nothing here computes: the parts do.
"""
from __future__ import annotations

import json

from ..config.registry import register_architecture
from ..config.vobolorn import VobolornConfig
from ..parts.base import PartSpec
from ..parts.model import LayerSpec, ModelSpec


def describe_vobolorn(cfg: VobolornConfig) -> ModelSpec:
    eps = cfg.eps
    norm = PartSpec("wide_scalar_rmsnorm", {"size": cfg.width, "eps": eps, "scalar": False})
    positions = {}
    mixing = cfg.mixing_layers()
    layers = []
    for i, L in enumerate(cfg.layers):
        m = L["mixer"]
        if L["type"] == "latent_attention":
            position = None
            if m["rot_dim"]:        # layers with the same rotation share its tables
                position = "rot:" + json.dumps([m["rot"]["dims"], m["rot"]["base"]])
                positions.setdefault(position, PartSpec("rotary_half", {"dim": m["rot"]["dims"], "theta": m["rot"]["base"],
                                                                        "max_positions": cfg.max_positions, "lazy": True,
                                                                        "pairing": "neighbours"}))
            mixer = PartSpec("latent_attention", {
                "n_heads": m["heads"], "dim": m["dim"], "rot_dim": m["rot_dim"], "vdim": m["vdim"], "kv_rank": m["kv_rank"],
                "q_rank": m["q_rank"], "scale": m["scale"], "eps": eps, "position": position, "sinks": False, "gate": True})
        else:
            plain = L["type"] == "attention"
            # every earlier key is visible: no window, no kept first positions
            mixer = PartSpec("kept_window_attention", {
                "n_heads": m["heads"], "n_kv_heads": m["kv_heads"], "dim": m["dim"], "vdim": m["vdim"], "scale": m["scale"], "window": 0,
                "eps": eps, "biases": "qkv" if plain else False, "gate": plain, "temperature": None if plain else m.get("q_temp"),
                "values": None if i not in mixing else "first" if i == mixing[0] else "blended"})
        f = L.get("mlp")
        ffn = PartSpec("gated_dense", {"intermediate_size": f["ff"], "act": "silu"}) if f is not None else None
        layers.append(LayerSpec(prefix=f"l{i}.", block=PartSpec("postnorm", {"norm": norm, "mixer": mixer, "feed_forward": ffn})))
    return ModelSpec(
        vocab_size=cfg.vocab,
        hidden_size=cfg.width,
        max_positions=cfg.max_positions,
        layers=layers,
        final_norm=None,
        positions=positions,
        ignorable=tuple(f"l{i}.mix.vmix" for i in range(len(cfg.layers)) if i not in mixing[1:]),
        embedding=PartSpec("token_table", {"vocab_size": cfg.vocab, "name": "embed", "wide": True}),
        head=PartSpec("linear", {"vocab_size": cfg.vocab, "norm": PartSpec(norm.kind, dict(norm.params, name="norm")), "tied": False,
                                 "name": "head", "norm_prefix": "final.", "softcap": float(cfg.logit_softcap or 0.0)}),
        stop_token_ids=cfg.stop_token_ids,
    )


register_architecture("Vobolorn", VobolornConfig, describe_vobolorn)
