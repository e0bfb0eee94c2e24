"""Small Mikipel configurations for the tests, each unlike the others in every size and option, and helpers to write a
model folder with random weights and to read it back for the plain implementation."""
from __future__ import annotations

import copy

import torch

from bolisun_cases import assert_close_logits  # noqa: F401  (the same rule for both types)


def _att(heads, kv, dim, vdim, scale, rot=None):
    m = {"heads": heads, "kv_heads": kv, "dim": dim, "vdim": vdim, "scale": scale}
    if rot:
        m["rot"] = {"base": rot[0], "dims": rot[1]}
        if len(rot) > 2:
            m["rot"]["scaling"] = {"factor": rot[2]}
    return m


def _lat(heads, dim, rot_dim, vdim, rank, scale, base=None):
    m = {"heads": heads, "dim": dim, "rot_dim": rot_dim, "vdim": vdim, "kv_rank": rank, "scale": scale}
    if base:
        m["rot"] = {"base": base, "dims": rot_dim}
    return m


def _delta(heads, kv, dim, vdim, conv):
    return {"heads": heads, "kv_heads": kv, "dim": dim, "vdim": vdim, "conv": conv}


def _dense(ff):
    return {"kind": "dense", "ff": ff}


def _moe(experts, top, ff):
    return {"kind": "moe", "expert": {"ff": ff}, "router": {"experts": experts, "top": top}}


def _layer(kind, mixer, mlp):
    return {"type": {"a": "attention", "l": "latent_attention", "d": "delta"}[kind], "mixer": mixer, "mlp": mlp}


CASES = {
    # every mixer and feed-forward, part of each head rotated with scaled frequencies, values narrower and wider than keys, a
    # layer without feed-forward, all constants away from one
    "P": {
        "architecture": "Mikipel", "vocab": 210, "width": 64, "norm": {"eps": 1e-5}, "embedding": {"scale": 2.5}, "residual_mult": 0.6,
        "logit_softcap": 7.0,
        "layers": [
            _layer("d", _delta(4, 2, 12, 20, 3), _moe(5, 2, 24)),
            _layer("a", _att(6, 2, 20, 12, 0.4, (300.0, 8, 2.5)), _dense(40)),
            _layer("l", _lat(3, 8, 4, 12, 20, 0.3, 50.0), _moe(6, 3, 16)),
            _layer("d", _delta(3, 1, 20, 8, 5), None),
        ],
    },
    # no embedding key, no multiplier, no soft cap; no rotation in the attention, nothing but a rotated part in the latent
    # attention's heads, and one without a rotated part; a convolution of one tap; one expert per token, and all of them
    "Q": {
        "architecture": "Mikipel", "vocab": 310, "width": 96, "norm": {"eps": 1e-6},
        "layers": [
            _layer("l", _lat(4, 0, 16, 8, 24, 0.25, 1e3), _moe(4, 1, 32)),
            _layer("a", _att(3, 3, 16, 32, 0.5), _dense(72)),
            _layer("l", _lat(2, 12, 0, 20, 40, 0.3), _moe(3, 3, 20)),
            _layer("d", _delta(1, 1, 64, 16, 1), _dense(24)),
        ],
    },
    # sizes that are multiples of nothing: a width of 50 and a vocabulary of 97, heads of 10, 6, 5 and 3 elements
    "R": {
        "architecture": "Mikipel", "vocab": 97, "width": 50, "norm": {"eps": 3e-6}, "embedding": {"scale": 0.5}, "residual_mult": 1.7,
        "logit_softcap": 40.0,
        "layers": [
            _layer("a", _att(3, 1, 10, 6, 0.3, (100.0, 6)), _moe(3, 2, 9)),
            _layer("d", _delta(2, 2, 5, 3, 2), _dense(11)),
            _layer("l", _lat(5, 3, 2, 7, 9, 0.5, 20.0), _dense(13)),
        ],
    },
    # heads of the sizes that real models use, which the tensor-core kernels take in bfloat16
    "S": {
        "architecture": "Mikipel", "vocab": 120, "width": 128, "norm": {"eps": 1e-5}, "embedding": {"scale": 4.0}, "residual_mult": 0.5,
        "logit_softcap": 25.0,
        "layers": [
            _layer("l", _lat(4, 64, 64, 128, 128, 0.09, 1e5), _moe(8, 2, 32)),
            _layer("d", _delta(4, 2, 128, 64, 4), _dense(64)),
            _layer("a", _att(4, 1, 128, 128, 0.09, (1e6, 128, 4.0)), _moe(4, 2, 64)),
            _layer("a", _att(4, 2, 64, 64, 0.2, (1e4, 32)), _dense(96)),
        ],
    },
    # many thin layers: a long history to average over
    "T": {
        "architecture": "Mikipel", "vocab": 130, "width": 40, "norm": {"eps": 1e-5}, "embedding": {"scale": 1.5}, "residual_mult": 0.8,
        "logit_softcap": 15.0,
        "layers": [
            _layer("a", _att(2, 1, 8, 8, 0.6, (1e3, 4)), None), _layer("d", _delta(2, 1, 8, 8, 2), _dense(16)),
            _layer("l", _lat(2, 6, 4, 8, 8, 0.4, 1e3), _dense(8)), _layer("d", _delta(2, 2, 12, 4, 4), None),
            _layer("a", _att(4, 2, 6, 10, 0.5, (1e2, 6, 8.0)), _moe(3, 1, 8)), _layer("d", _delta(1, 1, 8, 24, 8), None),
            _layer("l", _lat(3, 4, 2, 6, 12, 0.4, 1e2), None),
        ],
    },
}
SEEDS = {"P": 45, "Q": 46, "R": 47, "S": 48, "T": 49}


def case(name: str) -> dict:
    return copy.deepcopy(CASES[name])


def write_folder(name: str, path: str) -> str:
    from toyinfer_b200.weights import write_model_folder
    write_model_folder(case(name), SEEDS[name], path)
    return path


def read_folder(path: str):
    """(weights by name, config dict) for the plain implementation, through its own reader."""
    from plain.qwen3_plain import read_config, read_weights
    return read_weights(path), read_config(path)


def prompts(name: str, lengths, seed: int = 0):
    g = torch.Generator().manual_seed(12000 + seed)
    v = CASES[name]["vocab"]
    return [torch.randint(0, v, (n,), generator=g).tolist() for n in lengths]
