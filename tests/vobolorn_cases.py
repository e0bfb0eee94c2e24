"""Small Vobolorn configurations for the tests, each unlike the others in every size and option, and helpers to write a
model folder with random weights and to read it back for the plain implementation."""
from __future__ import annotations

import copy

import torch

from bolisun_cases import assert_close_logits  # noqa: F401  (the same rule for both types)


def _att(heads, kv, dim, vdim, scale, mix=True):
    return {"type": "attention", "mixer": {"heads": heads, "kv_heads": kv, "dim": dim, "vdim": vdim, "scale": scale, "v_mix": mix}}


def _warm(heads, kv, dim, vdim, scale, temp=None, mix=True):
    L = dict(_att(heads, kv, dim, vdim, scale, mix), type="attention_2")
    if temp:
        L["mixer"]["q_temp"] = {"coef": temp[0], "every": temp[1]}
    return L


def _lat(heads, dim, rot_dim, vdim, rank, q_rank, scale, base=None):
    m = {"heads": heads, "dim": dim, "rot_dim": rot_dim, "vdim": vdim, "kv_rank": rank, "q_rank": q_rank, "scale": scale}
    if base:
        m["rot"] = {"base": base, "dims": rot_dim}
    return {"type": "latent_attention", "mixer": m}


def _with(layer, ff):
    return dict(layer, mlp={"kind": "dense", "ff": ff} if ff else None)


def _model(vocab, width, eps, layers, cap=None):
    d = {"architecture": "Vobolorn", "vocab": vocab, "width": width, "norm": {"eps": eps}, "layers": layers}
    if cap:
        d["logit_softcap"] = cap
    return d


CASES = {
    # every mixer, a layer without feed-forward, values narrower than keys, a temperature that grows every few positions
    "A": _model(190, 72, 1e-5, [
        _with(_att(6, 2, 20, 12, 0.4), 40), _with(_lat(3, 8, 4, 12, 20, 28, 0.3, 50.0), 56), _with(_warm(4, 2, 16, 12, 0.5, (0.7, 5)), None),
        _with(_att(2, 2, 24, 12, 0.3), 24)], 9.0),
    # no soft cap; the first layer blends nothing and the values come from the second kind; values wider than keys; a
    # temperature that changes with every position, and none; latent heads that are all rotated and not rotated at all; a
    # layer that does not blend between two that do
    "B": _model(330, 96, 1e-6, [
        _with(_att(3, 1, 16, 24, 0.5, False), 72), _with(_warm(6, 3, 8, 20, 0.6, (0.2, 1)), 48), _with(_lat(4, 0, 16, 8, 24, 16, 0.25, 1e3), None),
        _with(_warm(8, 2, 12, 40, 0.4, None, False), 32), _with(_lat(2, 12, 0, 20, 40, 8, 0.3), 64), _with(_att(3, 3, 16, 20, 0.7), 40)]),
    # sizes that are multiples of nothing: a width of 50 and a vocabulary of 97, heads of 10, 6, 5 and 3 elements
    "C": _model(97, 50, 3e-6, [
        _with(_warm(3, 1, 10, 5, 0.5, (1.5, 3)), 9), _with(_lat(5, 3, 2, 7, 9, 11, 0.5, 20.0), 13), _with(_att(2, 1, 6, 5, 0.6), 11),
        _with(_lat(2, 5, 6, 3, 14, 5, 0.4, 7.0), None)], 40.0),
    # heads of the sizes that real models use, which the tensor-core kernels take in bfloat16
    "D": _model(120, 128, 1e-5, [
        _with(_warm(4, 1, 128, 128, 0.09, (0.3, 50)), 64), _with(_lat(4, 64, 64, 128, 128, 96, 0.09, 1e5), 96),
        _with(_att(8, 1, 64, 128, 0.12), 128), _with(_lat(20, 32, 16, 48, 64, 40, 0.14, 1e4), 64), _with(_warm(2, 1, 128, 128, 0.1, (0.6, 17)), None)], 25.0),
    # one layer, which has no other to blend with, and no feed-forward
    "E": _model(130, 40, 2e-5, [_with(_att(4, 4, 8, 8, 0.6), None)], 3.0),
    # heads of 64, all values blended, no latent attention
    "F": _model(210, 192, 1e-6, [
        _with(_att(6, 2, 64, 64, 0.2), 160), _with(_warm(4, 2, 64, 64, 0.17, (0.4, 31)), 96), _with(_att(2, 2, 128, 64, 0.11), 64)], 12.0),
}
SEEDS = {"A": 61, "B": 62, "C": 63, "D": 64, "E": 65, "F": 66}


def case(name: str) -> dict:
    return copy.deepcopy(CASES[name])


LOUDER = {"embed": 50.0, "head": 3.0, ".uq": 4.0, ".uk": 4.0, ".b": 5.0, ".gate": 2.0, ".up": 2.0}


def louder(name: str, t: torch.Tensor) -> torch.Tensor:
    """Random weights as drawn are small; these factors make scores, biases and gates large enough that each shows in the logits."""
    return t * next((f for end, f in LOUDER.items() if name.endswith(end)), 1.0)


def write_folder(name: str, path: str) -> str:
    """config.json and bfloat16 weights, drawn with the case's seed and made louder."""
    from toyinfer_b200.weights import open_model, write_model_folder, write_safetensors
    write_model_folder(case(name), SEEDS[name], path)
    files, where = open_model(path)
    tensors = [(n, louder(n, f.tensor(n)).clone()) for n, f in where.items()]
    for f in files:
        f.close()
    write_safetensors(f"{path}/model.safetensors", tensors)
    return path


def read_folder(path: str):
    """(weights by name, config dict) for the plain implementation, through its own reader."""
    from plain.qwen3_plain import read_config, read_weights
    return read_weights(path), read_config(path)


def prompts(name: str, lengths, seed: int = 0):
    g = torch.Generator().manual_seed(14000 + seed)
    v = CASES[name]["vocab"]
    return [torch.randint(0, v, (n,), generator=g).tolist() for n in lengths]
