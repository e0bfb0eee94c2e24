"""What of the Mikipel design needs no device: the configuration's checks, the memories of every layer, tensor names and
shapes, scaled rotation frequencies, the row order that stands for neighbour-paired rotation, and the plain implementation's
own invariants."""
from __future__ import annotations

import pytest
import torch

from mikipel_cases import CASES, case, prompts
from plain import mikipel_plain as plain


def config(d):
    from toyinfer_b200 import models  # noqa: F401
    from toyinfer_b200.config.registry import architecture_of
    arch = architecture_of(d)
    return arch, arch.config_cls.from_dict(d)


def build(d, dtype=torch.float32):
    from toyinfer_b200.parts.model import DecoderModel
    arch, cfg = config(d)
    return DecoderModel(arch.describe(cfg), dtype, "cpu")


@pytest.mark.parametrize("name", list(CASES))
def test_every_layer_asks_for_its_mixers_memory_and_the_last_normed_row(name):
    from toyinfer_b200.parts import KVRequest, StateRequest
    d = case(name)
    reqs = build(d).memory_requests()
    assert len(reqs) == len(d["layers"])
    for r, L in zip(reqs, d["layers"]):
        m = L["mixer"]
        assert isinstance(r, tuple) and len(r) == 2
        assert isinstance(r[1], StateRequest) and tuple(r[1].shape) == (d["width"],) and r[1].dtype == torch.float32
        if L["type"] == "attention":
            assert isinstance(r[0], KVRequest) and (r[0].n_kv_heads, r[0].head_dim, r[0].value_dim or r[0].head_dim, r[0].window) == \
                (m["kv_heads"], m["dim"], m["vdim"], 0)
        elif L["type"] == "latent_attention":
            assert (r[0].n_kv_heads, r[0].head_dim, r[0].values, r[0].window) == (1, m["kv_rank"] + m["rot_dim"], False, 0)
        else:
            channels = 2 * m["kv_heads"] * m["dim"] + m["heads"] * m["vdim"]
            assert tuple(r[0].shape) == ((m["conv"] - 1) * channels + m["heads"] * m["dim"] * m["vdim"],) and r[0].dtype == torch.float32


def test_tensor_names_and_shapes():
    s = build(case("P")).param_specs()
    shape = lambda n: tuple(s[n].shape)
    assert shape("embed") == (210, 64) and shape("final.norm") == (64,) and "head" not in s
    for i in range(4):
        assert shape(f"l{i}.norm1") == shape(f"l{i}.shift") == (64,) and shape(f"l{i}.dwa") == (i + 2,)
        assert f"l{i}.norm2" not in s
    assert shape("l0.mix.q") == shape("l0.mix.k") == (24, 64) and shape("l0.mix.v") == shape("l0.mix.g") == (80, 64)
    assert shape("l0.mix.q.conv") == (24, 3) and shape("l0.mix.v.conv") == (80, 3) and shape("l0.mix.o") == (64, 80)
    assert shape("l0.mix.a") == shape("l0.mix.b") == (4, 64) and shape("l0.mix.A_log") == shape("l0.mix.dt_bias") == (4,)
    assert shape("l0.mix.norm") == (20,) and shape("l0.mlp.e4.down") == (64, 24) and shape("l0.mlp.router") == (5, 64)
    assert shape("l0.mlp.router.b") == (5,) and "l0.mlp.correction" not in s
    assert shape("l1.mix.q") == (120, 64) and shape("l1.mix.v") == (24, 64) and shape("l1.mix.o") == (64, 72)
    assert not any(n.startswith("l1.mix.") and n.count(".") > 2 for n in s)                  # no biases, no norm weights
    assert shape("l1.mlp.up") == (40, 64) and shape("l1.mlp.down") == (64, 40) and "l1.mlp.gate" not in s
    assert shape("l2.mix.q") == (36, 64) and shape("l2.mix.dkv") == (24, 64) and shape("l2.mix.dkv.norm") == (20,)
    assert shape("l2.mix.uk") == (24, 20) and shape("l2.mix.uv") == (36, 20) and "l2.mix.sink" not in s
    assert not any(n.startswith("l3.mlp") for n in s)


def test_configuration_problems_are_all_reported():
    from toyinfer_b200.config.base import ConfigError
    d = case("P")
    d["layers"][0]["mixer"]["conv"] = 9
    d["layers"][1]["mixer"]["kv_heads"] = 4                             # 6 heads over 4
    d["layers"][1]["mlp"] = {"kind": "gated", "ff": 4}
    d["layers"][2]["mixer"]["rot"]["dims"] = 6                          # not rot_dim
    d["layers"][2]["mlp"]["router"]["top"] = 7
    d["layers"][3]["type"] = "nothing"
    d["logit_softcap"] = 0.0
    d["norm"] = {}
    with pytest.raises(ConfigError) as e:
        config(d)
    for piece in ("layers[0].mixer.conv", "6 heads", "layers[1].mlp.kind", "layers[2].mixer.rot.dims", "layers[2].mlp.router", "layers[3].type",
                  "logit_softcap", "norm.eps"):
        assert piece in str(e.value), (piece, str(e.value))
    d = case("P")
    del d["layers"][2]["mixer"]["rot"]
    d["layers"][1]["mixer"]["rot"] = {"base": 10.0, "dims": 7, "scaling": {"factor": -1.0}}
    with pytest.raises(ConfigError) as e:
        config(d)
    assert "layers[2].mixer.rot" in str(e.value) and "layers[1].mixer.rot.dims" in str(e.value) and "factor" in str(e.value)


@pytest.mark.parametrize("dims,base,factor", [(8, 300.0, 2.5), (128, 1e6, 4.0), (6, 50.0, 0.5), (24, 1e4, 1.0)])
def test_linearly_scaled_rotation_tables(dims, base, factor):
    from toyinfer_b200.parts.rope import rotary_tables
    cos, sin = rotary_tables(dims, base, 400, {"kind": "linear", "factor": factor})
    f = plain.frequencies({"dims": dims, "base": base, "scaling": {"factor": factor}})
    pos = torch.arange(400, dtype=torch.float64)[:, None]
    torch.testing.assert_close(cos.double(), torch.cos(pos * f), rtol=0, atol=1e-6)
    torch.testing.assert_close(sin.double(), torch.sin(pos * f), rtol=0, atol=1e-6)


def test_layers_with_the_same_rotation_share_tables_and_others_do_not():
    m = build(case("S"))
    assert len(m.ctx.positions) == 3                    # one latent, two different ones for the attention layers
    assert sorted(p.pairing for p in m.ctx.positions.values()) == ["half", "half", "neighbours"]


def test_neighbour_pairs_are_met_by_the_order_of_rows():
    """What the latent mixer binds, turned in half pairs, has the scores that the rows as stored have, turned in neighbour
    pairs."""
    from toyinfer_b200.weights import random_parameters
    d = case("P")
    model = build(d)
    w = random_parameters(model.param_specs(), 3, torch.float32, "cpu")
    keep = {k: v.clone().double() for k, v in w.items()}
    model.bind(w)
    mixer = model.blocks[2].mixer
    H, dim, rot, rank = mixer.n_heads, mixer.dim, mixer.rot, mixer.rank
    x = torch.randn(9, 64, dtype=torch.float64)
    mine = x @ mixer.w_qd.double().T
    cfg_rot = d["layers"][2]["mixer"]["rot"]
    q, b = mine[:, :H * (dim + rot)].view(9, H, dim + rot), mine[:, H * (dim + rot) + rank:][:, None]
    got = torch.einsum("ihe,je->hij", plain.turn(q[:, :, dim:], cfg_rot, "half"), plain.turn(b, cfg_rot, "half")[:, 0])
    q0, d0 = (x @ keep["l2.mix.q"].T).view(9, H, dim + rot), x @ keep["l2.mix.dkv"].T
    want = torch.einsum("ihe,je->hij", plain.turn(q0[:, :, dim:], cfg_rot, "neighbours"), plain.turn(d0[:, None, rank:], cfg_rot, "neighbours")[:, 0])
    torch.testing.assert_close(got, want)
    torch.testing.assert_close(q[:, :, :dim], q0[:, :, :dim])
    torch.testing.assert_close(mine[:, H * (dim + rot):H * (dim + rot) + rank], d0[:, :rank])


@pytest.mark.parametrize("name", ["P", "R"])
def test_the_plain_implementation_is_causal(name):
    """A later token changes nothing before it (so a prompt's logits are those of its pieces)."""
    from toyinfer_b200.weights import random_parameters
    d = case(name)
    w = random_parameters(build(d).param_specs(), 5, torch.float32, "cpu")
    a = prompts(name, [30], seed=1)[0]
    b = a[:20] + prompts(name, [10], seed=2)[0]
    la, lb = plain.forward(d, w, a)[0], plain.forward(d, w, b)[0]
    torch.testing.assert_close(la[:20], lb[:20])
    assert (la[20:] - lb[20:]).abs().max() > 1e-3
    if d.get("logit_softcap"):
        assert la.abs().max() < d["logit_softcap"]


def test_a_depth_beyond_the_history_is_refused():
    from toyinfer_b200.kernels import KernelError
    d = case("T")
    d["layers"] = [d["layers"][0] for _ in range(257)]
    with pytest.raises(KernelError, match="results before it"):
        build(d)
