"""What of the Vobolorn design needs no device: the configuration's checks, which layer's values the others blend in, the
memories of every layer, tensor names and shapes, what binding does to the latent mixer's rows, and the plain
implementation's own invariants."""
from __future__ import annotations

import math

import pytest
import torch

from plain import vobolorn_plain as plain
from vobolorn_cases import CASES, case, louder, prompts


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
def test_every_layer_asks_for_its_mixers_memory_and_no_more(name):
    from toyinfer_b200.parts import KVRequest
    d = case(name)
    reqs = build(d).memory_requests()
    assert len(reqs) == len(d["layers"])
    for r, L in zip(reqs, d["layers"]):
        m = L["mixer"]
        assert isinstance(r, KVRequest) and r.window == 0
        if L["type"] == "latent_attention":
            assert (r.n_kv_heads, r.head_dim, r.values) == (1, m["kv_rank"] + m["rot_dim"], False)
        else:
            assert (r.n_kv_heads, r.head_dim, r.value_dim or r.head_dim, r.values) == (m["kv_heads"], m["dim"], m["vdim"], True)


@pytest.mark.parametrize("name,roles", [("A", ["first", None, "blended", "blended"]), ("B", [None, "first", None, None, None, "blended"]),
                                        ("C", ["first", None, "blended", None]), ("E", ["first"]), ("F", ["first", "blended", "blended"])])
def test_the_first_layer_that_mixes_gives_the_values(name, roles):
    """Counted over both kinds of attention; layers without the switch are passed over."""
    assert [getattr(b.mixer, "values", None) for b in build(case(name)).blocks] == roles


def test_tensor_names_and_shapes():
    m = build(case("A"))
    s = m.param_specs()
    shape = lambda n: tuple(s[n].shape)
    assert shape("embed") == shape("head") == (190, 72) and shape("final.norm") == (72,)
    for i in range(4):
        assert shape(f"l{i}.norm1") == (72,)
        assert (f"l{i}.norm2" in s) == (i != 2) and (f"l{i}.mlp.up" in s) == (i != 2)
    assert shape("l0.mix.q") == (120, 72) and shape("l0.mix.q.b") == (120,) and shape("l0.mix.k.b") == (40,) and shape("l0.mix.v.b") == (24,)
    assert shape("l0.mix.q.norm") == shape("l0.mix.k.norm") == (20,) and shape("l0.mix.g") == (72, 72) and shape("l0.mix.o") == (72, 72)
    assert "l0.mix.o.b" not in s and "l0.mix.vmix" not in s and "l0.mix.vmix" in m.ignorable_names()
    assert shape("l0.mlp.gate") == shape("l0.mlp.up") == (40, 72) and shape("l0.mlp.down") == (72, 40)
    assert shape("l1.mix.dq") == (28, 72) and shape("l1.mix.dq.norm") == (28,) and shape("l1.mix.uq") == (36, 28)
    assert shape("l1.mix.dkv") == (24, 72) and shape("l1.mix.dkv.norm") == (20,) and shape("l1.mix.g") == (3, 72)
    assert shape("l1.mix.uk") == (24, 20) and shape("l1.mix.uv") == (36, 20) and "l1.mix.q" not in s and "l1.mix.sink" not in s
    assert shape("l2.mix.vmix") == shape("l3.mix.vmix") == () and "l2.mix.g" not in s and "l2.mix.q.b" not in s


def test_configuration_problems_are_all_reported():
    from toyinfer_b200.config.base import ConfigError
    d = case("A")
    d["layers"][0]["mixer"]["kv_heads"] = 4                             # 6 heads over 4
    d["layers"][0]["mlp"] = {"kind": "moe", "ff": 4}
    d["layers"][1]["mixer"]["rot"]["dims"] = 6                          # not rot_dim
    d["layers"][2]["mixer"]["q_temp"]["every"] = 2.5
    d["layers"][3]["type"] = "nothing"
    d["logit_softcap"] = -1.0
    d["norm"] = {}
    with pytest.raises(ConfigError) as e:
        config(d)
    for piece in ("6 heads", "layers[0].mlp.kind", "layers[1].mixer.rot.dims", "layers[2].mixer.q_temp.every", "layers[3].type",
                  "logit_softcap", "norm.eps"):
        assert piece in str(e.value), (piece, str(e.value))
    d = case("A")
    del d["layers"][1]["mixer"]["q_rank"]
    d["layers"][2]["mixer"]["v_mix"] = 1
    with pytest.raises(ConfigError, match="q_rank.*v_mix"):
        config(d)
    d = case("A")
    d["layers"][2]["mixer"]["vdim"] = 16                                # blended with values of 12 elements
    with pytest.raises(ConfigError, match="cannot be blended"):
        config(d)
    d["layers"][2]["mixer"]["v_mix"] = False
    config(d)


def test_a_checkpoint_may_hold_the_unused_factor_of_the_first_layer(tmp_path):
    """The first layer that mixes may carry a factor that nothing reads; any other tensor too many is an error."""
    from toyinfer_b200.weights import load_parameters, random_parameters
    from toyinfer_b200.weights.loader import WeightError
    from toyinfer_b200.weights.safetensors_io import write_safetensors
    d = case("A")
    m = build(d)
    w = random_parameters(m.param_specs(), 3, torch.float32, "cpu")
    w["l0.mix.vmix"] = torch.tensor(0.9)
    write_safetensors(str(tmp_path / "model.safetensors"), w.items())
    got = load_parameters(m.param_specs(), str(tmp_path), torch.float32, "cpu", m.ignorable_names())
    assert "l0.mix.vmix" not in got and got["l2.mix.vmix"].shape == ()
    w["l1.mix.vmix2"] = torch.tensor(0.9)
    write_safetensors(str(tmp_path / "model.safetensors"), w.items())
    with pytest.raises(WeightError, match="vmix2"):
        load_parameters(m.param_specs(), str(tmp_path), torch.float32, "cpu", m.ignorable_names())


def test_latent_rows_as_bound_give_the_scores_of_the_rows_as_stored():
    """The order of rows stands for the neighbours' pairing, through the query latent too; the first product's rows are the
    query latent's, the key/value latent's, the gate's and zeros up to a multiple of eight."""
    from toyinfer_b200.weights import random_parameters
    d = case("C")
    model = build(d)
    w = random_parameters(model.param_specs(), 3, torch.float32, "cpu")
    keep = {k: v.clone().double() for k, v in w.items()}
    model.bind(w)
    mixer, m = model.blocks[1].mixer, d["layers"][1]["mixer"]
    H, dim, rot, rank, qr = m["heads"], m["dim"], m["rot_dim"], m["kv_rank"], m["q_rank"]
    x = torch.randn(9, 50, dtype=torch.float64)
    y = x @ mixer.w_qd.double().T
    assert y.shape[1] == 32 and qr + rank + rot + H == 27 and y[:, 27:].abs().max() == 0
    p = {k[7:]: v for k, v in keep.items() if k.startswith("l1.mix.")}
    torch.testing.assert_close(y[:, :qr], x @ p["dq"].T)
    torch.testing.assert_close(y[:, qr:qr + rank], (x @ p["dkv"].T)[:, :rank])
    torch.testing.assert_close(y[:, qr + rank + rot:27], x @ p["g"].T)
    c = plain.rms_norm(y[:, :qr], p["dq.norm"], 3e-6)
    q, q0 = (c @ mixer.w_uq.double().T).view(9, H, dim + rot), (c @ p["uq"].T).view(9, H, dim + rot)
    torch.testing.assert_close(q[:, :, :dim], q0[:, :, :dim])

    def halves(t):              # pairs (e, e + rot / 2) turned
        out = t.clone()
        for e in range(rot // 2):
            a = torch.arange(9, dtype=torch.float64) * m["rot"]["base"] ** (-2.0 * e / rot)
            cs, sn = torch.cos(a)[:, None], torch.sin(a)[:, None]
            u, v = t[..., e], t[..., e + rot // 2]
            out[..., e], out[..., e + rot // 2] = u * cs - v * sn, v * cs + u * sn
        return out
    b, b0 = y[:, None, qr + rank:qr + rank + rot], (x @ p["dkv"].T)[:, None, rank:]
    got = torch.einsum("ihe,je->hij", halves(q[:, :, dim:]), halves(b)[:, 0])
    want = torch.einsum("ihe,je->hij", plain.neighbours_turned(q0[:, :, dim:], m["rot"]["base"]), plain.neighbours_turned(b0, m["rot"]["base"])[:, 0])
    torch.testing.assert_close(got, want)


def test_the_temperature_steps_where_it_should():
    t = plain.query_temperature(40, 0.5, 8)
    assert t[:7].eq(1.0).all()                          # floor((p + 1) / 8) = 0 up to position 6
    assert float(t[7]) == 1.0 + 0.5 * math.log(2.0) and float(t[14]) == float(t[7]) and float(t[15]) == 1.0 + 0.5 * math.log(3.0)
    assert len(set(t.tolist())) == 6


@pytest.mark.parametrize("name", ["A", "C"])
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
    assert la.abs().max() < d["logit_softcap"]


def test_every_option_counts_in_the_plain_implementation():
    """The tests' weights are large enough that leaving an option out shows."""
    from toyinfer_b200.weights import random_parameters
    d = case("A")
    w = {k: louder(k, t) for k, t in random_parameters(build(d).param_specs(), 5, torch.float32, "cpu").items()}
    ids = prompts("A", [40], seed=3)[0]
    base = plain.forward(d, w, ids)[0]
    moved = lambda cfg, ws: float((plain.forward(cfg, ws, ids)[0] - base).abs().max())
    without = lambda *names: {k: v for k, v in w.items() if k not in names}
    for change in (without("l0.mix.g"), without("l0.mix.q.b"), without("l0.mix.k.b"), without("l0.mix.v.b"),
                   dict(w, **{"l2.mix.vmix": torch.tensor(0.0)}), dict(w, **{"l1.mix.g": w["l1.mix.g"] * 0}),
                   dict(w, **{"l1.mix.dq.norm": w["l1.mix.dq.norm"] ** 2})):
        assert moved(d, change) > 0.02
    plainer = case("A")
    del plainer["layers"][2]["mixer"]["q_temp"]
    assert moved(plainer, w) > 0.02
