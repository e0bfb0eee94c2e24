"""Vobolorn's mechanisms one at a time against the plain implementation (tests/plain/vobolorn_plain.py): the stream whose
sublayers are normed on their outputs only, attention with value blending, query temperature, biases and an output gate,
latent attention with a query latent and gated heads, the silu-gated feed-forward.  Mixers run as prompts, single tokens,
pieces of several sizes and unequal batches, in slots and pages that another sequence used before; loud tokens and matching
pairs of tokens far apart make single keys stand out."""
from __future__ import annotations

import pytest
import torch

from plain import vobolorn_plain as plain
from test_bagasun_parts_gpu import loud_inputs, short_names
from test_kadodra_parts_gpu import DEV, DT, batch_for, bind_random, ctx_for, tol
from test_tusasun_parts_gpu import check_all_schedules, feed, inputs, schedules

pytestmark = pytest.mark.gpu
HID = 56


# ---------------------------------------------------------------------------
# the stream
# ---------------------------------------------------------------------------
@pytest.mark.parametrize("dtype", DT)
@pytest.mark.parametrize("H", [36, 50, 300, 1100, 2048, 4104])
@pytest.mark.parametrize("M", [7, 700])
def test_stream_takes_a_normed_output_and_is_read_as_it_is(dtype, H, M):
    from toyinfer_b200.kernels import wide
    g = torch.Generator().manual_seed(H)
    eps = 1e-3
    h = torch.randn(M, H, generator=g) * 2
    y = (torch.randn(M, H, generator=g) * 3).to(dtype)
    w = 1 + 0.3 * torch.randn(H, generator=g)
    dev = lambda t: t.to(DEV)
    want = h.double() + plain.rms_norm(y, w, eps)
    hd = dev(h).clone()
    pend = wide.PostNormed(dev(y), dev(w), eps)
    x = wide.post_norm_add_norm(hd, pend, None, eps, dtype, rounded=True)
    torch.testing.assert_close(hd.cpu().double(), want, rtol=1e-5, atol=1e-5)
    assert torch.equal(x, hd.to(dtype))                       # rounded once, from the 32-bit sum
    # nothing pending: the stream stays, and is read
    before = hd.clone()
    assert torch.equal(wide.post_norm_add_norm(hd, None, None, eps, dtype, rounded=True), before.to(dtype)) and torch.equal(hd, before)
    # the head's read: gathered rows with the pending output, normed once more; the stream stays
    w2 = dev(1 + 0.3 * torch.randn(H, generator=g))
    rows = torch.tensor([5, 0, 5, 6], dtype=torch.int32, device=DEV)
    hd = dev(h).clone()
    z = wide.post_norm_add_norm(hd, pend, w2, eps, dtype, rows=rows)
    torch.testing.assert_close(z.cpu().double(), plain.rms_norm(want, w2.cpu(), eps)[rows.cpu().long()], **tol(dtype, 2.0))
    assert torch.equal(hd.cpu(), h)
    # only the sum
    assert wide.post_norm_add_norm(hd, pend, None, eps, dtype) is None
    torch.testing.assert_close(hd.cpu().double(), want, rtol=1e-5, atol=1e-5)


class Tripler:
    """A mixer without memory: y = 3 x, rounded once."""
    captures_start = True

    def __init__(self, ctx, prefix):
        pass

    param_specs = lambda self: {}
    bind = lambda self, tensors: None
    check_kernels = lambda self, dtype: None
    memory_request = lambda self: None

    def forward(self, x, batch, mem, shared):
        return x * 3


@pytest.mark.parametrize("dtype", DT)
@pytest.mark.parametrize("ff", [False, True])
def test_layers_that_norm_outputs_only(dtype, ff):
    """The input is not normed: doubling the stream's scale changes what a silu-gated feed-forward gives."""
    from toyinfer_b200.kernels import wide
    from toyinfer_b200.parts import PartSpec, build_part, register_part, unregister_part
    hidden, eps = 44, 1e-4
    register_part("mixer", "tripler_for_a_test", Tripler)
    try:
        norm = PartSpec("wide_scalar_rmsnorm", {"size": hidden, "eps": eps, "scalar": False})
        blocks = [build_part("block", PartSpec("postnorm", {
            "norm": norm, "mixer": PartSpec("tripler_for_a_test"),
            "feed_forward": PartSpec("gated_dense", {"intermediate_size": 20, "act": "silu"}) if ff else None}), ctx_for(dtype, hidden), f"l{i}.")
            for i in range(3)]
    finally:
        unregister_part("mixer", "tripler_for_a_test")
    w = {}
    for i, b in enumerate(blocks):
        w.update(bind_random(b, 50 + i, dtype, lambda cpu: [t.mul_(4.0) for k, t in cpu.items() if "mlp" in k]))
    assert ("l0.norm2" in w) == ff and ("l0.mlp.up" in w) == ff
    x = torch.randn(9, hidden, generator=torch.Generator().manual_seed(1)) * 2

    def run(x):
        x = x.double()
        for i in range(3):
            x = x + plain.rms_norm(3 * x, w[f"l{i}.norm1"], eps)
            if ff:
                x = x + plain.rms_norm(plain.feed_forward(x, {k: w[f"l{i}.mlp.{k}"].double() for k in ("gate", "up", "down")}), w[f"l{i}.norm2"], eps)
        return x

    h, delta = x.to(DEV).clone(), None
    for b in blocks:
        h, delta = b.forward(h, delta, None, None, {})
    wide.post_norm_add_norm(h, delta, None, eps, dtype)
    torch.testing.assert_close(h.cpu().double(), run(x), **tol(dtype, 3.0))


# ---------------------------------------------------------------------------
# attention
# ---------------------------------------------------------------------------
class Layers:
    """Mixers one beside the other over the same rows, each with its memory, and one dict for what they leave each other in a
    step; their outputs side by side."""

    def __init__(self, mixers):
        self.mixers = mixers

    def memory_request(self):
        return tuple(m.memory_request() for m in self.mixers)

    def forward(self, x, batch, mem, shared):
        step = {}
        return torch.cat([m.forward(x, batch, v, {"step": step}) for m, v in zip(self.mixers, mem)], dim=1)


ATT = [
    dict(n_heads=6, n_kv_heads=2, dim=20, vdim=12),
    dict(n_heads=3, n_kv_heads=3, dim=16, vdim=40),
    dict(n_heads=5, n_kv_heads=1, dim=48, vdim=33),
    dict(n_heads=4, n_kv_heads=4, dim=3, vdim=5),
    dict(n_heads=2, n_kv_heads=1, dim=200, vdim=24),
    # sizes that the tensor-core kernels take in bfloat16
    dict(n_heads=8, n_kv_heads=1, dim=128, vdim=128),
    dict(n_heads=4, n_kv_heads=2, dim=64, vdim=64),
    dict(n_heads=2, n_kv_heads=2, dim=64, vdim=128),
    dict(n_heads=20, n_kv_heads=1, dim=64, vdim=64),
    dict(n_heads=3, n_kv_heads=1, dim=128, vdim=64),
]
KINDS = {"gated": dict(biases="qkv", gate=True), "warm": dict(biases=False, temperature={"coef": 0.8, "every": 37}),
         "both": dict(biases="qkv", gate=True, temperature={"coef": 0.3, "every": 1})}


def make_att(dtype, c, kind, values=None, seed=3, scale=0.35, edit=None):
    from toyinfer_b200.parts import PartSpec, build_part
    m = build_part("mixer", PartSpec("kept_window_attention", dict(c, scale=scale, eps=1e-5, window=0, values=values, **KINDS[kind])),
                   ctx_for(dtype, HID), "a.")
    w = short_names(bind_random(m, seed, dtype, edit))
    assert ("g" in w) == ("q.b" in w) == bool(KINDS[kind].get("gate")) and ("vmix" in w) == (values == "blended") and "o.b" not in w
    mcfg = {"heads": c["n_heads"], "kv_heads": c["n_kv_heads"], "dim": c["dim"], "vdim": c["vdim"], "scale": scale,
            "q_temp": KINDS[kind].get("temperature")}
    return m, w, mcfg


@pytest.mark.parametrize("dtype", DT)
@pytest.mark.parametrize("kind", ["gated", "warm"])
@pytest.mark.parametrize("c", ATT)
def test_attention_every_way_of_feeding(dtype, kind, c):
    """Loud rows (thirty times the others) at the first tokens and at both sides of page borders."""
    m, w, mcfg = make_att(dtype, c, kind)
    lens = [300, 129, 3]
    xs = [loud_inputs(n, HID, 5 + i, [j for j in (0, 2, 63, 64, 127, 128, 250) if j < n]).to(dtype) for i, n in enumerate(lens)]
    wants = [plain.grouped_attention(x.double(), w, mcfg, 1e-5)[0] for x in xs]
    check_all_schedules(m, xs, wants, dtype, scale=30.0)


@pytest.mark.parametrize("dtype", DT)
@pytest.mark.parametrize("c", [ATT[0], ATT[2], ATT[3], ATT[5], ATT[6], ATT[7]])
def test_values_of_the_first_layer_are_blended_into_later_ones(dtype, c):
    """Three layers on the same rows, of unequal kinds and head counts: the second and third read the first's values, not the
    second's blend, and from the cache what was blended when it was stored."""
    first = dict(c)
    other = dict(c, n_heads=c["n_kv_heads"], dim=c["dim"] + 4 if c["dim"] not in (64, 128) else c["dim"])
    made = [make_att(dtype, first, "gated", "first", 3), make_att(dtype, other, "warm", "blended", 4, edit=lambda p: p["a.vmix"].fill_(0.7)),
            make_att(dtype, first, "both", "blended", 5, edit=lambda p: p["a.vmix"].fill_(-0.4))]

    def run(x):
        y0, v0 = plain.grouped_attention(x, made[0][1], made[0][2], 1e-5)
        return torch.cat([y0] + [plain.grouped_attention(x, w, cfg, 1e-5, v0)[0] for _, w, cfg in made[1:]], dim=1)
    lens = [200, 75, 2]
    xs = [loud_inputs(n, HID, 8 + i, [j for j in (0, 63, 64, 128) if j < n], 10.0).to(dtype) for i, n in enumerate(lens)]
    wants = [run(x.double()) for x in xs]
    alone = torch.cat([plain.grouped_attention(xs[0].double(), w, cfg, 1e-5)[0] for _, w, cfg in made], dim=1)
    assert (alone - wants[0])[:, HID:].abs().max() > 0.1 * wants[0].abs().max()
    check_all_schedules(Layers([m for m, _, _ in made]), xs, wants, dtype, scale=12.0)


@pytest.mark.parametrize("dtype", DT)
@pytest.mark.parametrize("heads", [2, 4])
def test_values_of_a_layer_whose_rows_are_not_aligned(dtype, heads):
    """The first layer's heads of five elements leave its values at odd places; the second layer's sizes are the tensor cores'."""
    made = [make_att(dtype, dict(n_heads=heads, n_kv_heads=1, dim=5, vdim=64), "warm", "first", 3),
            make_att(dtype, dict(n_heads=4, n_kv_heads=1, dim=64, vdim=64), "gated", "blended", 4)]

    def run(x):
        y0, v0 = plain.grouped_attention(x, made[0][1], made[0][2], 1e-5)
        return torch.cat([y0, plain.grouped_attention(x, made[1][1], made[1][2], 1e-5, v0)[0]], dim=1)
    xs = inputs([150, 70, 2], HID, 13, dtype)
    check_all_schedules(Layers([m for m, _, _ in made]), xs, [run(x.double()) for x in xs], dtype, scale=4.0)


def test_blending_needs_values_from_an_earlier_layer():
    m, _, _ = make_att(torch.float32, ATT[0], "warm", "blended")
    x = inputs([5], HID, 1, torch.float32)[0]
    with pytest.raises(RuntimeError, match="none left any"):
        feed(Layers([m]), (m.memory_request(),), [x], [[(0, 5)]], torch.float32)
    with pytest.raises(RuntimeError, match="no place"):
        feed(m, m.memory_request(), [x], [[(0, 5)]], torch.float32)


@pytest.mark.parametrize("dtype", DT)
@pytest.mark.parametrize("dim,vdim", [(32, 16), (128, 128)])
@pytest.mark.parametrize("far", [0, 63, 64, 130])
def test_attention_finds_one_far_key(dtype, dim, vdim, far):
    """Queries read one half of a token, keys the other through the same matrix, and the halves match for late tokens and the
    one at ``far``: its key is the only one that lies along their queries, hundreds of positions back, and takes nearly all of
    their weight; a neighbour's would not."""
    def edit(cpu):
        cpu["a.q"][:, 28:] = 0.0
        cpu["a.k"].zero_()
        cpu["a.k"][:, 28:] = cpu["a.q"][:, :28]
    m, w, mcfg = make_att(dtype, dict(n_heads=1, n_kv_heads=1, dim=dim, vdim=vdim), "warm", scale=12.0 / dim, edit=edit)
    T = 500
    x = torch.randn(T, HID, generator=torch.Generator().manual_seed(31))
    for t in (400, 470, 499):
        x[t, :28] = x[far, 28:]
    x = x.to(dtype)
    run = lambda v: plain.grouped_attention(v.double(), w, mcfg, 1e-5)[0]
    want = run(x)
    moved = x.clone()
    moved[far] = x[far + 1]
    assert (want[400] - run(moved)[400]).abs().max() > 0.1 * want[400].abs().max()
    check_all_schedules(m, [x], [want], dtype)


@pytest.mark.parametrize("dtype", DT)
@pytest.mark.parametrize("every", [1, 8, 100])
def test_temperature_steps_at_its_positions(dtype, every):
    """Queries as they leave the preparing kernels, both forms: the factor is constant between steps and right on both sides of
    each, at positions up to a hundred thousand, for the position in the sequence and not in the step."""
    from toyinfer_b200.kernels import attention_window as KW
    from toyinfer_b200.cache import CacheManager
    from toyinfer_b200.parts import KVRequest
    coef = 0.9
    places = sorted({0, 1, every - 2, every - 1, every, 2 * every - 2, 2 * every - 1, 2 * every, 37 * every - 2, 37 * every - 1, 3999} & set(range(4000)))
    for H, G, d, vd in ((2, 1, 12, 6), (2, 1, 64, 64)):
        cache = CacheManager([KVRequest(G, d, 0, True, vd if vd != d else 0)], 64 * 70, 1, 4096, dtype, DEV)
        s = cache.allocate_slot()
        cache.reserve(s, 4000)
        cache.flush()
        w = torch.rand(d, generator=torch.Generator().manual_seed(2)) + 0.5
        for p in places:
            x = torch.randn(2, H * d + G * (d + vd), generator=torch.Generator().manual_seed(p)).to(dtype)
            y = x.to(DEV)
            KW.head_prepare(y, None, w.to(DEV), w.to(DEV), 1e-5, None, "half", H, G, d, vd, cache.view(0),
                            batch_for("mixed", [s], [p], [2], cache.scratch_slot), temperature=(coef, every))
            t = plain.query_temperature(p + 2, coef, every)[p:]
            want = plain.rms_norm(x[:, :H * d].double().view(2, H, d), w, 1e-5) * t[:, None, None]
            torch.testing.assert_close(y[:, :H * d].cpu().double().view(2, H, d), want, rtol=8e-3 if dtype == torch.bfloat16 else 5e-6, atol=1e-6)
            torch.testing.assert_close(y[:, H * d:(H + G) * d].cpu().double(), plain.rms_norm(x[:, H * d:(H + G) * d].double(), w, 1e-5),
                                       rtol=8e-3 if dtype == torch.bfloat16 else 5e-6, atol=1e-6)


def test_which_kernels_apply_the_gate(monkeypatch):
    """bfloat16 heads of 64 or 128 run prompts, pieces and single tokens on the tensor-core kernels, gate and all, with one
    range of keys and with several: single tokens as one kernel with their preparation, or, switched off, after it; the
    CUDA-core kernels give the same within the rounding of the weights."""
    from toyinfer_b200.kernels import attention
    from toyinfer_b200.kernels import attention_window as KW
    dtype = torch.bfloat16
    m, w, mcfg = make_att(dtype, ATT[6], "gated")
    whole = []
    real_fused = attention.decode_fused
    monkeypatch.setattr(attention, "decode_fused", lambda *a, **k: (whole.append(1), real_fused(*a, **k)))
    xs = [loud_inputs(n, HID, 5 + n, [j for j in (0, 65, 66, 130) if j < n], 8.0).to(dtype) for n in (530, 67)]
    calls = []
    real = KW._fn

    def spy(name, sig):
        calls.append(name)
        return real(name, sig)
    monkeypatch.setattr(KW, "_fn", spy)
    sch = schedules([530, 67])
    got = {name: feed(m, m.memory_request(), xs, s_, dtype) for name, s_ in sch.items()}
    assert len(whole) > 40 and "ti_attn_window_tc" in calls and not {"ti_attn_decode_mma_scored", "ti_attn_window", "ti_attn_window_decode"} & set(calls)
    wants = [plain.grouped_attention(x.double(), w, mcfg, 1e-5)[0] for x in xs]
    for g, want in zip(got["decode"], wants):
        torch.testing.assert_close(g, want, **tol(dtype, 8.0))
    monkeypatch.setattr(attention, "decode_fused_eligible", lambda *a: False)
    got = {name: feed(m, m.memory_request(), xs, s_, dtype) for name, s_ in sch.items()}
    short = feed(m, m.memory_request(), [x[:40] for x in xs], [[(0, 20), (1, 20)]] + [[(0, 1), (1, 1)]] * 20, dtype)
    assert "ti_attn_window_tc" in calls and "ti_attn_decode_mma_scored" in calls and "ti_attn_window_merge" in calls
    assert "ti_attn_window" not in calls and "ti_attn_window_decode" not in calls
    monkeypatch.setattr(KW, "tensor_cores", False)
    calls.clear()
    other = {name: feed(m, m.memory_request(), xs, s_, dtype) for name, s_ in sch.items()}
    assert "ti_attn_window" in calls and "ti_attn_window_decode" in calls and "ti_attn_window_tc" not in calls
    for name in sch:
        for g, o, want in zip(got[name], other[name], wants):
            torch.testing.assert_close(g, want, **tol(dtype, 8.0), msg=lambda e: f"{name}, tensor cores: {e}")
            torch.testing.assert_close(o, want, **tol(dtype, 8.0), msg=lambda e: f"{name}, CUDA cores: {e}")
    for g, want in zip(short, wants):
        torch.testing.assert_close(g, want[:40], **tol(dtype, 8.0))


@pytest.mark.parametrize("mode", [0, 1, 2])
@pytest.mark.parametrize("c", [ATT[5], ATT[8]])
@pytest.mark.parametrize("kind", list(KINDS))
def test_single_tokens_in_one_kernel_however_their_splits_meet(kind, c, mode, monkeypatch):
    """The splits of a sequence's keys merged by a kernel of its own or within a cluster, over hundreds of positions, with a layer
    that keeps its values and one that blends them in."""
    from toyinfer_b200.kernels import attention
    monkeypatch.setattr(attention, "force_merge_mode", mode)
    dtype = torch.bfloat16
    made = [make_att(dtype, c, kind, "first", 3), make_att(dtype, dict(c, n_heads=2), kind, "blended", 4, edit=lambda p: p["a.vmix"].fill_(0.6))]
    xs = [loud_inputs(n, HID, 60 + i, [j for j in (0, 63, 64, 385, 448, 460) if j < n], 6.0).to(dtype) for i, n in enumerate((500, 125))]
    sched = [[(0, 470), (1, 95)]] + [[(0, 1), (1, 1)]] * 30
    got = feed(Layers([m for m, _, _ in made]), tuple(m.memory_request() for m, _, _ in made), xs, sched, dtype)
    for g, x in zip(got, xs):
        y0, v0 = plain.grouped_attention(x.double(), made[0][1], made[0][2], 1e-5)
        y1, _ = plain.grouped_attention(x.double(), made[1][1], made[1][2], 1e-5, v0)
        torch.testing.assert_close(g[-30:], torch.cat([y0, y1], dim=1)[-30:], **tol(dtype, 6.0))


@pytest.mark.parametrize("dtype", DT)
@pytest.mark.parametrize("c", [ATT[0], ATT[5]])
def test_attention_decodes_for_long(dtype, c):
    m, w, mcfg = make_att(dtype, c, "both")
    xs = inputs([420], HID, 8, dtype)
    want = plain.grouped_attention(xs[0].double(), w, mcfg, 1e-5)[0]
    got = feed(m, m.memory_request(), xs, [[(0, 1)]] * 420, dtype)[0]
    torch.testing.assert_close(got, want, **tol(dtype, 3.0))


# ---------------------------------------------------------------------------
# latent attention
# ---------------------------------------------------------------------------
LAT = [
    dict(n_heads=3, dim=8, rot_dim=4, vdim=12, kv_rank=20, q_rank=12),
    dict(n_heads=4, dim=0, rot_dim=16, vdim=8, kv_rank=24, q_rank=40),
    dict(n_heads=2, dim=12, rot_dim=0, vdim=20, kv_rank=40, q_rank=7),
    dict(n_heads=34, dim=6, rot_dim=2, vdim=5, kv_rank=10, q_rank=16),
    # what the tensor-core kernels take in bfloat16: heads that fill 128 and 64 elements exactly, and ones that leave room
    dict(n_heads=2, dim=64, rot_dim=64, vdim=128, kv_rank=64, q_rank=96),
    dict(n_heads=6, dim=24, rot_dim=16, vdim=40, kv_rank=96, q_rank=48),
    dict(n_heads=20, dim=40, rot_dim=24, vdim=64, kv_rank=136, q_rank=50),
]


def make_latent(dtype, c, seed=3, scale=0.3, edit=None, **options):
    from toyinfer_b200.parts import PartSpec, build_part
    ctx = ctx_for(dtype, HID)
    if c["rot_dim"]:
        ctx.positions["r"] = build_part("position", PartSpec("rotary_half", {"dim": c["rot_dim"], "theta": 3e3, "max_positions": 1024,
                                                                             "pairing": "neighbours"}), ctx, "")
    options.setdefault("gate", True)
    m = build_part("mixer", PartSpec("latent_attention", dict(c, scale=scale, eps=1e-5, position="r" if c["rot_dim"] else None, sinks=False, **options)),
                   ctx, "a.")
    w = short_names(bind_random(m, seed, dtype, edit))
    mcfg = {"heads": c["n_heads"], "dim": c["dim"], "rot_dim": c["rot_dim"], "vdim": c["vdim"], "kv_rank": c["kv_rank"], "scale": scale,
            "rot": {"base": 3e3, "dims": c["rot_dim"]}}
    return m, w, mcfg


@pytest.mark.parametrize("dtype", DT)
@pytest.mark.parametrize("c", LAT)
def test_latent_attention_every_way_of_feeding(dtype, c):
    """Loud rows at the first tokens and page borders: the rotated key part is not normed, so their scores stand out for
    every later query (one way or the other).  The gates are spread wide, so that heads differ."""
    m, w, mcfg = make_latent(dtype, c, edit=lambda cpu: cpu["a.g"].mul_(4.0))
    assert set(w) == {"dq", "dq.norm", "uq", "dkv", "dkv.norm", "uk", "uv", "g", "o"}
    lens = [300, 129, 3]
    xs = [loud_inputs(n, HID, 5 + i, [j for j in (0, 2, 63, 64, 127, 128, 250) if j < n]).to(dtype) for i, n in enumerate(lens)]
    wants = [plain.latent_attention(x.double(), w, mcfg, 1e-5) for x in xs]
    check_all_schedules(m, xs, wants, dtype, scale=6.0)


@pytest.mark.parametrize("dtype", DT)
@pytest.mark.parametrize("c", [LAT[0], LAT[5]])
def test_query_latent_and_gate_are_options_of_their_own(dtype, c):
    """A gate without a query latent and a query latent without a gate."""
    xs = inputs([150, 30], HID, 9, dtype)
    m, w, mcfg = make_latent(dtype, dict(c, q_rank=0))
    assert "q" in w and "g" in w and "dq" not in w
    real = plain.rms_norm       # without a query latent the plain function runs behind an identity, its norm left out

    def run(x, w, gate):
        p = dict(w)
        if "q" in p:
            p.update({"dq": torch.eye(HID, dtype=torch.float64), "dq.norm": torch.ones(HID), "uq": p["q"]})
        if not gate:
            p["g"] = torch.zeros(c["n_heads"], HID, dtype=torch.float64)
        if "q" in w:            # leave the query latent's norm out
            plain.rms_norm = lambda u, wt, eps: u.double() if u.shape[-1] == HID and wt.numel() == HID else real(u, wt, eps)
        try:
            y = plain.latent_attention(x, p, mcfg, 1e-5)
        finally:
            plain.rms_norm = real
        return y if gate else 2.0 * y           # sigmoid(0) = 1/2 on every head
    check_all_schedules(m, xs, [run(x.double(), w, True) for x in xs], dtype, scale=4.0)
    m, w, mcfg = make_latent(dtype, c, gate=False)
    assert "g" not in w and "dq" in w
    check_all_schedules(m, xs, [run(x.double(), w, False) for x in xs], dtype, scale=4.0)


@pytest.mark.parametrize("dtype", DT)
@pytest.mark.parametrize("far", [0, 63, 64, 130])
def test_latent_attention_finds_one_far_key(dtype, far):
    """The query latent is a token's first 28 elements, the key/value latent its last 28;
    both up-projections are the same matrix, so where a late token's first half is the far token's last half, its query lies
    along that one key."""
    c = dict(n_heads=2, dim=28, rot_dim=2, vdim=16, kv_rank=28, q_rank=28)

    def edit(cpu):
        eye = torch.eye(28)
        cpu["a.dq"].zero_(); cpu["a.dkv"].zero_()
        cpu["a.dq"][:, :28] = eye
        cpu["a.dkv"][:28, 28:] = eye
        cpu["a.dq.norm"].fill_(1.0); cpu["a.dkv.norm"].fill_(1.0)
        cpu["a.uk"][:28] = eye; cpu["a.uk"][28:] = eye
        cpu["a.uq"].zero_()
        cpu["a.uq"][:28] = eye; cpu["a.uq"][30:58] = eye
    m, w, mcfg = make_latent(dtype, c, scale=0.7, edit=edit)
    T = 500
    x = torch.randn(T, HID, generator=torch.Generator().manual_seed(32))
    for t in (400, 470, 499):
        x[t, :28] = x[far, 28:]
    x = x.to(dtype)
    run = lambda v: plain.latent_attention(v.double(), w, mcfg, 1e-5)
    want = run(x)
    moved = x.clone()
    moved[far] = x[far + 1]
    assert (want[400] - run(moved)[400]).abs().max() > 0.1 * want[400].abs().max()
    check_all_schedules(m, [x], [want], dtype)


@pytest.mark.parametrize("dtype", DT)
def test_latent_attention_decodes_for_long(dtype):
    m, w, mcfg = make_latent(dtype, LAT[5])
    xs = inputs([420], HID, 8, dtype)
    want = plain.latent_attention(xs[0].double(), w, mcfg, 1e-5)
    got = feed(m, m.memory_request(), xs, [[(0, 1)]] * 420, dtype)[0]
    torch.testing.assert_close(got, want, **tol(dtype, 3.0))


# ---------------------------------------------------------------------------
@pytest.mark.parametrize("dtype", DT)
@pytest.mark.parametrize("hidden,ff,M", [(56, 40, 5), (64, 200, 130), (41, 9, 1)])
def test_silu_gated_feed_forward(dtype, hidden, ff, M):
    from toyinfer_b200.parts import PartSpec, build_part
    m = build_part("feed_forward", PartSpec("gated_dense", {"intermediate_size": ff, "act": "silu"}), ctx_for(dtype, hidden), "f.")
    w = short_names(bind_random(m, 4, dtype, lambda cpu: [t.mul_(8.0) for t in cpu.values()]), "f.")
    x = inputs([M], hidden, 6, dtype)[0]
    want = plain.feed_forward(x.double(), w)
    atol = 1e-5 * want.abs().max() if dtype == torch.float32 else 0.02 * want.abs().max()         # (sums of large terms)
    torch.testing.assert_close(m.forward(x.to(DEV), None).cpu().double(), want, rtol=tol(dtype)["rtol"], atol=float(atol))


def test_schedules_of_these_tests_hold_pieces_of_two_tokens():
    assert any(n == 2 for step in schedules([300, 129, 3])["pieces"] for _, n in step)
