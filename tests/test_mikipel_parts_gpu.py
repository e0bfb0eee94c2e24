"""Mikipel's mechanisms one at a time against the plain implementation (tests/plain/mikipel_plain.py): the depth-averaged
stream with its norm and token shift, attention with weightless head norms and scaled rotation, latent attention on
neighbour pairs without a window, the gated delta rule with one decay per head, the gelu feed-forward, and experts under a
biased router.  Mixers run as prompts, single tokens, pieces of several sizes and unequal batches, in slots and pages that
another sequence used before; loud tokens and matching pairs of tokens far apart make single keys stand out."""
from __future__ import annotations

import pytest
import torch

from plain import mikipel_plain as plain
from test_bagasun_parts_gpu import loud_inputs, short_names
from test_kadodra_parts_gpu import DEV, DT, batch_for, bind_random, ctx_for, tol
from test_tusasun_parts_gpu import check_all_schedules, feed, inputs, schedules

pytestmark = pytest.mark.gpu


# ---------------------------------------------------------------------------
# the stream
# ---------------------------------------------------------------------------
def plain_read(results, c_in, c_out, a, f, mult):
    """(the pending layer's result, what goes on)."""
    y = sum(float(c) * x.double() for c, x in zip(c_in, results)) if c_in is not None else results[-1].double()
    X = y + mult * (a.double() + (f.double() if f is not None else 0.0))
    if c_out is None:
        return X, X
    return X, sum(float(c) * x.double() for c, x in zip(c_out, results)) + float(c_out[-1]) * X


@pytest.mark.parametrize("dtype", DT)
@pytest.mark.parametrize("H", [36, 50, 300, 1100, 4104])            # whole runs of four, and not
@pytest.mark.parametrize("n,second", [(1, True), (3, False), (9, True)])
def test_stream_average_and_norm(dtype, H, n, second):
    from toyinfer_b200.kernels import depth
    g = torch.Generator().manual_seed(H + n)
    M, eps, mult = 7, 1e-5, 0.37
    results = [torch.randn(M, H, generator=g) * (j + 1) for j in range(n)]
    a = (torch.randn(M, H, generator=g) * 3).to(dtype)
    f = (torch.randn(M, H, generator=g) * 2).to(dtype) if second else None
    c_in = torch.randn(n, generator=g) if n > 1 else None
    c_out = torch.randn(n + 1, generator=g)
    w = torch.rand(H, generator=g) + 0.5
    dev = lambda t: None if t is None else t.to(DEV)
    X, y = plain_read(results, c_in, c_out, a, f, mult)
    kept = [dev(x) for x in results]
    pend = depth.DepthUpdate(list(kept), dev(a), dev(f), mult, dev(c_in), dev(c_out))
    z, zs, history, total = depth.depth_norm(kept[0], pend, dev(w), eps, dtype, want_sum=True)
    assert zs is None and len(history) == n + 1 and len(pend.results) == n
    torch.testing.assert_close(history[-1].cpu().double(), X, rtol=1e-5, atol=1e-5 * n)
    torch.testing.assert_close(total.cpu().double(), y, rtol=1e-5, atol=3e-5 * n)
    torch.testing.assert_close(z.cpu().double(), plain.rms_norm(y, w, eps), **tol(dtype, 2.0))
    for x, k in zip(results, kept):
        assert torch.equal(k.cpu(), x)
    # gathered rows: no result is written
    rows = torch.tensor([5, 0, 5, 6], dtype=torch.int32, device=DEV)
    zr, _, history, tr = depth.depth_norm(kept[0], pend, dev(w), eps, dtype, rows=rows, want_sum=True)
    assert len(history) == n and torch.equal(zr, z[rows.long()]) and torch.equal(tr, total[rows.long()])
    # no averaging: the result itself goes on
    X1, _ = plain_read(results, c_in, None, a, f, mult)
    z1, _, history, t1 = depth.depth_norm(kept[0], depth.DepthUpdate(list(kept), dev(a), dev(f), mult, dev(c_in), None), dev(w), eps, dtype, want_sum=True)
    assert len(history) == 1
    torch.testing.assert_close(history[0].cpu().double(), X1, rtol=1e-5, atol=1e-5 * n)
    torch.testing.assert_close(t1.cpu().double(), X1, rtol=1e-5, atol=1e-5 * n)
    # nothing pending: the embedding's rows
    z0 = depth.depth_norm(kept[0], None, dev(w), eps, dtype)[0]
    torch.testing.assert_close(z0.cpu().double(), plain.rms_norm(results[0], w, eps), **tol(dtype, 2.0))


@pytest.mark.parametrize("dtype", DT)
@pytest.mark.parametrize("H", [36, 51])
@pytest.mark.parametrize("lens", [[1], [2], [9, 1, 30], [1500, 1, 2, 1300], [700] * 4 + [3, 1] * 30])
def test_token_shift_over_many_rows(dtype, H, lens):
    """Enough rows that a block walks several of them (the row before a block's first is formed again), sequences that begin
    and end inside a block; from the start, and going on from a state that another slot's junk surrounds."""
    from toyinfer_b200.kernels import depth
    g = torch.Generator().manual_seed(H + len(lens))
    M, B, eps = sum(lens), len(lens), 1e-5
    x0, x1 = torch.randn(M, H, generator=g), torch.randn(M, H, generator=g)
    a = torch.randn(M, H, generator=g).to(dtype)
    c_in, c_out = torch.tensor([0.5, 0.7]), torch.tensor([0.3, -0.8, 1.1])
    w, mix = torch.rand(H, generator=g) + 0.5, torch.rand(H, generator=g) * 1.4 - 0.2
    _, y = plain_read([x0, x1], c_in, c_out, a, None, 0.9)
    z = plain.rms_norm(y, w, eps)
    before = torch.randn(B + 3, H, generator=g)
    slots = [(7 * b) % (B + 2) if (B + 2) % 7 else (5 * b) % (B + 2) for b in range(B)]
    assert len(set(slots)) == B
    dev = lambda t: t.to(DEV)
    for mode in ("start", "mixed"):
        state = dev(before).clone()
        pend = depth.DepthUpdate([dev(x0), dev(x1)], dev(a), None, 0.9, dev(c_in), dev(c_out))
        batch = batch_for(mode, slots, [0 if mode == "start" else 3] * B, lens, B + 2)
        got, zs, _, _ = depth.depth_norm(pend.results[0], pend, dev(w), eps, dtype, depth.ShiftedRead(dev(mix), state, batch))
        torch.testing.assert_close(got.cpu().double(), z, **tol(dtype, 2.0))
        want_state, o = before.double().clone(), 0
        for b, n in enumerate(lens):
            first = torch.zeros(1, H, dtype=torch.float64) if mode == "start" else before[slots[b]:slots[b] + 1].double()
            prev = torch.cat([first, z[o:o + n - 1]])
            torch.testing.assert_close(zs[o:o + n].cpu().double(), z[o:o + n] + (prev - z[o:o + n]) * mix.double(), **tol(dtype, 3.0),
                                       msg=lambda e: f"{mode}, sequence {b}: {e}")
            want_state[slots[b]] = z[o + n - 1]
            o += n
        torch.testing.assert_close(state.cpu().double(), want_state, rtol=1e-4, atol=1e-5)


class Doubler:
    """A mixer without memory: y = 2 x, rounded once."""
    captures_start = True

    def __init__(self, ctx, prefix):
        pass

    def param_specs(self):
        return {}

    def bind(self, tensors):
        pass

    def check_kernels(self, dtype):
        pass

    def memory_request(self):
        return None

    def forward(self, x, batch, mem, shared):
        return x * 2


class Stack:
    """Blocks one after the other over the rows they are given, so that what the cache holds for each is used as in a model."""

    def __init__(self, blocks):
        self.blocks = blocks

    def memory_request(self):
        return sum((b.memory_request() for b in self.blocks), ())

    def forward(self, x, batch, mem, shared):
        from toyinfer_b200.kernels import depth
        h, delta = x.float(), None
        for i, b in enumerate(self.blocks):
            h, delta = b.forward(h, delta, batch, mem[i:i + 1], {})
        return depth.depth_norm(h, delta, None, 0.0, x.dtype, want_sum=True)[3]


@pytest.mark.parametrize("dtype", DT)
@pytest.mark.parametrize("ff", [False, True])
def test_layers_with_shift_and_average_every_way_of_feeding(dtype, ff):
    """Three layers around a mixer without memory of its own: prompts, single tokens and pieces (the last row of a piece is
    the next one's row before), in slots used before, with and without a feed-forward beside the mixer."""
    from toyinfer_b200.parts import PartSpec, build_part, register_part, unregister_part
    hidden, eps = 44, 1e-5
    register_part("mixer", "doubler_for_a_test", Doubler)
    try:
        blocks = [build_part("block", PartSpec("averaged_parallel", {
            "norm": PartSpec("depth_rmsnorm", {"size": hidden, "eps": eps, "name": "norm1"}), "mixer": PartSpec("doubler_for_a_test"),
            "feed_forward": PartSpec("ungated_dense", {"intermediate_size": 20, "act": "gelu"}) if ff else None, "depth": i, "mult": 0.65}),
            ctx_for(dtype, hidden), f"l{i}.") for i in range(3)]
    finally:
        unregister_part("mixer", "doubler_for_a_test")
    w = {}
    for i, b in enumerate(blocks):
        w.update(bind_random(b, 40 + i, dtype))
    assert ("l0.mlp.up" in w) == ff

    def run(x):
        y = x.double()
        results = [y]
        for i in range(3):
            z = plain.rms_norm(y, w[f"l{i}.norm1"], eps)
            out = 2 * plain.token_shift(z, w[f"l{i}.shift"])
            if ff:
                out = out + plain.dense_ff(z, {k: w[f"l{i}.mlp.{k}"].double() for k in ("up", "down")})
            results.append(y + 0.65 * out)
            y = plain.depth_average(results, w[f"l{i}.dwa"])
        return y
    xs = inputs([150, 70, 2, 1], hidden, 3, dtype)
    check_all_schedules(Stack(blocks), xs, [run(x) for x in xs], dtype, scale=4.0)


# ---------------------------------------------------------------------------
# mixers
# ---------------------------------------------------------------------------
ATT = [
    dict(n_heads=6, n_kv_heads=2, dim=20, vdim=12, rot=dict(base=300.0, dims=8, scaling={"factor": 2.5})),
    dict(n_heads=3, n_kv_heads=3, dim=16, vdim=40),
    dict(n_heads=5, n_kv_heads=1, dim=48, vdim=48, rot=dict(base=1e4, dims=48)),
    dict(n_heads=4, n_kv_heads=4, dim=3, vdim=5),
    dict(n_heads=2, n_kv_heads=1, dim=200, vdim=24, rot=dict(base=1e3, dims=100, scaling={"factor": 16.0})),
    # sizes that the tensor-core kernels take in bfloat16
    dict(n_heads=4, n_kv_heads=1, dim=128, vdim=128, rot=dict(base=1e6, dims=128, scaling={"factor": 8.0})),
    dict(n_heads=4, n_kv_heads=2, dim=64, vdim=64, rot=dict(base=1e4, dims=32)),
    dict(n_heads=2, n_kv_heads=2, dim=64, vdim=128),
]


def make_att(dtype, c, hidden=56, seed=3, scale=0.35, edit=None):
    from toyinfer_b200.parts import PartSpec, build_part
    c = dict(c)
    rot = c.pop("rot", None)
    positions, position = {}, None
    if rot:
        position = "r"
        sc = dict(rot["scaling"], kind="linear") if rot.get("scaling") else None
        positions["r"] = build_part("position", PartSpec("rotary_half", {"dim": rot["dims"], "theta": rot["base"], "max_positions": 2048,
                                                                         "scaling": sc}), ctx_for(dtype, hidden), "")
    m = build_part("mixer", PartSpec("kept_window_attention", dict(c, scale=scale, eps=1e-5, position=position, window=0, biases=False,
                                                                   head_norm="unit")), ctx_for(dtype, hidden, positions), "a.")
    w = short_names(bind_random(m, seed, dtype, edit))
    assert set(w) == {"q", "k", "v", "o"}
    mcfg = {"heads": c["n_heads"], "kv_heads": c["n_kv_heads"], "dim": c["dim"], "vdim": c["vdim"], "scale": scale}
    if rot:
        mcfg["rot"] = rot
    return m, w, mcfg


@pytest.mark.parametrize("dtype", DT)
@pytest.mark.parametrize("c", ATT)
def test_attention_every_way_of_feeding(dtype, c):
    """Loud rows (values thirty times the others) at the first tokens and at both sides of page borders."""
    m, w, mcfg = make_att(dtype, c)
    lens = [300, 129, 3]
    xs = [loud_inputs(n, 56, 5 + i, [j for j in (0, 2, 63, 64, 127, 128, 250) if j < n]).to(dtype) for i, n in enumerate(lens)]
    wants = [plain.attention(x.double(), w, mcfg, 1e-5) for x in xs]
    check_all_schedules(m, xs, wants, dtype, scale=30.0)


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
    m, w, mcfg = make_att(dtype, dict(n_heads=1, n_kv_heads=1, dim=dim, vdim=vdim), scale=20.0 / dim, edit=edit)
    T = 500
    x = torch.randn(T, 56, generator=torch.Generator().manual_seed(31))
    for t in (400, 470, 499):
        x[t, :28] = x[far, 28:]
    x = x.to(dtype)
    want = plain.attention(x.double(), w, mcfg, 1e-5)
    moved = x.clone()
    moved[far] = x[far + 1]
    assert (want[400] - plain.attention(moved.double(), w, mcfg, 1e-5)[400]).abs().max() > 0.1 * want[400].abs().max()
    check_all_schedules(m, [x], [want], dtype)


LAT = [
    dict(n_heads=3, dim=8, rot_dim=4, vdim=12, kv_rank=20),
    dict(n_heads=4, dim=0, rot_dim=16, vdim=8, kv_rank=24),
    dict(n_heads=2, dim=12, rot_dim=0, vdim=20, kv_rank=40),
    dict(n_heads=34, dim=6, rot_dim=2, vdim=5, kv_rank=10),
    # what the tensor-core kernels take in bfloat16: heads that fill 128 and 64 elements exactly, and ones that leave room
    dict(n_heads=2, dim=64, rot_dim=64, vdim=128, kv_rank=64),
    dict(n_heads=6, dim=24, rot_dim=16, vdim=40, kv_rank=96),
    dict(n_heads=20, dim=40, rot_dim=24, vdim=64, kv_rank=136),
]


@pytest.mark.parametrize("dtype", DT)
@pytest.mark.parametrize("c", LAT)
def test_latent_attention_on_neighbour_pairs(dtype, c):
    """Loud rows at the first tokens and page borders: the rotated key part is not normed, so their scores stand out for
    every later query (one way or the other)."""
    from toyinfer_b200.parts import PartSpec, build_part
    hidden = 56
    ctx = ctx_for(dtype, hidden)
    if c["rot_dim"]:
        ctx.positions["r"] = build_part("position", PartSpec("rotary_half", {"dim": c["rot_dim"], "theta": 3e3, "max_positions": 1024,
                                                                             "pairing": "neighbours"}), ctx, "")
    m = build_part("mixer", PartSpec("latent_attention", dict(c, scale=0.3, eps=1e-5, position="r" if c["rot_dim"] else None, sinks=False)), ctx, "a.")
    w = short_names(bind_random(m, 3, dtype))
    assert set(w) == {"q", "dkv", "dkv.norm", "uk", "uv", "o"}
    mcfg = {"heads": c["n_heads"], "dim": c["dim"], "rot_dim": c["rot_dim"], "vdim": c["vdim"], "kv_rank": c["kv_rank"], "scale": 0.3,
            "rot": {"base": 3e3, "dims": c["rot_dim"]}}
    lens = [300, 129, 3]
    xs = [loud_inputs(n, hidden, 5 + i, [j for j in (0, 2, 63, 64, 127, 128, 250) if j < n]).to(dtype) for i, n in enumerate(lens)]
    wants = [plain.latent_attention(x.double(), w, mcfg, 1e-5) for x in xs]
    check_all_schedules(m, xs, wants, dtype, scale=6.0)


DELTA = [dict(n_heads=4, n_qk_heads=2, dim=16, vdim=24, conv=3), dict(n_heads=2, n_qk_heads=2, dim=40, vdim=72, conv=2),
         dict(n_heads=3, n_qk_heads=1, dim=128, vdim=8, conv=4), dict(n_heads=1, n_qk_heads=1, dim=64, vdim=150, conv=1),
         dict(n_heads=2, n_qk_heads=1, dim=200, vdim=20, conv=8), dict(n_heads=6, n_qk_heads=3, dim=5, vdim=3, conv=5)]


def make_delta(dtype, c, hidden=48, seed=5, slow=2.0):
    from toyinfer_b200.parts import PartSpec, build_part
    m = build_part("mixer", PartSpec("head_delta", dict(c, eps=1e-5)), ctx_for(dtype, hidden), "a.")
    # decays near one: what was written hundreds of tokens ago still counts
    w = short_names(bind_random(m, seed, dtype, lambda cpu: cpu["a.dt_bias"].sub_(slow)))
    return m, w, {"heads": c["n_heads"], "kv_heads": c["n_qk_heads"], "dim": c["dim"], "vdim": c["vdim"], "conv": c["conv"]}


@pytest.mark.parametrize("dtype", DT)
@pytest.mark.parametrize("c", DELTA)
def test_delta_rule_with_one_decay_per_head(dtype, c):
    m, w, cfg = make_delta(dtype, c)
    xs = inputs([180, 70, 2], 48, 7, dtype)
    check_all_schedules(m, xs, [plain.delta(x.double(), w, cfg, 1e-5) for x in xs], dtype)


@pytest.mark.parametrize("dtype", DT)
def test_delta_rule_decodes_for_long(dtype):
    m, w, cfg = make_delta(dtype, dict(n_heads=2, n_qk_heads=1, dim=32, vdim=32, conv=4), seed=6, slow=4.0)
    xs = inputs([400], 48, 8, dtype)
    want = plain.delta(xs[0].double(), w, cfg, 1e-5)
    got = feed(m, m.memory_request(), xs, [[(0, 5)]] + [[(0, 1)]] * 395, dtype)[0]
    torch.testing.assert_close(got, want, **tol(dtype, 3.0))


@pytest.mark.parametrize("dtype", DT)
def test_delta_rule_keeps_one_early_write(dtype):
    """The recurrence alone: every token but one writes nothing (beta near zero) and nothing decays; the value written at
    position 1 is read back by its own key three hundred tokens later, across pieces, and another key finds nothing."""
    from toyinfer_b200.kernels import recurrent as KR
    T, H, d, dv = 320, 2, 16, 24
    g = torch.Generator().manual_seed(4)
    k = torch.randn(T, H, d, generator=g)
    k[300] = k[1]
    q = k.clone()
    v = torch.randn(T, H, dv, generator=g)
    beta = torch.full((T, H), -40.0)
    beta[1] = 40.0
    decay, dt, rate = torch.full((T, H), -40.0), torch.zeros(H), torch.ones(H)
    state = torch.randn(3, H * d * dv + 5, generator=g)
    state[2] = 0.0
    sd = state.to(DEV)
    dev = lambda t: t.to(dtype).to(DEV).contiguous()
    out = []
    for a, b in ((0, 64), (64, 66), (66, 67), (67, T)):
        batch = batch_for("start" if a == 0 else "extend" if b - a == 1 else "mixed", [2], [a], [b - a], 0)
        out.append(KR.delta_rule(dev(q[a:b]), dev(k[a:b]), dev(v[a:b]), dev(decay[a:b]), dt.to(DEV), rate.to(DEV), dev(beta[a:b]), sd, 5,
                                 batch, head_decay=True).cpu())
    o = torch.cat(out).view(T, H, dv)
    torch.testing.assert_close(o[300], v[1].to(dtype).float() * d ** -0.5, rtol=1e-3, atol=1e-3)
    assert o[0].abs().max() < 1e-12 and torch.equal(sd[:2].cpu(), state[:2]) and torch.equal(sd[2, :5].cpu(), state[2, :5])


# ---------------------------------------------------------------------------
# feed-forwards
# ---------------------------------------------------------------------------
@pytest.mark.parametrize("dtype", DT)
@pytest.mark.parametrize("hidden,ff,M", [(56, 40, 5), (64, 200, 130), (41, 9, 1)])
def test_gelu_feed_forward(dtype, hidden, ff, M):
    from toyinfer_b200.kernels import moe as KM
    from toyinfer_b200.parts import PartSpec, build_part
    m = build_part("feed_forward", PartSpec("ungated_dense", {"intermediate_size": ff, "act": "gelu"}), ctx_for(dtype, hidden), "f.")
    w = short_names(bind_random(m, 4, dtype, lambda cpu: [t.mul_(8.0) for t in cpu.values()]), "f.")
    x = inputs([M], hidden, 6, dtype)[0]
    torch.testing.assert_close(m.forward(x.to(DEV), None).cpu().double(), plain.dense_ff(x.double(), w), **tol(dtype, 2.0))
    a = (torch.linspace(-9, 9, 1000)[None] * torch.ones(3, 1)).to(dtype)                 # the tails, where the tanh form differs
    torch.testing.assert_close(KM.pointwise_act(a.to(DEV), "gelu").cpu().double(), plain.gelu(a.double()),
                               rtol=1e-2 if dtype == torch.bfloat16 else 1e-5, atol=1e-6)


@pytest.mark.parametrize("act", ["gelu", "relu2"])
@pytest.mark.parametrize("M,N,K", [(1, 200, 136), (1, 4096, 1024), (3, 77, 64), (8, 1000, 512), (16, 136, 264), (40, 512, 2048), (130, 264, 96),
                                   (700, 1032, 520), (2100, 2048, 256), (256, 2560, 4096)])
def test_activation_in_the_products_epilogue(act, M, N, K):
    """Every product kernel (one token, few tokens, many tokens, a contraction cut into pieces) with the activation on its
    32-bit results, against the activation of the exact product."""
    import toyinfer_b200.kernels as TK
    g = torch.Generator(device=DEV).manual_seed(M + N)
    x = torch.randn(M, K, generator=g, device=DEV).to(torch.bfloat16)
    w = (torch.randn(N, K, generator=g, device=DEV) * (2.5 / K ** 0.5)).to(torch.bfloat16)
    before = TK.launch_count
    got = TK.linear_act(x, w, act).double()
    assert TK.launch_count == before + 1                 # no kernel of its own for the activation
    z = x.double() @ w.double().T
    want = plain.gelu(z) if act == "gelu" else torch.clamp(z, min=0.0) ** 2
    torch.testing.assert_close(got, want, rtol=1e-2, atol=2e-4)


def test_biased_router_against_the_rule():
    """The bias changes the choice and the weights; equal logits go to the lower index; logits so far below the largest that
    their softmax is zero are still chosen in their order."""
    from toyinfer_b200.kernels import moe as KM
    g = torch.Generator().manual_seed(4)
    for E, top in [(6, 2), (8, 4), (16, 3), (5, 5), (4, 1), (20, 16)]:
        M = 64
        z = torch.randn(M, E + 3, generator=g) * 2
        b = torch.randn(E, generator=g)
        z[5, :E] = -b                                   # all equal
        z[6, :E] = torch.arange(E) * -300.0 - b
        z[7, :E] = torch.arange(E) * 300.0 - b
        perm, off, weight = (t.cpu() for t in KM.route_softmax(z.to(DEV)[:, :E], None, E, top, logit_bias=b.to(DEV)))
        expert_of = torch.empty(M * top, dtype=torch.long)
        for e in range(E):
            expert_of[perm[off[e]:off[e + 1]].long()] = e
        assert off[0] == 0 and off[E] == M * top and sorted(perm.tolist()) == list(range(M * top))
        for m in range(M):
            chosen, w = plain.route(z[m, :E] + b, top)
            if m != 5:                                  # (-b + b need not be exactly zero for every expert)
                assert expert_of[m * top:(m + 1) * top].tolist() == chosen, (E, top, m)
            torch.testing.assert_close(weight[m * top:(m + 1) * top].double(), w.double(), rtol=1e-5, atol=1e-6)


@pytest.mark.parametrize("dtype", DT)
@pytest.mark.parametrize("M", [1, 7, 700])           # single tokens, a few, and enough pairs per expert for the padded tensor-core groups
@pytest.mark.parametrize("E,top,ff,hidden", [(6, 2, 24, 64), (4, 1, 32, 64), (3, 3, 9, 50), (8, 4, 40, 72)])
def test_experts_under_the_biased_router(dtype, E, top, ff, hidden, M):
    from toyinfer_b200.parts import PartSpec, build_part
    m = build_part("feed_forward", PartSpec("softmax_moe", {"n_experts": E, "top": top, "intermediate_size": ff, "correction": False,
                                                            "router_bias": True}), ctx_for(dtype, hidden), "f.")
    w = short_names(bind_random(m, 8, dtype, lambda cpu: (cpu["f.router"].mul_(3.0), cpu["f.router.b"].mul_(5.0))), "f.")
    x = inputs([M], hidden, 10 + M, dtype)[0]
    got = m.forward(x.to(DEV), None).cpu().double()
    want = plain.experts_ff(x.double(), w, {"router": {"experts": E, "top": top}})
    if dtype == torch.float32:
        torch.testing.assert_close(got, want, **tol(dtype, 2.0))
    else:           # a close call of the router may fall the other way for a token: all but a few rows agree
        bad = ((got - want).abs() > 3e-2 * want.abs() + 4e-2).any(dim=1)
        assert int(bad.sum()) <= max(1, M // 50), f"{int(bad.sum())} of {M} rows differ"


def test_schedules_of_these_tests_hold_pieces_of_two_tokens():
    assert any(n == 2 for step in schedules([300, 129, 3])["pieces"] for _, n in step)
