"""Sofunex on the GPU against the plain restatement in oracle_sofunex.py."""
import ctypes as C
import json
import os
import subprocess
import sys

import pytest
import torch

import oracle_sofunex as O
import sofunex_cases as R
from saber_engine_b200.sched.scheduler import Scheduler, SchedulerConfig
from saber_engine_b200.serve.engine_api import EngineRequest, SamplingParams

pytestmark = pytest.mark.gpu
F32, BF16 = torch.float32, torch.bfloat16
REPO = os.path.dirname(os.path.dirname(os.path.abspath(__file__)))


# ------------------------------------------------------------------------------ mechanisms, a layer or two each
ALONE = {
    "attention_only": [R.layer(right=0.0)],
    "delta_only": [R.layer(left=0.0)],
    "both": [R.layer()],
    "negative_factors": [R.layer(left=-0.8, right=1.3)],
    "as_many_key_heads": [R.layer(heads=4, kv_heads=4, dim=40, vdim=8, rot=40, factor=1.0, right=0.1)],
    "odd_pairs": [R.layer(heads=4, kv_heads=2, dim=20, vdim=12, rot=6, factor=None, right=0.1)],
    "one_pair_one_key": [R.layer(heads=2, kv_heads=1, dim=8, vdim=48, rot=2, window=1, right=0.1)],
    "wide_attention": [R.layer(heads=2, kv_heads=1, dim=272, vdim=200, rot=264, right=0.1)],
    "one_tap": [R.layer(conv=1)],
    "many_taps": [R.layer(conv=7, window=7)],
    "odd_heads": [R.layer(heads=3, kv_heads=1, dim=18, vdim=7, rot=14, delta_heads=2, delta_dim=7)],
    "delta_of_64": [R.layer(left=0.0, delta_heads=2, delta_dim=64)],
    "delta_of_72": [R.layer(left=0.0, delta_heads=7, delta_dim=72)],
    "delta_of_200": [R.layer(left=0.0, delta_heads=1, delta_dim=200)],
    "delta_of_400": [R.layer(left=0.0, delta_heads=1, delta_dim=400)],
    "dense": [R.layer(mlp=R.dense(130))],
    "narrow_dense": [R.layer(mlp=R.dense(33))],
    "experts": [R.layer(mlp=R.moe())],
    "experts_without_groups": [R.layer(mlp=R.moe(10, 4, 24, None))],
    "experts_without_shared": [R.layer(mlp=R.moe(ff=136, shared=0))],
    "one_of_many_experts": [R.layer(mlp=R.moe(72, 1, 40, (9, 1), 248))],
    "second_layer": [R.layer(mlp=R.dense()), R.layer(window=20, conv=2)],
    "odd_width": [R.layer(mlp=R.dense(50)), R.layer(mlp=R.moe(ff=12, shared=20))],
}


@pytest.mark.parametrize("name", ALONE)
@pytest.mark.parametrize("dtype", [F32, BF16])
def test_mechanism_alone_residual_stream(name, dtype):
    cfg = R.config(ALONE[name], **({"width": 91} if name == "odd_width" else {}))
    t = R.tensors(cfg, seed=3)
    toks = R.tokens(cfg, 140)
    trace = []
    O.Oracle(cfg, t).forward(toks, trace)
    tol = (2e-5 if dtype == F32 else 0.02) * float(trace[-1].abs().max())
    eng = R.engine(cfg, t, dtype, rungs=(160,))
    eng.step([("a", toks)])
    b = next(iter(eng.model.buckets.values()))
    assert float((b.x[:140, : cfg["width"]].cpu().double() - trace[-1]).abs().max()) < tol
    for tok in toks[:70]:
        eng.step([("b", [tok])])
    x = eng.model.buckets[("decode", 1, 1)].x[:1, : cfg["width"]].cpu().double()
    assert float((x - trace[-1][69:70]).abs().max()) < tol


def _near(got, want, rel):
    assert float((got.double() - want).abs().max()) < rel * float(want.abs().max())


def _delta(H, D, rank, lens, pieces, w2_f32, seed, decays=None):
    """Read-outs [T, H, D] of sequences that arrive in pieces, and their states; and the oracle's."""
    from saber_engine_b200.models.stack_config import ChannelDeltaMixer
    from saber_engine_b200.ops import native as NN
    m, g = ChannelDeltaMixer(H, D, rank), torch.Generator().manual_seed(seed)
    n, DP, VP = H * D, m.dim_pad, m.vdim_pad
    rnd = lambda *s: torch.randn(*s, generator=g)      # noqa: E731
    w2, w0 = (rnd(n, rank) / rank ** 0.5).bfloat16(), rnd(n) if decays is None else torch.full((n,), decays)
    ld = (5 * n + rank + 8 * 6 + 7) // 8 * 8
    offs, at = {}, 0
    for name, k in m.segments():
        offs[name], at = at, (at + k + 7) // 8 * 8
    xs = [rnd(T, ld) for T in lens]
    S = len(lens)
    dev = dict(state=torch.zeros(S + 1, H, VP, DP, device="cuda"), w2=torch.nn.functional.pad(w2, (0, -rank % 16)).to(F32 if w2_f32 else BF16).contiguous().cuda(), w0=w0.cuda(),
               norm=(1 + 0.3 * rnd(n)).cuda())
    outs = [[] for _ in lens]
    done = [0] * S
    for piece in pieces:
        todo = [(j, min(p, lens[j] - done[j])) for j, p in enumerate(piece) if min(p, lens[j] - done[j]) > 0]
        M, nseq = sum(k for _, k in todo) + 3, len(todo) + 1                       # padding rows and a padding sequence
        x = torch.full((M, ld), 0.25)
        cu, slots, pos, r = [], [], torch.zeros(M, dtype=torch.int32), 0
        for j, k in todo:
            cu.append(r)
            slots.append(j + 1)
            x[r:r + k], pos[r:r + k] = xs[j][done[j]:done[j] + k], torch.arange(done[j], done[j] + k)
            r += k
        cu += [r, r]
        i32 = lambda v: torch.tensor(v, dtype=torch.int32, device="cuda")          # noqa: E731
        single = all(k == 1 for _, k in todo)
        blk = M // 4 + nseq
        buf = dict(x=x.cuda(), cu=i32(cu), slots=i32(slots + [-1]), pos=pos.cuda(), rec=torch.zeros(blk * H * (17 * DP + 64), device="cuda"),
                   vb=torch.zeros(blk * H * ((VP + 31) // 32) * 128, device="cuda"), o=torch.zeros(M * H * VP, device="cuda"),
                   out=torch.full((M, n + 64), 7.0, device="cuda"), err=torch.zeros(1, dtype=torch.int32, device="cuda"))
        p = NN.CdeltaParams()
        p.x, p.ldx, p.w2, p.w2_f32, p.rank, p.w0, p.norm_w, p.state = buf["x"].data_ptr(), ld, dev["w2"].data_ptr(), int(w2_f32), rank, dev["w0"].data_ptr(), \
            dev["norm"].data_ptr(), dev["state"].data_ptr()
        p.r_off, p.k_off, p.v_off, p.a_off, p.l_off, p.g_off = (offs[k] for k in ("r", "k", "v", "a", "w1", "g"))
        p.rec, p.vb, p.o, p.cu_rows, p.slots, p.pos, p.err = (buf[k].data_ptr() for k in ("rec", "vb", "o", "cu", "slots", "pos", "err"))
        p.out, p.out_k0, p.out_scale = NN.Operand(buf["out"].data_ptr(), M, n + 64, 1), 64, 0.5
        p.M, p.nseq, p.H, p.D, p.DP, p.VP, p.n_slots, p.eps, p.unit_eps = M, nseq, H, D, DP, VP, S + 1, 1e-5, 1e-6
        NN.check(NN.lib().saber_cdelta_launch(C.byref(p), int(single), NN.stream_handle()), "cdelta")
        torch.cuda.synchronize()
        assert int(buf["err"]) == 0
        got, r = buf["out"].cpu(), 0
        assert torch.all(got[:, :64] == 7.0) and torch.all(got[M - 3:] == 7.0)
        for j, k in todo:
            outs[j].append(got[r:r + k, 64:])
            r += k
            done[j] += k
    part = lambda x, name: x[:, offs[name]: offs[name] + n].double().view(-1, H, D)    # noqa: E731
    want, states = [], []
    for x in xs:
        z = torch.tanh(x[:, offs["w1"]: offs["w1"] + rank].double()) @ w2.double().T + w0.double()
        decay = torch.exp(-torch.exp(torch.tensor(-0.5).double()) * torch.sigmoid(z)).view(-1, H, D)
        o, s = O.delta_states(part(x, "r"), part(x, "k"), part(x, "v"), decay, torch.sigmoid(part(x, "a")))
        gate = torch.sigmoid(part(x, "g")).reshape(-1, n)
        want.append(O.rms(o, 1e-5).reshape(-1, n) * dev["norm"].cpu().double() * gate * 0.5)
        states.append(s)
    got = [torch.cat(o) if o else torch.zeros(0, n) for o in outs]
    return got, want, dev["state"].cpu(), states


@pytest.mark.parametrize("H,D,rank", [(3, 20, 9), (2, 64, 16), (5, 72, 1), (4, 128, 96), (2, 130, 33), (1, 7, 3), (1, 256, 70), (1, 321, 20), (1, 512, 130), (9, 48, 64)])
def test_channel_delta_rule(H, D, rank):
    """Ragged portions, single tokens and mixtures of them; read-outs and states."""
    lens = [90, 33, 5, 1]
    ragged = [[2, 7, 1, 1], [61, 1, 3, 0], [5, 20, 2, 0], [30, 30, 0, 0]]
    for pieces, w2_f32 in (([[90, 33, 5, 1]], True), ([[1, 1, 1, 1]] * 90, False), (ragged, False), (ragged, True)):
        got, want, st, states = _delta(H, D, rank, lens, pieces, w2_f32, H + D)
        for j in range(4):
            assert len(got[j]) == lens[j]
            _near(got[j], want[j], 2e-5)
            _near(st[j + 1, :, :D, :D].transpose(1, 2), states[j], 2e-5)
            assert not st[j + 1, :, D:].any() and not st[j + 1, :, :, D:].any()
        assert not st[0].any()


@pytest.mark.parametrize("decays", [-30.0, 0.0, 30.0])
def test_channel_delta_rule_over_long_sequences(decays):
    """From no decay at all to the fastest there is."""
    got, want, st, states = _delta(2, 40, 4, [700], [[650], *[[1]] * 20, [30]], True, 5, decays)
    _near(got[0], want[0], 5e-5)
    _near(st[1, :, :40, :40].transpose(1, 2), states[0], 5e-5)


def _route(z, corr, top, groups, keep, nt, live, scale=1.3):
    """Device routing tables of fp32 logits z [M, E]."""
    from saber_engine_b200.ops import native as NN
    M, E = z.shape
    zd = torch.zeros(M, E + 5, device="cuda")
    zd[:, :E] = z
    i32 = lambda *s: torch.full(s, -7, dtype=torch.int32, device="cuda")     # noqa: E731
    cap = (M * top + 15 * min(E, M * top) + 15) // 16 * 16 + 128
    d = dict(topk_id=i32(M, top), slot_of=i32(M, top), counts=i32(E).zero_(), offsets=i32(E + 1), cursors=i32(E), ntiles=i32(2),
             tiles=i32(min(E, M * top) + M * top // nt, 4), src_row=i32(cap), topk_w=torch.zeros(M, top, device="cuda"))
    lv, cd = torch.tensor([live], dtype=torch.int32, device="cuda"), corr.float().cuda()
    p = NN.MoeRouteParams()
    p.logits_f32, p.ld, p.M, p.E, p.top_k, p.nt, p.rows_cap, p.e_n, p.live, p.groups, p.keep = zd.data_ptr(), E + 5, M, E, top, nt, cap, E, lv.data_ptr(), groups, keep
    p.sigmoid, p.correction, p.scale = 1, cd.data_ptr(), scale
    for k, v in d.items():
        setattr(p, k, v.data_ptr())
    NN.check(NN.lib().saber_moe_route_launch(C.byref(p), NN.stream_handle()), "route")
    torch.cuda.synchronize()
    return {k: v.cpu() for k, v in d.items()}


@pytest.mark.parametrize("M,live", [(1, 1), (7, 5), (64, 64), (65, 60), (300, 300)])
@pytest.mark.parametrize("E,top,groups,keep", [(16, 4, 4, 3), (6, 6, 3, 3), (5, 1, 5, 1), (33, 5, 11, 2), (160, 8, 8, 3), (40, 3, 1, 1), (600, 32, 20, 5), (64, 8, 32, 9)])
def test_routing_by_sigmoid(M, live, E, top, groups, keep):
    """Choices and weights are the oracle's, with corrections that make every choice score negative or change the order."""
    g = torch.Generator().manual_seed(M * E)
    z, corr = torch.randn(M, E, generator=g) * 2, torch.randn(E, generator=g).float() * 0.7 - (2.0 if M % 2 else 0.0)
    nt = 16 if M <= 64 else 64
    d = _route(z, corr, top, groups, keep, nt, live)
    s = torch.sigmoid(z.double())
    for m in range(M):
        ids = d["topk_id"][m].tolist()
        if m >= live:
            assert ids == [-1] * top and d["slot_of"][m].tolist() == [-1] * top
            continue
        want = O.route(s[m].tolist(), corr.double().tolist(), top, {"count": groups, "keep": keep})
        assert ids == [e for e, _ in want]
        assert torch.allclose(d["topk_w"][m].double(), 1.3 * torch.tensor([w for _, w in want]).double(), rtol=3e-6, atol=1e-12)
        assert all(int(d["src_row"][int(r)]) == m for r in d["slot_of"][m])
    assert int((d["src_row"] >= 0).sum()) == live * top


def test_equal_choices_take_the_lower_group_and_expert():
    z, none = torch.zeros(3, 12), torch.zeros(12)
    assert _route(z, none, 4, 3, 2, 16, 3)["topk_id"].tolist() == [[0, 1, 2, 3]] * 3
    z[1, 9] = z[1, 4] = 1.0
    assert _route(z, none, 3, 3, 1, 16, 3)["topk_id"][1].tolist() == [4, 5, 6]
    z[2, 8:10], z[2, 0] = 0.6, 1.0                     # two good members beat one of the best
    d = _route(z, none, 2, 3, 1, 16, 3)
    assert d["topk_id"][2].tolist() == [8, 9] and torch.allclose(d["topk_w"][2], torch.tensor([0.65, 0.65]))
    low = torch.full((12,), -5.0)
    low[3] = -4.0
    d = _route(torch.full((1, 12), -200.0), low, 2, 3, 1, 16, 1)       # scores of zero: no share is infinite
    assert d["topk_id"][0].tolist() == [3, 0] and not d["topk_w"][0].any()


@pytest.mark.parametrize("M,W,rows", [(1, 40, 1), (7, 91, 4), (9, 130, 2), (40, 264, 4), (5, 5120, 1), (300, 72, 4)])
@pytest.mark.parametrize("what", ["embed", "result", "routed", "both"])
def test_join(M, W, rows, what):
    """Normed results, steps, the next norm and the blend with the token before, over sequence and strip borders."""
    from saber_engine_b200.ops import native as NN
    g = torch.Generator().manual_seed(M + W)
    rnd = lambda *s: torch.randn(*s, generator=g)      # noqa: E731
    wide, ldx = (W + 7) // 8 * 8, (W + 31) // 32 * 32
    pad = lambda v, n: torch.nn.functional.pad(v, (0, n - v.shape[-1])).contiguous().cuda()       # noqa: E731
    x, y, table, ids = rnd(M, W), rnd(M, W), rnd(11, W).bfloat16(), torch.randint(0, 11, (M,), generator=g)
    post, step, norm_w, shift = 1 + 0.3 * rnd(W), rnd(W), 1 + 0.3 * rnd(W), torch.rand(W, generator=g)
    routed, slot_of, route_w = rnd(2 * M, W).bfloat16(), torch.randint(-1, 2 * M, (M, 3), generator=g), torch.rand(M, 3, generator=g)
    cuts = sorted({0, min(M, 1), min(M, 6), M // 2, M - M // 5, M - M // 5})       # sequences of unequal lengths, then padding rows
    starts, ends = cuts[:-1], cuts[1:]
    if not starts:
        starts, ends = [0], [M]
    n = len(starts)
    pos = torch.zeros(M, dtype=torch.int64)
    for j, (a, b) in enumerate(zip(starts, ends)):
        pos[a:b] = torch.arange(b - a) + (0 if j == 1 else 17)
    state = rnd(n + 2, W)
    i32 = lambda v: torch.as_tensor(v, dtype=torch.int32).cuda()                   # noqa: E731
    dev = dict(x=pad(x, ldx), x_out=torch.zeros(M, ldx, device="cuda"), y=pad(y, wide), routed=pad(routed, wide), slot_of=i32(slot_of), route_w=route_w.cuda(),
               post_w=pad(post, wide), step=pad(step, wide), table=table.cuda(), ids=i32(ids), norm_w=pad(norm_w, wide), shift=pad(shift, wide), state=state.cuda(),
               cu_rows=i32(starts + [ends[-1]]), slots=i32(list(range(1, n + 1))), pos=i32(pos))
    op = torch.full((M, ldx), 5.0, device="cuda")
    p = NN.JoinParams()
    use = {"embed": ("table", "ids"), "result": ("y", "post_w", "x"), "routed": ("routed", "slot_of", "route_w", "post_w", "x"),
           "both": ("y", "routed", "slot_of", "route_w", "post_w", "x")}[what]
    for k in (*use, "x_out", "step", "norm_w", "shift", "state", "cu_rows", "slots", "pos"):
        setattr(p, k, dev[k].data_ptr())
    p.op, p.M, p.width, p.ldx, p.ldy, p.ldr, p.routes, p.vocab, p.nseq, p.n_slots = NN.Operand(op.data_ptr(), M, ldx, 1), M, W, ldx, wide, wide, 3, 11, n, n + 2
    p.rows, p.mult, p.embed_scale, p.eps = rows, 0.4, 2.5, 1e-5
    NN.check(NN.lib().saber_join_launch(C.byref(p), NN.stream_handle()), "join")
    torch.cuda.synchronize()
    z = torch.zeros(M, W).double()
    if what in ("result", "both"):
        z = z + y.double()
    if what in ("routed", "both"):
        for m in range(M):
            z[m] += sum((route_w[m, k].double() * routed[slot_of[m, k]].double() for k in range(3) if slot_of[m, k] >= 0), torch.zeros(W).double())
    new = (table[ids].double() * 2.5 if what == "embed" else x.double() + 0.4 * O.rms(z, 1e-5, post.double())) + step.double()
    h = O.rms(new, 1e-5, norm_w.double())
    live = ends[-1]
    _near(dev["x_out"][:live, :W].cpu(), new[:live], 2e-6)
    for j, (a, b) in enumerate(zip(starts, ends)):
        first = state[j + 1].double() if pos[a] > 0 else torch.zeros(W).double()
        before = torch.cat([first[None], h[a:b - 1]])
        _near(op[a:b, :W].cpu(), h[a:b] + (before - h[a:b]) * shift.double(), 4e-6)
        _near(dev["state"][j + 1].cpu(), h[b - 1], 4e-6)
    assert torch.equal(dev["state"][0].cpu(), state[0]) and torch.equal(dev["state"][n + 1].cpu(), state[n + 1])
    # without a blend the stream is updated in place
    p.shift, p.state, p.x_out = None, None, dev["x_out"].data_ptr()
    op.fill_(5.0)
    if what != "embed":
        dev["x_out"].copy_(dev["x"])
        p.x = dev["x_out"].data_ptr()
    NN.check(NN.lib().saber_join_launch(C.byref(p), NN.stream_handle()), "join")
    torch.cuda.synchronize()
    _near(op[:, :W].cpu(), h, 4e-6)
    _near(dev["x_out"][:, :W].cpu(), new, 2e-6)


@pytest.mark.parametrize("fuse", [True, False])
@pytest.mark.parametrize("act", ["gelu_tanh", "silu"])
@pytest.mark.parametrize("M,K,ff,splits,f32", [(3, 64, 40, 1, 0), (17, 640, 300, 5, 0), (300, 192, 250, 1, 0), (5, 64, 130, 1, 1)])
def test_gated_units(M, K, ff, splits, f32, act, fuse):
    """Stored columns with a bias, then gate | up tiles through either activation, out to large arguments."""
    from saber_engine_b200.models import stack_weights as SW
    from saber_engine_b200.models.stack_config import GATED_ACTS
    from saber_engine_b200.ops import functional as F
    from saber_engine_b200.ops import layouts as L
    from saber_engine_b200.ops import native as NN
    dt = F32 if f32 else BF16
    g = torch.Generator().manual_seed(M + K)
    rnd = lambda *s: torch.randn(*s, generator=g)      # noqa: E731
    gate, up, rows, a = (3 * rnd(ff, K) / K ** 0.5).to(BF16), (rnd(ff, K) / K ** 0.5).to(BF16), (rnd(20, K) / K ** 0.5).to(BF16), rnd(M, K).to(BF16)
    a[0] *= 30
    w = torch.zeros(256, K, dtype=BF16)
    w[:20] = rows
    lin = SW.pack_linear(torch.cat([w, SW.gated_rows(gate, up, K)]).cuda(), dt)
    m_pad, ka, bias = L.padded_rows(M), L.round_up(ff, 128), rnd(24).cuda()
    if f32:
        op = torch.zeros(m_pad, K)
        op[:M] = a.float()
        op, act_op = op.cuda(), torch.full((m_pad, ka), 5.0, device="cuda")
    else:
        op, act_op = torch.zeros(K // 64, m_pad, 8, 8, dtype=BF16), torch.full((ka // 64, m_pad, 8, 8), 5.0, dtype=BF16, device="cuda")
        r, ch = torch.arange(M)[:, None], torch.arange(8)[None, :]
        for kb in range(K // 64):
            op[kb, r, ch ^ (r & 7)] = a[:, kb * 64:(kb + 1) * 64].reshape(M, 8, 8)
        op = op.cuda()
    out, ws, sc = torch.full((M, 32), 7.0, device="cuda"), torch.zeros(M * lin.N_pad + (1 << 22), device="cuda"), F.scratch("cuda")
    p = NN.LinParams()
    p.w, p.a, p.err, p.ws, p.counters = lin.w.data_ptr(), op.data_ptr(), sc.err.data_ptr(), ws.data_ptr(), sc.counters.data_ptr()
    p.M, p.M_pad, p.N_pad, p.K, p.nt, p.splits, p.fuse, p.fp32, p.mtiles = M, m_pad, lin.N_pad, K, L.token_tile(M), splits, int(fuse), f32, 1
    e = p.e
    e.out, e.ldo, e.n_plain, e.act_tile0, e.bias = out.data_ptr(), 32, 24, 1, bias.data_ptr()
    e.act, e.act_kind = NN.Operand(act_op.data_ptr(), m_pad, ka, f32), GATED_ACTS[act]
    NN.check(NN.lib().saber_linear_launch(C.byref(p), NN.stream_handle()), "linear")
    torch.cuda.synchronize()
    sc.check()
    _near(out[:, :20].cpu(), a.double() @ rows.double().T + bias[:20].cpu().double(), 2e-5)
    assert torch.all(out[:, 24:] == 7.0)
    want = getattr(O, act)(a.double() @ gate.double().T) * (a.double() @ up.double().T)
    got = act_op.cpu()
    if not f32:
        got = torch.cat([got[kb, r, ch ^ (r & 7)].reshape(M, 64) for kb in range(ka // 64)], 1)
    assert float(((got[:M, :ff].double() - want).abs() / (want.abs() + 0.05)).max()) < (2e-4 if f32 else 0.01)
    assert torch.all(got[:M, ff:] == 0)


# ------------------------------------------------------------------------------ whole models
@pytest.fixture(scope="module", params=list(R.CASES))
def case(request):
    cfg = R.CASES[request.param]
    t = R.tensors(cfg, seed=len(request.param))
    toks = R.tokens(cfg, 150)
    return cfg, t, toks, O.Oracle(cfg, t).forward(toks)


@pytest.mark.parametrize("dtype", [F32, BF16])
def test_whole_decode_and_portions(case, dtype):
    cfg, t, toks, want = case
    eng = R.engine(cfg, t, dtype, kv_blocks=4)                   # three pages: every request uses them again
    for cuts in ([150], [1], [2, 2, 3, 61, 2, 5, 64, 2], [63, 1, 1, 64, 2], [100, 2]):
        assert R.error(R.feed(eng, "r", toks, cuts), want) < R.TOL[dtype], cuts


@pytest.mark.parametrize("dtype", [F32, BF16])
def test_unequal_batch_against_each_alone_with_pages_and_slots_used_again(case, dtype):
    cfg, t, _, _ = case
    orc = O.Oracle(cfg, t)
    lens = {"a": 131, "b": 3, "c": 66, "d": 20, "e": 64, "f": 1, "g": 90}
    toks = {k: R.tokens(cfg, n, seed=i) for i, (k, n) in enumerate(lens.items())}
    eng = R.engine(cfg, t, dtype, kv_blocks=9)
    g = torch.Generator().manual_seed(5)
    at, out, queue, live = {k: 0 for k in lens}, {k: [] for k in lens}, list(lens), []
    while queue or live:
        while queue and len(live) < 4:
            live.append(queue.pop(0))
        entries = []
        for k in live:
            if len(live) > 1 and float(torch.rand((), generator=g)) < 0.2:
                continue                                         # left out of this step
            n = [1, 2, 40, 7][int(torch.randint(0, 4, (), generator=g))]
            entries.append((k, toks[k][at[k]: at[k] + n]))
        if not entries:
            continue
        for (k, tk), rows in zip(entries, eng.step(entries)):
            out[k].append(rows)
            at[k] += len(tk)
        for k in [k for k in live if at[k] == lens[k]]:
            eng.end(k)
            live.remove(k)
    for k in lens:
        assert R.error(torch.cat(out[k]), orc.forward(toks[k])) < R.TOL[dtype], k
    assert eng.arenas.kv.free_blocks == 8 and eng.arenas.gdn.free_slots == 4


def test_attention_forms_agree():
    cfg = R.config([R.layer(heads=12, kv_heads=3, dim=72, vdim=100, rot=40, window=150, right=0.1), R.layer(heads=4, kv_heads=1, dim=40, vdim=128, rot=24, window=90)], width=264)
    t = R.tensors(cfg, seed=9)
    toks = R.tokens(cfg, 333)
    want = O.Oracle(cfg, t).forward(toks)
    for impl, form in (("tc", 2), ("mma", 1)):
        eng = R.engine(cfg, t, BF16, attn_impl=impl)
        assert eng.model._gqa_form(eng.model.cfg.layers[0].mixer.left, 256, False) == form
        for cuts in ([333], [70, 130, 2]):
            assert R.error(R.feed(eng, "r", toks, cuts), want) < R.TOL[BF16]


# ------------------------------------------------------------------------------ windows, far keys, borders, long runs
def _needle(cfg: dict, seed: int):
    """Weights with a needle: the query of the last token id meets the key of token id 1 with a score far above all others, wherever that token
    stands inside the window.  Its coordinate passes blend and convolution untouched, so that one position alone holds the key."""
    t = R.tensors(cfg, seed)
    W, m = cfg["width"], cfg["layers"][0]["mixer"]["left"]
    t["embed"][:, :2] = 0.0
    t["embed"][1, 0] = 9.0                                       # only the needle has this coordinate
    t["embed"][cfg["vocab"] - 1, 1] = 9.0
    t["l0.norm1"][:2], t["l0.shift"][:2], t["head"][:, :2] = 1.0, 0.0, 0.0
    for n, heads, coord in (("q", m["heads"], 1), ("k", m["kv_heads"], 0)):
        w, last = t[f"l0.mix.left.{n}"].view(heads, m["dim"], W), m["dim"] - 1
        w[:, :, coord] = 0.0
        w[:, last, coord] = 6.0
        w[:, last, [c for c in range(W) if c != coord]] = 0.0    # the last value of a head (it does not turn) is the needle's
        t[f"l0.mix.left.{n}.b"].view(heads, m["dim"])[:, last] = 0.0
        conv = t[f"l0.mix.left.{n}.conv"].view(heads, m["dim"], -1)
        conv[:, last] = 0.0
        conv[:, last, -1] = 1.0
        t[f"l0.mix.left.{n}.norm"].view(heads, m["dim"])[:, last] = 1.0
    return t


def _asking(cfg, n, place, seed=0):
    """A prompt whose last token asks for a needle at `place`."""
    toks = [2 + x % (cfg["vocab"] - 4) for x in R.tokens(cfg, n, seed)]
    toks[place], toks[-1] = 1, cfg["vocab"] - 1
    return toks


@pytest.mark.parametrize("dtype", [F32, BF16])
@pytest.mark.parametrize("window", [1000, 300, 128, 64, 65, 7, 2])
def test_one_key_far_back_at_page_edges_and_at_the_window_edge(dtype, window):
    cfg = R.config([R.layer(heads=6, kv_heads=2, dim=24, vdim=20, rot=8, scale=1.0, window=window, right=0.1)], vocab=131, mult=4.0)
    t = _needle(cfg, 2)
    n = 420
    orc = O.Oracle(cfg, t)
    tol = {F32: 5e-5, BF16: 0.08}[dtype]
    engs = [R.engine(cfg, t, dtype, rungs=(64, 512), **kw) for kw in ({}, {"attn_impl": "mma"})]
    edge = n - window                                            # the first key that the last token sees
    places = {n - 2, max(edge, 0), max(edge + 1, 0)} | {p for p in (edge - 1, edge - 2, 0, 63, 64, 127, 128, 383, 384) if 0 <= p < n - 1}
    for place in sorted(p for p in places if p < n - 1):
        toks = _asking(cfg, n, place)
        want = orc.forward(toks)
        without = list(toks)
        without[place] = 2
        far = R.error(orc.forward(without)[-1:], want[-1:])
        if edge <= place:
            assert far > 0.2                                     # the answer hangs on that one key
        for eng in engs:
            for cuts in ([n], [n - 1, 1], [n - 2, 2], [max(1, place), 1, 2, 200, 255, 1]):
                assert R.error(R.feed(eng, "r", toks, cuts)[-1:], want[-1:]) < tol, (place, cuts)
    if 0 < edge:                                                 # a key that has just left the window shows in nobody's scores
        other = json.loads(json.dumps(cfg))
        other["layers"][0]["mixer"]["left"]["mask"]["size"] = window + 1
        toks = _asking(cfg, n, edge - 1)
        assert R.error(O.Oracle(other, t).forward(toks)[-1:], orc.forward(toks)[-1:]) > 0.2


@pytest.mark.parametrize("dtype", [F32, BF16])
def test_window_edge_passes_over_decoded_tokens(dtype):
    """Needles are written while decoding and leave the window while decoding; every token asks."""
    cfg = R.config([R.layer(heads=4, kv_heads=2, dim=24, vdim=20, rot=8, scale=1.0, window=66, right=0.1)], vocab=131, mult=4.0)
    t = _needle(cfg, 3)
    toks = [2 + x % 120 for x in R.tokens(cfg, 260)]
    for i in range(5, 260, 9):
        toks[i] = 1 if i % 4 else 130
    want = O.Oracle(cfg, t).forward(toks)
    for cuts in ([260], [63, 1, 1, 63, 2, 50, 1], [120, 1], [1]):
        eng = R.engine(cfg, t, dtype)
        assert R.error(R.feed(eng, "r", toks, cuts), want) < {F32: 5e-5, BF16: 0.1}[dtype], cuts


@pytest.mark.parametrize("dtype", [F32, BF16])
def test_a_token_far_back_in_the_state(dtype):
    """Slow decays and one token whose value stands out: the state alone carries it over portions, steps and page borders."""
    cfg = R.config([R.layer(window=3, left=0.05, delta_heads=2, delta_dim=40)], vocab=131, mult=1.0)
    t = R.tensors(cfg, 4)
    t["l0.mix.right.w0"][:] = -9.0
    t["l0.mix.right.a.b"][:] = -6.0
    t["embed"][:, 0] = 0.0
    t["embed"][1, 0] = 9.0
    t["l0.mix.right.v"][:, 0] *= 300
    n, orc = 400, O.Oracle(cfg, t)
    for place in (0, 1, 63, 64, 200):
        toks = [2 + x % 120 for x in R.tokens(cfg, n)]
        without = list(toks)
        toks[place] = 1
        want = orc.forward(toks)
        assert R.error(orc.forward(without)[-1:], want[-1:]) > 0.2
        eng = R.engine(cfg, t, dtype)
        for cuts in ([n], [n - 1, 1], [max(1, place), 1, 2, 200, 3, 1]):
            assert R.error(R.feed(eng, "r", toks, cuts), want) < R.TOL[dtype], (place, cuts)


@pytest.mark.parametrize("dtype", [F32, BF16])
@pytest.mark.parametrize("conv", [1, 2, 3, 6])
def test_neighbours_over_portion_borders(dtype, conv):
    """The token before and the convolution's inputs cross every cut: taps and blends that count fully."""
    cfg = R.config([R.layer(conv=conv, window=40), R.layer(conv=conv, window=5)], mult=1.0)
    t = R.tensors(cfg, 6)
    for i in range(2):
        t[f"l{i}.shift"][:] = torch.linspace(-0.5, 1.5, cfg["width"]).bfloat16()
        for n in "qkv":
            t[f"l{i}.mix.left.{n}.conv"][:] = torch.linspace(1.0, 0.5, conv).bfloat16()
    toks = R.tokens(cfg, 70)
    want = O.Oracle(cfg, t).forward(toks)
    for i in (3, 17, 64):
        changed = list(toks)
        changed[i - 1] = (changed[i - 1] + 1) % cfg["vocab"]
        assert R.error(O.Oracle(cfg, t).forward(changed)[i:i + 1], want[i:i + 1]) > 0.1
    eng = R.engine(cfg, t, dtype)
    for cuts in ([70], [1], [2], [3], [4, 1], [5, 2, 7, 1], [64, 1, 5], [63, 2]):
        assert R.error(R.feed(eng, "r", toks, cuts), want) < R.TOL[dtype], cuts


@pytest.mark.parametrize("a", [dict(dim=64, rot=48, base=20.0, factor=1.0), dict(dim=64, rot=64, base=5000.0, factor=16.0), dict(dim=8, rot=8, base=40.0, factor=0.5)])
def test_rotations(a):
    cfg = R.config([R.layer(heads=2, kv_heads=1, vdim=24, scale=0.8, window=300, right=0.1, **a)])
    t = R.tensors(cfg, 6)
    toks = R.tokens(cfg, 300)
    want = O.Oracle(cfg, t).forward(toks)
    for change in ({"base": a["base"] * 1.5}, {"scaling": {"factor": a["factor"] * 2}}):
        other = json.loads(json.dumps(cfg))
        other["layers"][0]["mixer"]["left"]["rot"].update(change)
        assert R.error(O.Oracle(other, t).forward(toks), want) > 0.01
    for dtype in (F32, BF16):
        eng = R.engine(cfg, t, dtype)
        for cuts in ([300], [255, 2, 43], [64, 1]):
            assert R.error(R.feed(eng, "r", toks, cuts), want) < R.TOL[dtype], (dtype, cuts)


def test_passes_of_a_loop_have_their_own_vectors_and_states():
    cfg = R.config([R.layer(mlp=R.dense()), R.layer(window=12, mlp=R.moe())], loop=(0, 2, 3))
    t = R.tensors(cfg, 7)
    toks = R.tokens(cfg, 90)
    want = O.Oracle(cfg, t).forward(toks)
    swapped = {**t, "loop.step": t["loop.step"][[0, 2, 1]]}
    assert R.error(O.Oracle(cfg, swapped).forward(toks), want) > 0.02
    for dtype in (F32, BF16):
        eng = R.engine(cfg, t, dtype)
        assert len(eng.model.slot_tensors()) == 3 * 6 and len(eng.model.page_pools()) == 6
        for cuts in ([90], [30, 1], [2, 40, 3]):
            assert R.error(R.feed(eng, "r", toks, cuts), want) < R.TOL[dtype], cuts


@pytest.mark.parametrize("lens", [(300,), (129, 64, 1, 257), (1, 1, 2, 3)])
def test_unequal_prompts_in_one_bucket(lens):
    cfg = R.config([R.layer(heads=6, kv_heads=3, dim=48, vdim=56, window=100, mlp=R.moe()), R.layer(mlp=R.moe(ff=72))], vocab=800)
    t = R.tensors(cfg, 5)
    toks = [R.tokens(cfg, n, seed=i) for i, n in enumerate(lens)]
    orc = O.Oracle(cfg, t)
    for dtype in (BF16, F32):
        eng = R.engine(cfg, t, dtype, rungs=(1024,))
        for _ in range(2):                                       # the second time in slots and pages used before
            got = eng.step([(i, x) for i, x in enumerate(toks)])
            for i, (g, x) in enumerate(zip(got, toks)):
                assert R.error(g, orc.forward(x)) < R.TOL[dtype]
                eng.end(i)


@pytest.mark.parametrize("dtype", [F32, BF16])
@pytest.mark.parametrize("spread", ["one_expert", "all"])
def test_expert_rows_fill_and_overflow_tiles(dtype, spread):
    """All tokens on one expert (many tiles of it), or spread evenly."""
    cfg = R.config([R.layer(mlp=R.moe(16, 1, 24, (4, 2), 0))], vocab=64)
    t = R.tensors(cfg, 5)
    t["l0.mlp.router"][:], t["l0.mlp.correction"][:] = 0, 0
    t["l0.norm1b"][:16] = 0
    if spread == "one_expert":
        t["l0.mlp.correction"][11] = 0.5
    else:
        t["embed"][:, :16], t["l0.norm2"][:16] = 0, 1.0
        t["embed"][torch.arange(64), torch.arange(64) % 16] = 2.0
        t["l0.mlp.router"][torch.arange(16), torch.arange(16)] = 8.0
    for n in (300, 16, 1):
        toks = [x % 64 for x in range(n)]
        want = O.Oracle(cfg, t).forward(toks)
        eng = R.engine(cfg, t, dtype)
        for cuts in ([n], [max(1, n - 3), 1]):
            assert R.error(R.feed(eng, "r", toks, cuts), want) < R.TOL[dtype]


@pytest.mark.parametrize("n", [1, 2, 3, 4, 5])
def test_first_tokens(n):
    cfg = R.CASES["every_kind"]
    t = R.tensors(cfg, 8)
    toks = R.tokens(cfg, n)
    want = O.Oracle(cfg, t).forward(toks)
    for dtype in (F32, BF16):
        eng = R.engine(cfg, t, dtype)
        for cuts in ([n], [1], [2]):
            assert R.error(R.feed(eng, "r", toks, cuts), want) < R.TOL[dtype]


def test_long_decoding_over_page_borders():
    cfg = R.CASES["every_kind"]
    t = R.tensors(cfg, 10)
    toks = R.tokens(cfg, 330)
    want = O.Oracle(cfg, t).forward(toks)
    for dtype in (F32, BF16):
        eng = R.engine(cfg, t, dtype, capture=True)
        assert R.error(R.feed(eng, "r", toks, [10, 1]), want) < R.TOL[dtype]


def test_mixers_beside_each_other_and_in_line_agree():
    """Captured and eager, with the first mixer on a stream of its own or not: the same numbers."""
    cfg = R.CASES["every_kind"]
    t = R.tensors(cfg, 13)
    toks = R.tokens(cfg, 80)
    got = [R.feed(R.engine(cfg, t, BF16, capture=capture, side_stream=side), "r", toks, [40, 1]) for side in (True, False) for capture in (True, False)]
    assert R.error(got[0], O.Oracle(cfg, t).forward(toks)) < R.TOL[BF16]
    assert all(torch.equal(g, got[0]) for g in got[1:])


def test_unfused_linears_agree():
    cfg = R.CASES["every_kind"]
    t = R.tensors(cfg, 11)
    toks = R.tokens(cfg, 90)
    want = O.Oracle(cfg, t).forward(toks)
    eng = R.engine(cfg, t, BF16, fuse=False)
    for cuts in ([90], [80, 1]):
        assert R.error(R.feed(eng, "r", toks, cuts), want) < R.TOL[BF16]


# ------------------------------------------------------------------------------ through the engine
def _collect(sub):
    toks = []
    while True:
        ev = sub.events.get(timeout=60)
        toks += ev.new_token_ids
        if ev.finished:
            return toks, ev


@pytest.fixture(scope="module")
def served():
    from saber_engine_b200.runtime.hybrid_executor import HybridExecutor
    cfg = R.CASES["every_kind"]
    t = R.tensors(cfg, 12)
    m = R.model(cfg, t, F32, max_seqs=4, max_ctx=512)
    return cfg, O.Oracle(cfg, t), HybridExecutor(m, decode_batches=(1, 2, 4), decode_widths=(1,), prefill_rungs=(32, 128))


def _sched(ex, **kw):
    from saber_engine_b200.serve.sampler import HostSampler
    return Scheduler(ex, SchedulerConfig(max_seqs=4, max_ctx=512, prefix_cache_min_tokens=64, prefix_cache_interval=64, **kw), sampler=HostSampler())


def _greedy(sched, prompts, n):
    subs = [sched.submit(EngineRequest(p, SamplingParams(max_tokens=n, ignore_eos=True))) for p in prompts]
    sched.run_until_idle()
    return [_collect(s) for s in subs]


def test_greedy_generation_through_the_scheduler(served):
    cfg, orc, ex = served
    prompts = [R.tokens(cfg, n, seed=20 + n) for n in (3, 45, 140, 64, 9)]       # five requests, four slots
    want = [orc.greedy(p, 12) for p in prompts]
    assert min(gap for _, gap in want) > 1e-4
    got = _greedy(_sched(ex, prefix_cache=False), prompts, 12)
    assert [g[0] for g in got] == [w[0] for w in want]
    assert ex.census["graph_replays"] > 0


def test_prefix_cache_parking_and_sampling(served, tmp_path):
    cfg, orc, ex = served
    shared = R.tokens(cfg, 128, seed=31)
    p1, p2 = shared + R.tokens(cfg, 10, seed=32), shared + R.tokens(cfg, 17, seed=33)
    want = [orc.greedy(p, 8)[0] for p in (p1, p2)]
    s = _sched(ex)
    assert _greedy(s, [p1], 8)[0][0] == want[0]
    toks, ev = _greedy(s, [p2], 8)[0]
    assert toks == want[1] and ev.cached_tokens == 128
    # a parked session comes back in other pages and another slot
    from saber_engine_b200.sched.park import ParkTier
    s = _sched(ex, prefix_cache=False)
    s.park_tier = ParkTier(ram_budget=1, directory=str(tmp_path))
    sub = s.submit(EngineRequest(p1, SamplingParams(max_tokens=8, ignore_eos=True)))
    for _ in range(5):
        s.step()
    key = s.park(sub.seq_id)
    other = s.submit(EngineRequest(p2, SamplingParams(max_tokens=8, ignore_eos=True)))
    for _ in range(2):
        s.step()
    s.restore(key)
    s.run_until_idle()
    assert _collect(sub)[0] == want[0] and _collect(other)[0] == want[1]
    # sampled: top_k = 1 is greedy, a seed fixes the ids
    s = _sched(ex, prefix_cache=False)
    kw = dict(max_tokens=8, ignore_eos=True)
    subs = [s.submit(EngineRequest(p1, SamplingParams(temperature=1.0, top_k=1, seed=3, **kw))),
            s.submit(EngineRequest(p1, SamplingParams(temperature=1.3, seed=4, **kw))),
            s.submit(EngineRequest(p1, SamplingParams(temperature=1.3, seed=4, logprobs=2, **kw)))]
    s.run_until_idle()
    a, b, c = [_collect(x)[0] for x in subs]
    assert a == want[0] and b == c


@pytest.mark.parametrize("dtype", ["bfloat16", "float32"])
def test_trace_replay_process(tmp_path, dtype):
    cfg = R.CASES["loop_first_to_last"]
    t = R.tensors(cfg, 14)
    R.write_model(tmp_path / "m", cfg, t)
    a, b = R.tokens(cfg, 75, seed=1), R.tokens(cfg, 30, seed=2)
    steps = [{"step": 0, "entries": [{"id": "a", "tokens": a[:70], "want": [0, 69]}, {"id": "b", "tokens": b[:1], "want": []}], "end": []},
             {"step": 1, "entries": [{"id": "a", "tokens": a[70:71], "want": []}, {"id": "b", "tokens": b[1:29], "want": []}], "end": []},
             {"step": 2, "entries": [{"id": "b", "tokens": b[29:], "want": [0]}, {"id": "a", "tokens": a[71:], "want": [3, 1]}], "end": ["a", "b"]},
             {"step": 3, "entries": [{"id": "c", "tokens": a[:64], "want": [63]}], "end": ["c"]}]
    r = subprocess.run([os.path.join(REPO, "bin", "trace_run"), "--model", str(tmp_path / "m"), "--dtype", dtype, "--out", str(tmp_path),
                        "--max-tokens", "192"], input="".join(json.dumps(s) + "\n" for s in steps), capture_output=True, text=True, timeout=240,
                       env={**os.environ, "PATH": os.path.dirname(sys.executable) + os.pathsep + os.environ["PATH"]})
    assert r.returncode == 0, r.stderr[-2000:]
    assert [x for x in r.stdout.splitlines() if x.startswith("done")] == [f"done {i}" for i in range(4)]
    import numpy as np
    orc = O.Oracle(cfg, t)
    la, lb = orc.forward(a), orc.forward(b)
    want = {0: la[[0, 69]], 2: torch.stack([lb[29], la[74], la[72]]), 3: la[[63]]}
    assert not (tmp_path / "1.f32").exists()
    for k, w in want.items():
        got = torch.from_numpy(np.fromfile(tmp_path / f"{k}.f32", dtype="<f4").reshape(-1, cfg["vocab"]))
        assert R.error(got, w) < R.TOL[getattr(torch, dtype)]


def test_engine_command_serves_a_model_folder(tmp_path):
    """`saber engine --engine-config DIR`: plan, weights, scheduler; greedy ids of the oracle."""
    from saber_engine_b200.cli.main import build_engine, make_parser
    cfg = R.CASES["groups_of_one"]
    t = R.tensors(cfg, 15)
    R.write_model(tmp_path / "m", cfg, t)
    a = make_parser().parse_args(["engine", "--engine-config", str(tmp_path / "m"), "--engine-dtype", "float32", "--engine-max-ctx", "512",
                                  "--engine-max-seqs", "2", "--engine-prefill-rows", "64", "--engine-decode-batches", "1,2",
                                  "--engine-budget-mib", "12000", "--engine-race-check", "shadow"])
    ex, sched = build_engine(a)
    prompts = [R.tokens(cfg, n, seed=50 + n) for n in (5, 70, 33)]
    want = [O.Oracle(cfg, t).greedy(p, 8)[0] for p in prompts]
    assert [g[0] for g in _greedy(sched, prompts, 8)] == want
    b = ex.model.buckets[("decode", 2, 1)]
    assert int((b.digests.cpu() != 0).sum()) >= len(cfg["layers"])
