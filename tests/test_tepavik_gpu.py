"""Tepavik on the GPU against the plain restatement in oracle_tepavik.py."""
import ctypes as C
import json
import os
import subprocess
import sys

import pytest
import torch

import oracle_tepavik as O
import tepavik_cases as R
from saber_engine_b200.sched.scheduler import Scheduler, SchedulerConfig
from saber_engine_b200.serve.engine_api import EngineRequest, SamplingParams

pytestmark = pytest.mark.gpu
F32, BF16 = torch.float32, torch.bfloat16
REPO = os.path.dirname(os.path.dirname(os.path.abspath(__file__)))


# ------------------------------------------------------------------------------ mechanisms, one or two layers each
ALONE = {
    "lightning": [R.lightning(ff=None)],
    "lightning_one_head": [R.lightning(heads=1, dim=128, vdim=8, decay=(0.97,), ff=None)],
    "lightning_wide_norm": [R.lightning(heads=70, dim=8, vdim=64, decay=[0.9 + h / 1000 for h in range(70)], ff=None)],
    "lightning_small_heads": [R.lightning(heads=80, dim=16, vdim=8, decay=[0.9 + h / 1000 for h in range(80)], ff=None)],
    "mamba": [R.mamba(ff=None)],
    "mamba_one_group_no_history": [R.mamba(heads=4, groups=1, conv=1, norm_groups=1, ff=None)],
    "mamba_groups_across_heads": [R.mamba(heads=6, groups=6, vdim=8, conv=6, norm_groups=16, state=130, ff=None)],
    "attention": [R.attention(ff=None)],
    "attention_small_chunk": [R.attention(chunk=3, heads=4, kv_heads=4, dim=40, vdim=8, ff=None)],
    "attention_of_another_layer": [R.attention(ff=None), R.attention(ff=None, kv_from=0, chunk=9, scale=0.7)],
    "feed_forward": [R.lightning(ff=130)],
    "narrow_feed_forward": [R.attention(ff=33)],
}


@pytest.mark.parametrize("name", ALONE)
@pytest.mark.parametrize("dtype", [F32, BF16])
def test_mechanism_alone_residual_stream(name, dtype):
    cfg = R.config(ALONE[name])
    t = R.tensors(cfg, seed=3)
    toks = R.tokens(cfg, 140)
    trace = []
    O.Oracle(cfg, t).forward(toks, trace)
    eng = R.engine(cfg, t, dtype, rungs=(160,))
    eng.step([("a", toks)])
    b = next(iter(eng.model.buckets.values()))
    x = b.x[:140, : cfg["width"]].cpu().double()
    assert float((x - trace[-1]).abs().max() / trace[-1].abs().max()) < (1e-5 if dtype == F32 else 0.03)
    for tok in toks[:70]:
        eng.step([("b", [tok])])
    x = eng.model.buckets[("decode", 1, 1)].x[:1, : cfg["width"]].cpu().double()
    assert float((x - trace[-1][69:70]).abs().max() / trace[-1].abs().max()) < (1e-5 if dtype == F32 else 0.03)


@pytest.mark.parametrize("fuse", [True, False])
@pytest.mark.parametrize("M,N,K,splits", [(1, 40, 64, 1), (7, 520, 640, 5), (130, 300, 192, 1), (300, 1000, 128, 1)])
def test_linear_bias_and_squared_relu(M, N, K, splits, fuse):
    """Stored columns with a bias behind the row scale, then tiles of 256 through max(., 0)^2."""
    from saber_engine_b200.models import stack_weights as SW
    from saber_engine_b200.ops import functional as F
    from saber_engine_b200.ops import layouts as L
    from saber_engine_b200.ops import native as NN
    g = torch.Generator().manual_seed(M + N)
    plain = N // 2
    tile0 = (plain + 255) // 256
    ff = N - plain
    w = (torch.randn(N, K, generator=g) / K ** 0.5).bfloat16()
    a = torch.randn(M, K, generator=g).bfloat16()
    n_pad = tile0 * 256 + L.round_up(ff, 256)
    wp = torch.zeros(n_pad, K, dtype=BF16)
    wp[:plain], wp[tile0 * 256: tile0 * 256 + ff] = w[:plain], w[plain:]
    lin = SW.pack_linear(wp.cuda(), BF16)
    m_pad = L.padded_rows(M)
    op = torch.zeros(K // 64, m_pad, 8, 8, dtype=BF16)
    rows, chunk = torch.arange(M)[:, None], torch.arange(8)[None, :]
    for kb in range(K // 64):
        op[kb, rows, chunk ^ (rows & 7)] = a[:, kb * 64:(kb + 1) * 64].reshape(M, 8, 8)
    op = op.cuda()
    sc = F.scratch("cuda")
    ss = torch.rand(m_pad, 3, generator=g).cuda() + 0.5
    ws = torch.zeros(M * n_pad + (1 << 22), dtype=F32, device="cuda")
    bias = torch.randn(L.round_up(plain, 8), generator=g).cuda()
    out = torch.full((M, L.round_up(plain, 8) + 8), 7.0, dtype=F32, device="cuda")
    ka = L.round_up(ff, 64)
    act = torch.full((ka // 64, m_pad, 8, 8), 5.0, dtype=BF16, device="cuda")
    p = NN.LinParams()
    p.w, p.a, p.err, p.ws, p.counters = lin.w.data_ptr(), op.data_ptr(), sc.err.data_ptr(), ws.data_ptr(), sc.counters.data_ptr()
    p.M, p.M_pad, p.N_pad, p.K, p.nt, p.splits, p.fp32, p.fuse = M, m_pad, n_pad, K, L.token_tile(M), splits, 0, int(fuse)
    p.mtiles = 2 if m_pad % 256 == 0 else 1
    e = p.e
    e.ss, e.ss_n, e.inv_width, e.eps, e.out, e.ldo, e.n_plain, e.act_tile0 = ss.data_ptr(), 3, 0.25, 1e-3, out.data_ptr(), out.stride(0), plain, tile0
    e.bias, e.act_kind = bias.data_ptr(), 1
    e.act.p, e.act.M_pad, e.act.ld, e.act.fmt = act.data_ptr(), m_pad, ka, 0
    NN.check(NN.lib().saber_linear_launch(C.byref(p), NN.stream_handle()), "linear")
    torch.cuda.synchronize()
    sc.check()
    want = (a.double() @ w.double().T) / torch.sqrt(ss[:M].cpu().double().sum(1) * 0.25 + 1e-3)[:, None]
    ref = want[:, :plain] + bias[:plain].cpu().double()
    assert (out[:, :plain].cpu().double() - ref).abs().max() < 2e-5 * ref.abs().max() and torch.all(out[:, plain:] == 7.0)
    got, dev = torch.zeros(M, ka, dtype=BF16), act.cpu()
    for kb in range(ka // 64):
        got[:, kb * 64:(kb + 1) * 64] = dev[kb, rows, chunk ^ (rows & 7)].reshape(M, 64)
    sq = torch.relu(want[:, plain:]) ** 2
    assert (got[:, :ff].double() - sq).abs().max() < 0.01 * sq.abs().max() and torch.all(got[:, ff:] == 0)


@pytest.mark.parametrize("H,HK,N,V,lens", [(4, 2, 24, 40, (200,)), (3, 3, 128, 100, (64, 1, 130)), (2, 1, 200, 24, (63, 65)), (2, 2, 250, 64, (150,))])
def test_chunk_form_keeps_fp32_digits(H, HK, N, V, lens):
    """q, k, v in bf16 and everything else in fp32: against float64 on the rounded inputs, the chunk form is as close as
    fp32 sums are, with decays from none to total inside one chunk, and carries the state over."""
    from saber_engine_b200.models.stack_config import OuterMixer
    from saber_engine_b200.ops import functional as F
    from saber_engine_b200.ops import native as NN
    g = torch.Generator().manual_seed(H + N)
    mix = OuterMixer(H, HK, N, V)
    DP, VP, M, nseq = mix.dim_pad, mix.vdim_pad, sum(lens), len(lens)
    cols, off = 0, {}
    for name, n in mix.segments():
        off[name] = cols
        cols = (cols + n + 7) // 8 * 8
    x = torch.randn(M, cols, generator=g)
    end = off["v"] + H * V                                       # inputs whose silu is a bf16 number: no doubt about its rounding
    y = O.silu(x[:, :end].double().clamp(min=-1.0)).bfloat16().double()
    z = x[:, :end].double().clamp(min=-1.0)
    for _ in range(30):
        sg = torch.sigmoid(z)
        z = z - (z * sg - y) / (sg * (1 + z * (1 - sg)))
    x[:, :end] = z.float()
    x[:, off["dt"]:off["dt"] + H] = torch.randn(M, H, generator=g) * 4
    A_log, dt_bias, skip = torch.randn(H, generator=g) * 2, torch.randn(H, generator=g), torch.randn(H, generator=g)
    S0 = torch.randn(nseq, H, V, N, generator=g)
    state = torch.zeros(nseq + 1, H, VP, DP)
    state[1:, :, :V, :N] = S0
    dev = {k: v.float().cuda() for k, v in dict(x=x, A=A_log, b=dt_bias, d=skip, st=state, nw=torch.ones(H * V)).items()}
    cu = torch.tensor([0] + [sum(lens[:i + 1]) for i in range(nseq)], dtype=torch.int32).cuda()
    slots = torch.arange(1, nseq + 1, dtype=torch.int32).cuda()
    pos = torch.cat([torch.arange(n) for n in lens]).int().cuda()
    o, out = torch.zeros(M, H, VP, device="cuda"), torch.zeros(M, H * V, device="cuda")
    p = NN.SsdParams()
    p.x, p.ldx, p.q_off, p.k_off, p.v_off, p.dt_off, p.g_off = dev["x"].data_ptr(), cols, off["q"], off["k"], off["v"], off["dt"], off["g"]
    p.A_log, p.dt_bias, p.skip, p.norm_w, p.state, p.o = (t.data_ptr() for t in (dev["A"], dev["b"], dev["d"], dev["nw"], dev["st"], o))
    p.cu_rows, p.slots, p.pos, p.M, p.nseq = cu.data_ptr(), slots.data_ptr(), pos.data_ptr(), M, nseq
    p.out.p, p.out.M_pad, p.out.ld, p.out.fmt = out.data_ptr(), M, H * V, 1
    p.H, p.HK, p.N, p.DP, p.V, p.VP, p.taps, p.groups, p.n_slots, p.eps = H, HK, N, DP, V, VP, 0, 1, nseq + 1, 1e-5
    sc = F.scratch("cuda")
    p.err = sc.err.data_ptr()
    chunk = torch.zeros(NN.lib().saber_ssd_chunk_floats(C.byref(p)), device="cuda")
    p.chunk = chunk.data_ptr()
    NN.check(NN.lib().saber_ssd_launch(C.byref(p), 0, NN.stream_handle()), "ssd")
    torch.cuda.synchronize()
    sc.check()
    xd = x.double()
    act = lambda n, h, d: O.silu(x[:, off[n]:off[n] + h * d]).bfloat16().double().view(M, h, d)      # noqa: E731
    q, k, v = (a[:, torch.arange(H) // (H // a.shape[1])] for a in (act("q", HK, N), act("k", HK, N), act("v", H, V)))
    dt = O.softplus(xd[:, off["dt"]:off["dt"] + H] + dt_bias.double())
    a = torch.exp(-torch.exp(A_log.double()) * dt)
    for s, n in enumerate(lens):
        r0, S = int(cu[s]), S0[s].double()
        want = torch.zeros(n, H, V).double()
        for t in range(n):
            S = a[r0 + t][:, None, None] * S + (dt[r0 + t][:, None] * v[r0 + t])[:, :, None] * k[r0 + t][:, None, :]
            want[t] = torch.einsum("hvn,hn->hv", S, q[r0 + t]) + skip.double()[:, None] * v[r0 + t]
        got = o[r0: r0 + n, :, :V].cpu().double()
        assert (got - want).abs().max() < 2e-6 * want.abs().max(), s
        back = dev["st"][s + 1, :, :V, :N].cpu().double()
        assert (back - S).abs().max() < 2e-6 * S.abs().max(), s


def test_scan_serves_sizes_the_chunk_form_does_not():
    cfg = R.config([R.mamba(heads=2, groups=1, state=300, ff=None)])
    t = R.tensors(cfg, 4)
    toks = R.tokens(cfg, 130)
    eng = R.engine(cfg, t, BF16)
    assert eng.model._chunk_floats(eng.model.cfg.layers[0].mixer, 256, 4) == 0
    want = O.Oracle(cfg, t).forward(toks)
    for cuts in ([130], [70, 1]):
        assert R.error(R.feed(eng, "r", toks, cuts), want) < R.TOL[BF16]


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
def test_unequal_batch_against_each_alone_with_slots_used_again(case, dtype):
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
    cfg = R.config([R.attention(heads=12, kv_heads=3, dim=72, vdim=100, chunk=150, ff=None),
                    R.attention(heads=3, kv_heads=3, dim=72, vdim=100, chunk=1000, kv_from=0, ff=None)], width=264)
    t = R.tensors(cfg, seed=9)
    toks = R.tokens(cfg, 333)
    want = O.Oracle(cfg, t).forward(toks)
    for impl, form in (("tc", 2), ("mma", 1)):
        eng = R.engine(cfg, t, BF16, attn_impl=impl)
        assert eng.model._gqa_form(eng.model.cfg.layers[0].mixer, 256, False) == form
        assert R.error(R.feed(eng, "r", toks, [333]), want) < R.TOL[BF16]
        assert R.error(R.feed(eng, "r", toks, [70, 130, 2]), want) < R.TOL[BF16]
    many = R.CASES["many_query_heads"]                           # more heads on a key head than a tile holds: the row form
    eng = R.engine(many, R.tensors(many), BF16)
    assert [eng.model._gqa_form(l.mixer, 256, False) for l in eng.model.cfg.layers[:2]] == [2, 0]


# ------------------------------------------------------------------------------ far keys, borders, long runs
def _needle(cfg: dict, seed: int):
    """Weights with a needle: the query of the last token id meets the key of token id 1 with a score far above all
    others, wherever that token stands."""
    t = R.tensors(cfg, seed)
    W, m = cfg["width"], cfg["layers"][0]["mixer"]
    t["embed"][:, :2] = 0.0
    t["embed"][1, 0] = 9.0                                       # only the needle has this coordinate
    t["embed"][cfg["vocab"] - 1, 1] = 9.0
    t["l0.norm1"][:] = 0.0
    for n, heads, coord in (("q", m["heads"], 1), ("k", m["kv_heads"], 0)):
        t[f"l0.mix.{n}.b"][:] = 0.0
        w = t[f"l0.mix.{n}"].view(heads, m["dim"], W)
        w[:, :, coord] = 0.0
        w[:, 0, :] = 0.0
        w[:, 0, coord] = 8.0                                     # head coordinate 0, far above the rest of the vector
    return t


@pytest.mark.parametrize("dtype", [F32, BF16])
@pytest.mark.parametrize("chunk,place", [(1000, 0), (1000, 1), (1000, 63), (1000, 64), (1000, 127), (1000, 128), (1000, 500), (300, 300), (300, 299),
                                         (300, 383), (300, 384), (64, 512), (64, 511), (128, 512), (128, 511), (17, 510), (17, 509), (519, 519), (520, 0),
                                         (40, 480), (40, 518)])
def test_one_key_at_chunk_and_page_edges(dtype, chunk, place):
    cfg = R.config([R.attention(heads=6, kv_heads=2, dim=24, vdim=20, chunk=chunk, scale=0.9, softcap=30.0, ff=None)], vocab=131)
    t = _needle(cfg, 2)
    n = 520
    toks = [2 + x % 120 for x in R.tokens(cfg, n)]
    toks[place] = 1
    if place != n - 1:
        toks[-1] = cfg["vocab"] - 1
    orc = O.Oracle(cfg, t)
    want = orc.forward(toks)
    without = list(toks)
    without[place] = 2
    gap = R.error(orc.forward(without)[-1:], want[-1:])
    inside = place >= (n - 1) - (n - 1) % chunk
    assert gap > 0.3 if inside else gap < 1e-9                   # the answer hangs on that one key, or not at all
    tol = {F32: 5e-5, BF16: 0.08}[dtype]
    for kw in ({}, {"attn_impl": "mma"}):
        eng = R.engine(cfg, t, dtype, rungs=(64, 256, 1024), **kw)
        assert R.error(R.feed(eng, "r", toks, [n])[-1:], want[-1:]) < tol               # asked in the prompt
        assert R.error(R.feed(eng, "r", toks, [n - 1, 1])[-1:], want[-1:]) < tol        # asked by a decoded token
        assert R.error(R.feed(eng, "r", toks, [n - 2, 2])[-1:], want[-1:]) < tol        # in a portion of two
        assert R.error(R.feed(eng, "r", toks, [max(1, place), 1, 2, 200, 255, 1])[-1:], want[-1:]) < tol


@pytest.mark.parametrize("dtype", [F32, BF16])
def test_every_row_around_chunk_edges(dtype):
    """Needles all over the prompt: each asking token sees those of its own chunk only."""
    cfg = R.config([R.attention(heads=4, kv_heads=2, dim=24, vdim=20, chunk=90, scale=0.9, softcap=30.0, ff=None)], vocab=131)
    t = _needle(cfg, 3)
    toks = [2 + x % 120 for x in R.tokens(cfg, 400)]
    for i in range(5, 400, 9):
        toks[i] = 1 if i % 4 else 130
    want = O.Oracle(cfg, t).forward(toks)
    for cuts in ([400], [89, 1, 1, 88, 2, 90, 1], [399, 1], [1]):
        eng = R.engine(cfg, t, dtype)
        assert R.error(R.feed(eng, "r", toks, cuts), want) < {F32: 5e-5, BF16: 0.1}[dtype], cuts


@pytest.mark.parametrize("scale,softcap", [(0.05, 1.0), (2.0, 50.0), (2.0, 3.0), (0.3, 1e4)])
@pytest.mark.parametrize("lens", [(300,), (129, 64, 1, 257)])
def test_capped_scores_over_unequal_prompts(lens, scale, softcap):
    cfg = R.config([R.attention(heads=6, kv_heads=3, dim=48, vdim=56, scale=scale, softcap=softcap, chunk=111, ff=None)], vocab=800)
    t = R.tensors(cfg, 5)
    toks = [sorted(R.tokens(cfg, n, seed=i)) for i, n in enumerate(lens)]
    orc = O.Oracle(cfg, t)
    for dtype, tol in ((BF16, 0.06 * max(1.0, 2 * scale)), (F32, 5e-5)):
        eng = R.engine(cfg, t, dtype, rungs=(1024,))
        got = eng.step([(i, x) for i, x in enumerate(toks)])
        for g, x in zip(got, toks):
            assert R.error(g, orc.forward(x)) < tol


@pytest.mark.parametrize("kind", ["lightning", "mamba"])
def test_state_carries_far_and_a_lost_state_shows(kind):
    """Slow decay: the first tokens' writes are still read hundreds of tokens later, over every cut."""
    layer = R.lightning(ff=None, decay=(0.9999, 0.999, 1.0)) if kind == "lightning" else R.mamba(ff=None)
    cfg = R.config([layer])
    t = R.tensors(cfg, 6)
    if kind == "mamba":
        t["l0.mix.A_log"][:] = -7.0
    toks = R.tokens(cfg, 300)
    orc = O.Oracle(cfg, t)
    want = orc.forward(toks)
    assert R.error(orc.forward(R.tokens(cfg, 20, 9) + toks[20:])[-1:], want[-1:]) > 0.005
    for dtype in (F32, BF16):
        eng = R.engine(cfg, t, dtype)
        for cuts in ([300], [255, 2, 43], [4, 3, 5, 1, 2, 6, 200, 1], [64, 64, 65, 63]):
            assert R.error(R.feed(eng, "r", toks, cuts), want) < {F32: 3e-5, BF16: 0.02}[dtype], (dtype, cuts)


def test_strong_and_unequal_decays():
    """Steps and rates that forget everything within a token beside ones that forget nothing."""
    cfg = R.config([R.mamba(heads=6, groups=2, ff=None), R.lightning(ff=None, decay=(0.0, 1e-4, 1.0))])
    t = R.tensors(cfg, 7)
    t["l0.mix.A_log"][:] = torch.tensor([4.0, -8.0, 3.0, 0.0, 5.0, -2.0]).bfloat16()
    t["l0.mix.dt_bias"][:] = torch.tensor([3.0, 1.0, -3.0, 2.0, 4.0, -6.0]).bfloat16()
    toks = R.tokens(cfg, 200)
    want = O.Oracle(cfg, t).forward(toks)
    for dtype in (F32, BF16):
        eng = R.engine(cfg, t, dtype)
        for cuts in ([200], [190, 1], [7, 70, 2]):
            assert R.error(R.feed(eng, "r", toks, cuts), want) < R.TOL[dtype]


@pytest.mark.parametrize("n", [1, 2, 3, 4, 5, 6])
def test_first_tokens(n):
    cfg = R.config([R.mamba(conv=4), R.attention(chunk=3), R.mamba(conv=5, ff=None), R.lightning(), R.attention(chunk=2, kv_from=1)])
    t = R.tensors(cfg, 8)
    toks = R.tokens(cfg, n)
    want = O.Oracle(cfg, t).forward(toks)
    for dtype in (F32, BF16):
        eng = R.engine(cfg, t, dtype)
        for cuts in ([n], [1], [2]):
            assert R.error(R.feed(eng, "r", toks, cuts), want) < R.TOL[dtype]


def test_long_decoding_over_page_and_chunk_borders():
    cfg = R.CASES["every_kind"]
    t = R.tensors(cfg, 10)
    toks = R.tokens(cfg, 330)
    want = O.Oracle(cfg, t).forward(toks)
    for dtype in (F32, BF16):
        eng = R.engine(cfg, t, dtype, capture=True)
        assert R.error(R.feed(eng, "r", toks, [10, 1]), want) < R.TOL[dtype]


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
    cfg = R.CASES["two_readers"]
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
    cfg = R.CASES["equal_heads"]
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
