"""Fitatar on the GPU against the plain restatement in oracle_fitatar.py."""
import ctypes as C
import json
import os
import subprocess
import sys

import pytest
import torch

import fitatar_cases as R
import oracle_fitatar as O
from saber_engine_b200.sched.scheduler import Scheduler, SchedulerConfig
from saber_engine_b200.serve.engine_api import EngineRequest, SamplingParams

pytestmark = pytest.mark.gpu
F32, BF16 = torch.float32, torch.bfloat16
REPO = os.path.dirname(os.path.dirname(os.path.abspath(__file__)))


# ------------------------------------------------------------------------------ mechanisms, one or two layers each
ALONE = {
    "attention": [R.attention()],
    "attention_whole_head_turns": [R.attention(heads=4, kv_heads=4, dim=40, vdim=8, rot=40, factor=1.0)],
    "attention_odd_pairs": [R.attention(heads=4, kv_heads=2, dim=20, vdim=12, rot=6)],
    "attention_one_pair": [R.attention(heads=2, kv_heads=1, dim=8, vdim=48, rot=2, base=50.0)],
    "attention_wide": [R.attention(heads=2, kv_heads=1, dim=272, vdim=200, rot=264)],
    "latent": [R.latent()],
    "latent_small_query_rank": [R.latent(heads=5, q_rank=8, kv_rank=24, vdim=72)],
    "latent_large_query_rank": [R.latent(heads=2, dim=64, rot_dim=64, vdim=64, q_rank=520, kv_rank=72, yarn=(8.0, 32, 16.0, 1.0))],
    "latent_of_another_layer": [R.latent(), R.latent(heads=7, dim=40, vdim=24, q_rank=24, scale=0.4, kv_from=0)],
    "dense": [R.attention(mlp=R.dense(130))],
    "narrow_dense": [R.latent(mlp=R.dense(33))],
    "experts": [R.attention(mlp=R.moe())],
    "experts_without_groups": [R.latent(mlp=R.moe(groups=1, keep=1, experts=10, top=4, ff=24))],
    "experts_without_shared": [R.attention(mlp=R.moe(shared=0, ff=136))],
    "one_of_many_experts": [R.attention(mlp=R.moe(experts=72, groups=9, keep=1, top=1, shared=248))],
    "odd_width": [R.attention(mlp=R.dense(50)), R.latent(mlp=R.moe(ff=12, shared=20))],
    "groups_of_one": [R.attention(mlp=R.moe(experts=7, groups=7, keep=4, top=4, shared=249))],
}


@pytest.mark.parametrize("name", ALONE)
@pytest.mark.parametrize("dtype", [F32, BF16])
def test_mechanism_alone_residual_stream(name, dtype):
    cfg = R.config(ALONE[name], **({"width": 91} if name == "odd_width" else {}))
    t = R.tensors(cfg, seed=3)
    toks = R.tokens(cfg, 140)
    trace = []
    O.Oracle(cfg, t).forward(toks, trace)
    tol = (2e-5 if dtype == F32 else 0.03) * float(trace[-1].abs().max())
    eng = R.engine(cfg, t, dtype, rungs=(160,))
    eng.step([("a", toks)])
    b = next(iter(eng.model.buckets.values()))
    assert float((b.x[:140, : cfg["width"]].cpu().double() - trace[-1]).abs().max()) < tol
    for tok in toks[:70]:
        eng.step([("b", [tok])])
    x = eng.model.buckets[("decode", 1, 1)].x[:1, : cfg["width"]].cpu().double()
    assert float((x - trace[-1][69:70]).abs().max()) < tol


def _operand(a, m_pad):
    """Rows [M, K] (K a multiple of 64) in the GEMM's tile order."""
    M, K = a.shape
    op = torch.zeros(K // 64, m_pad, 8, 8, dtype=BF16)
    rows, chunk = torch.arange(M)[:, None], torch.arange(8)[None, :]
    for kb in range(K // 64):
        op[kb, rows, chunk ^ (rows & 7)] = a[:, kb * 64:(kb + 1) * 64].reshape(M, 8, 8)
    return op.cuda()


def _rows(op, M):
    op = op.cpu()
    rows, chunk = torch.arange(M)[:, None], torch.arange(8)[None, :]
    return torch.cat([op[kb, rows, chunk ^ (rows & 7)].reshape(M, 64) for kb in range(op.shape[0])], 1)


def _near(got, want, rel):
    assert float((got.double() - want).abs().max()) < rel * float(want.abs().max())


@pytest.mark.parametrize("fuse", [True, False])
@pytest.mark.parametrize("M,K,lat,plain,ff,splits", [(3, 64, 40, 24, 30, 1), (17, 640, 300, 500, 250, 5), (130, 128, 256, 300, 600, 1), (300, 192, 24, 40, 248, 1)])
@pytest.mark.parametrize("kind", [2, 3])
def test_project_linear_parts(M, K, lat, plain, ff, splits, fuse, kind):
    """One product: a latent as the next operand, stored columns, and behind the second operand stored columns and activations
    (squared ReLU times the sigmoid of its tile's gate row; gelu with a bias)."""
    from saber_engine_b200.models import stack_weights as SW
    from saber_engine_b200.ops import functional as F
    from saber_engine_b200.ops import layouts as L
    from saber_engine_b200.ops import native as NN
    g = torch.Generator().manual_seed(M + K)
    rnd = lambda *s: torch.randn(*s, generator=g)      # noqa: E731
    lt, p0 = (lat + 255) // 256, (lat + 255) // 256 * 256
    tile2 = (p0 + plain + 255) // 256
    tile0, per = tile2 + 1, 248 if kind == 2 else 256
    n = tile0 + (ff + per - 1) // per
    w = torch.zeros(n, 256, K)
    flat = w.view(-1, K)
    flat[:lat], flat[p0:p0 + plain] = rnd(lat, K) / K ** 0.5, rnd(plain, K) / K ** 0.5
    flat[tile2 * 256: tile2 * 256 + 20] = rnd(20, K) / K ** 0.5
    up, gate = (rnd(ff, K) / K ** 0.5).bfloat16(), (rnd(1, K) / K ** 0.5).bfloat16()
    full = torch.zeros((n - tile0) * per, K)
    full[:ff] = up.float()
    w[tile0:, :per] = full.view(-1, per, K)
    if kind == 2:
        w[tile0:, 248] = gate.float()
    wb = flat.bfloat16()
    a, a2 = rnd(M, K).bfloat16(), rnd(M, K).bfloat16()
    lin, m_pad = SW.pack_linear(wb.cuda(), BF16), L.padded_rows(M)
    op, op2 = _operand(a, m_pad), _operand(a2, m_pad)
    sc = F.scratch("cuda")
    ss = (torch.rand(m_pad, 2, generator=g) + 0.5).cuda()
    n_plain = tile2 * 256 + 24
    bias, lat_w, act_bias = rnd(n_plain).cuda(), rnd(lat).cuda(), rnd((n - tile0) * 256).cuda()
    act_bias[ff:] = 0
    out = torch.full((M, n_plain + 8), 7.0, dtype=F32, device="cuda")
    lat_op = torch.full((L.round_up(lat, 64) // 64, m_pad, 8, 8), 5.0, dtype=BF16, device="cuda")
    lat_ss = torch.full((m_pad, 2 * lt), -1.0, dtype=F32, device="cuda")
    ka = 64 + L.round_up(ff, 64)
    act = torch.full((ka // 64, m_pad, 8, 8), 5.0, dtype=BF16, device="cuda")
    ws = torch.zeros(M * n * 256 + (1 << 22), dtype=F32, device="cuda")
    p = NN.LinParams()
    p.w, p.a, p.err, p.ws, p.counters = lin.w.data_ptr(), op.data_ptr(), sc.err.data_ptr(), ws.data_ptr(), sc.counters.data_ptr()
    p.M, p.M_pad, p.N_pad, p.K, p.nt, p.splits, p.fuse = M, m_pad, n * 256, K, L.token_tile(M), splits, int(fuse)
    p.a2, p.a2_tile0, p.mtiles = op2.data_ptr(), tile2, 2 if m_pad % 256 == 0 else 1
    e = p.e
    e.ss, e.ss_n, e.inv_width, e.eps, e.out, e.ldo, e.n_plain, e.act_tile0 = ss.data_ptr(), 2, 0.25, 1e-3, out.data_ptr(), out.stride(0), n_plain, tile0
    e.bias, e.act_kind, e.act_bias, e.cap = bias.data_ptr(), kind, act_bias.data_ptr() if kind == 3 else None, 1.5
    e.lat_tiles, e.lat_n, e.lat, e.lat_w, e.lat_ss, e.lat_ss_n = lt, lat, NN.Operand(lat_op.data_ptr(), m_pad, L.round_up(lat, 64), 0), lat_w.data_ptr(), lat_ss.data_ptr(), 2 * lt
    e.act, e.act_k0 = NN.Operand(act.data_ptr(), m_pad, ka, 0), 64
    NN.check(NN.lib().saber_linear_launch(C.byref(p), NN.stream_handle()), "linear")
    torch.cuda.synchronize()
    sc.check()
    r = 1 / torch.sqrt(ss[:M].cpu().double().sum(1) * 0.25 + 1e-3)[:, None]
    y1, y2 = a.double() @ wb.double().T * r, a2.double() @ wb.double().T * r
    _near(_rows(lat_op, M)[:, :lat], y1[:, :lat] * lat_w.cpu().double(), 0.01)
    assert torch.all(_rows(lat_op, M)[:, lat:] == 0) or not fuse
    _near(lat_ss[:M].sum(1).cpu(), (y1[:, :lat] ** 2).sum(1), 1e-5)
    cap = lambda z: 1.5 * torch.tanh(z / 1.5)          # noqa: E731
    _near(out[:, p0:p0 + plain].cpu(), cap(y1[:, p0:p0 + plain] + bias[p0:p0 + plain].cpu().double()), 2e-5)
    _near(out[:, tile2 * 256: n_plain].cpu(), cap(y2[:, tile2 * 256: n_plain] + bias[tile2 * 256:].cpu().double()), 2e-5)
    assert torch.all(out[:, n_plain:] == 7.0)
    z = a2.double() @ up.double().T * r
    want = torch.relu(z) ** 2 * torch.sigmoid(a2.double() @ gate.double().T * r) if kind == 2 else O.gelu(z + act_bias[:ff].cpu().double())
    got = _rows(act, M)
    _near(got[:, 64: 64 + ff], want, 0.01)
    assert torch.all(got[:, :64] == 5.0) and torch.all(got[:, 64 + ff: 64 + (n - tile0) * per] == 0)      # (columns past the tiles meet zero weights)


def _route(z, top, groups, keep, nt, live):
    """Device routing tables of fp32 logits z [M, E]."""
    from saber_engine_b200.ops import native as NN
    M, E = z.shape
    zd = torch.zeros(M, E + 5, device="cuda")
    zd[:, :E] = z
    i32 = lambda *s: torch.full(s, -7, dtype=torch.int32, device="cuda")     # noqa: E731
    cap = (M * top + 15 * min(E, M * top) + 15) // 16 * 16 + 128
    d = dict(topk_id=i32(M, top), slot_of=i32(M, top), counts=i32(E).zero_(), offsets=i32(E + 1), cursors=i32(E), ntiles=i32(2),
             tiles=i32(min(E, M * top) + M * top // nt, 4), src_row=i32(cap), topk_w=torch.zeros(M, top, device="cuda"))
    lv = torch.tensor([live], dtype=torch.int32, device="cuda")
    p = NN.MoeRouteParams()
    p.logits_f32, p.ld, p.M, p.E, p.top_k, p.nt, p.rows_cap, p.e_n, p.live, p.groups, p.keep = zd.data_ptr(), E + 5, M, E, top, nt, cap, E, lv.data_ptr(), groups, keep
    for k, v in d.items():
        setattr(p, k, v.data_ptr())
    NN.check(NN.lib().saber_moe_route_launch(C.byref(p), NN.stream_handle()), "route")
    torch.cuda.synchronize()
    return {k: v.cpu() for k, v in d.items()}


@pytest.mark.parametrize("M,live", [(1, 1), (7, 5), (64, 64), (65, 60), (300, 300)])
@pytest.mark.parametrize("E,top,groups,keep", [(16, 4, 4, 3), (6, 6, 3, 3), (5, 1, 5, 1), (33, 5, 11, 2), (160, 8, 8, 3), (40, 3, 1, 1), (600, 32, 20, 5)])
def test_routing(M, live, E, top, groups, keep):
    """Choices and weights are the oracle's; every live route has a row of its own in its expert's tiles."""
    z = torch.randn(M, E, generator=torch.Generator().manual_seed(M * E)) * 2
    nt = 16 if M <= 64 else 64
    d = _route(z, top, groups, keep, nt, live)
    s = torch.softmax(z.double(), -1)
    for m in range(M):
        ids = d["topk_id"][m].tolist()
        if m >= live:
            assert ids == [-1] * top and d["slot_of"][m].tolist() == [-1] * top
            continue
        assert ids == O.route(s[m].tolist(), top, {"count": groups, "keep": keep})
        assert torch.allclose(d["topk_w"][m].double(), s[m][ids], rtol=2e-6, atol=1e-12)
    slots = d["slot_of"][:live].flatten()
    assert len(set(slots.tolist())) == live * top
    expert_of = {}
    for e, first, n, _ in d["tiles"][: int(d["ntiles"][0])].tolist():
        assert first % 16 == 0 and 0 < n <= nt
        expert_of.update({r: e for r in range(first, first + n)})
    assert len(expert_of) == live * top
    for m in range(live):
        for k in range(top):
            r = int(d["slot_of"][m, k])
            assert expert_of[r] == int(d["topk_id"][m, k]) and int(d["src_row"][r]) == m
    assert int((d["src_row"] >= 0).sum()) == live * top


def test_equal_scores_take_the_lower_expert():
    z = torch.zeros(3, 12)
    d = _route(z, 4, 3, 2, 16, 3)
    assert d["topk_id"].tolist() == [[0, 1, 2, 3]] * 3
    z[1, 9] = z[1, 4] = 1.0
    assert _route(z, 3, 3, 1, 16, 3)["topk_id"][1].tolist() == [4, 5, 6]


@pytest.mark.parametrize("dtype", [F32, BF16])
@pytest.mark.parametrize("spread", ["one_expert", "all"])
def test_expert_rows_fill_and_overflow_tiles(dtype, spread):
    """All tokens on one expert (many tiles of it), or one token for each."""
    cfg = R.config([R.attention(mlp=R.moe(experts=16, top=1, groups=1, keep=1, ff=24, shared=0))], vocab=64)
    t = R.tensors(cfg, 5)
    t["l0.mlp.router"][:] = 0
    if spread == "one_expert":
        t["l0.mlp.router"][11, 0], t["embed"][:, 0], t["l0.norm2"][0] = 8.0, 2.0, 1.0
    else:
        t["embed"][:, :16], t["l0.norm2"][:16] = 0, 1.0
        t["embed"][torch.arange(64), torch.arange(64) % 16] = 2.0
        t["l0.mlp.router"][torch.arange(16), torch.arange(16)] = 8.0
        for n in ("mix.o", "mlp.e0.down"):
            t["l0." + n][:16] = 0
    for n in (300, 16, 1):
        toks = [x % 64 for x in range(n)]
        want = O.Oracle(cfg, t).forward(toks)
        eng = R.engine(cfg, t, dtype)
        for cuts in ([n], [max(1, n - 3), 1]):
            assert R.error(R.feed(eng, "r", toks, cuts), want) < R.TOL[dtype]


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
def test_unequal_batch_against_each_alone_with_pages_used_again(case, dtype):
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
    cfg = R.config([R.attention(heads=12, kv_heads=3, dim=72, vdim=100, rot=40), R.latent(heads=6, dim=72, rot_dim=24, vdim=100, kv_rank=130, q_rank=72),
                    R.latent(heads=3, dim=40, rot_dim=24, vdim=128, kv_rank=130, q_rank=80, kv_from=1)], width=264)
    t = R.tensors(cfg, seed=9)
    toks = R.tokens(cfg, 333)
    want = O.Oracle(cfg, t).forward(toks)
    for impl, form in (("tc", 2), ("mma", 1)):
        eng = R.engine(cfg, t, BF16, attn_impl=impl)
        ms = [l.mixer for l in eng.model.cfg.layers]
        assert (eng.model._gqa_form(ms[0], 256, False), eng.model._expanded(ms[1], 256, False)) == (form, form)
        for cuts in ([333], [70, 130, 2]):
            assert R.error(R.feed(eng, "r", toks, cuts), want) < R.TOL[BF16]
    eng = R.engine(cfg, t, BF16, expand_bytes=0)                 # no room for expanded keys: the latent space serves prompts
    assert R.error(R.feed(eng, "r", toks, [333]), want) < R.TOL[BF16]


# ------------------------------------------------------------------------------ far keys, borders, sinks, rotations, long runs
def _needle(cfg: dict, seed: int, turning: bool = False):
    """Weights with a needle: the query of the last token id meets the key of token id 1 with a score far above all others, wherever that token
    stands (turning: in a rotated pair, where the score falls with the distance)."""
    t = R.tensors(cfg, seed)
    W, kind, m = cfg["width"], cfg["layers"][0]["type"], cfg["layers"][0]["mixer"]
    t["embed"][:, :2] = 0.0
    t["embed"][1, 0] = 9.0                                       # only the needle has this coordinate
    t["embed"][cfg["vocab"] - 1, 1] = 9.0
    t["l0.norm1"][:2] = 1.0
    if kind == "attention":
        for n, heads, coord in (("q", m["heads"], 1), ("k", m["kv_heads"], 0)):
            w = t[f"l0.mix.{n}"].view(heads, m["dim"], W)
            w[:, :, coord] = 0.0
            w[:, 0 if turning else m["dim"] - 1, coord] = 2.0
        t["l0.mix.sink"][:] = 0.5
        return t
    t["l0.mix.dq"][0], t["l0.mix.dkv"][0] = 0.0, 0.0
    t["l0.mix.dq"][0, 1], t["l0.mix.dkv"][0, 0] = 6.0, 6.0       # the latents' first value, then the head's first
    t["l0.mix.dq.norm"][0] = t["l0.mix.dkv.norm"][0] = 1.0
    uq, uk = t["l0.mix.uq"].view(m["heads"], -1, m["q_rank"]), t["l0.mix.uk"].view(m["heads"], -1, m["kv_rank"])
    uq[:, 0], uk[:, 0] = 0.0, 0.0
    uq[:, 0, 0], uk[:, 0, 0] = 3.0, 3.0
    return t


PLACES = [0, 1, 63, 64, 127, 128, 255, 256, 500, 512, 517, 518]


@pytest.mark.parametrize("dtype", [F32, BF16])
@pytest.mark.parametrize("kind", ["attention", "latent"])
def test_one_key_far_back_and_at_page_edges(dtype, kind):
    layer = R.attention(heads=6, kv_heads=2, dim=24, vdim=20, rot=8, scale=0.9) if kind == "attention" else R.latent(heads=4, scale=0.9)
    cfg = R.config([layer], vocab=131)
    t = _needle(cfg, 2)
    n = 520
    orc = O.Oracle(cfg, t)
    tol = {F32: 5e-5, BF16: 0.08}[dtype]
    engs = [R.engine(cfg, t, dtype, rungs=(64, 256, 1024), **kw) for kw in ({}, {"attn_impl": "mma"})]
    for place in PLACES:
        toks = [2 + x % 120 for x in R.tokens(cfg, n)]
        toks[place], toks[-1] = 1, cfg["vocab"] - 1
        want = orc.forward(toks)
        without = list(toks)
        without[place] = 2
        assert R.error(orc.forward(without)[-1:], want[-1:]) > 0.2               # the answer hangs on that one key
        for eng in engs:
            for cuts in ([n], [n - 1, 1], [n - 2, 2], [max(1, place), 1, 2, 200, 255, 1]):
                assert R.error(R.feed(eng, "r", toks, cuts)[-1:], want[-1:]) < tol, (place, cuts)


@pytest.mark.parametrize("dtype", [F32, BF16])
def test_later_keys_are_not_seen(dtype):
    """Needles all over the prompt: each asking token sees those before it only."""
    for layer in (R.attention(heads=4, kv_heads=2, dim=24, vdim=20, rot=8, scale=0.9), R.latent(heads=4, scale=0.9)):
        cfg = R.config([layer], vocab=131)
        t = _needle(cfg, 3)
        toks = [2 + x % 120 for x in R.tokens(cfg, 200)]
        for i in range(5, 200, 9):
            toks[i] = 1 if i % 4 else 130
        want = O.Oracle(cfg, t).forward(toks)
        for cuts in ([200], [63, 1, 1, 63, 2, 50, 1], [199, 1], [1]):
            eng = R.engine(cfg, t, dtype)
            assert R.error(R.feed(eng, "r", toks, cuts), want) < {F32: 5e-5, BF16: 0.1}[dtype], cuts


@pytest.mark.parametrize("sink", [-80.0, 0.0, 4.0, 9.0, 100.0])
def test_sink_of_any_size(sink):
    """From none to one that takes everything; heads differ."""
    cfg = R.config([R.attention(heads=6, kv_heads=3, dim=40, vdim=24, scale=0.6)])
    t = R.tensors(cfg, 4)
    t["l0.mix.sink"][:] = torch.tensor([sink, 0.0, sink, -1.0, sink, 2.0]).bfloat16()
    toks = R.tokens(cfg, 140)
    want = O.Oracle(cfg, t).forward(toks)
    plain = {k: v.clone() for k, v in t.items()}
    plain["l0.mix.sink"][:] = -1000.0
    assert R.error(O.Oracle(cfg, plain).forward(toks), want) > 0.02
    for dtype in (F32, BF16):
        for kw in ({}, {"attn_impl": "mma"}):
            eng = R.engine(cfg, t, dtype, **kw)
            for cuts in ([140], [1], [65, 2, 70, 1]):
                assert R.error(R.feed(eng, "r", toks, cuts), want) < R.TOL[dtype]


@pytest.mark.parametrize("layer", [R.attention(heads=2, kv_heads=1, dim=64, vdim=24, rot=48, base=20.0, factor=1.0, scale=0.8),
                                   R.attention(heads=2, kv_heads=1, dim=64, vdim=24, rot=64, base=5000.0, factor=16.0, scale=0.8),
                                   R.latent(heads=2, dim=8, rot_dim=64, base=2000.0, yarn=(16.0, 128, 8.0, 0.5), scale=0.5),
                                   R.latent(heads=2, dim=8, rot_dim=32, base=50.0, yarn=(4.0, 1e5, 4.0, 2.0), scale=0.5),
                                   R.latent(heads=2, dim=8, rot_dim=48, base=1e6, yarn=(4.0, 16, 64.0, 30.0), scale=0.5)])
def test_rotations(layer):
    """Slow and fast pairs, all or some of them scaled; every part of the rotation shows in the oracle."""
    cfg = R.config([layer])
    t = R.tensors(cfg, 6)
    toks = R.tokens(cfg, 300)
    want = O.Oracle(cfg, t).forward(toks)
    for change in ({"base": layer["mixer"]["rot"]["base"] * 1.5}, {"scaling": None}):
        other = json.loads(json.dumps(cfg))
        rot = other["layers"][0]["mixer"]["rot"]
        if change == {"scaling": None} and rot["scaling"] == {"factor": 1.0}:
            continue
        rot.update(change)
        assert R.error(O.Oracle(other, t).forward(toks), want) > 0.01
    for dtype in (F32, BF16):
        eng = R.engine(cfg, t, dtype)
        for cuts in ([300], [255, 2, 43], [64, 1]):
            assert R.error(R.feed(eng, "r", toks, cuts), want) < R.TOL[dtype], (dtype, cuts)


@pytest.mark.parametrize("lens", [(300,), (129, 64, 1, 257)])
def test_unequal_prompts_in_one_bucket(lens):
    cfg = R.config([R.attention(heads=6, kv_heads=3, dim=48, vdim=56, mlp=R.moe()), R.latent(mlp=R.moe(ff=72))], vocab=800)
    t = R.tensors(cfg, 5)
    toks = [R.tokens(cfg, n, seed=i) for i, n in enumerate(lens)]
    orc = O.Oracle(cfg, t)
    for dtype in (BF16, F32):
        eng = R.engine(cfg, t, dtype, rungs=(1024,))
        got = eng.step([(i, x) for i, x in enumerate(toks)])
        for g, x in zip(got, toks):
            assert R.error(g, orc.forward(x)) < R.TOL[dtype]


@pytest.mark.parametrize("n", [1, 2, 3, 4])
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
    cfg = R.CASES["all_equal_heads"]
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
    cfg = R.CASES["every_expert"]
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
