"""Renosun on the GPU against the plain restatement in oracle_renosun.py."""
import json
import os
import subprocess
import sys

import pytest
import torch

import oracle_renosun as O
import renosun_cases as R
from saber_engine_b200.sched.scheduler import Scheduler, SchedulerConfig
from saber_engine_b200.serve.engine_api import EngineRequest, SamplingParams

pytestmark = pytest.mark.gpu
F32, BF16 = torch.float32, torch.bfloat16
REPO = os.path.dirname(os.path.dirname(os.path.abspath(__file__)))


# ------------------------------------------------------------------------------ mechanisms, one layer each
ALONE = {
    "delta": [R.delta(ff=None)],
    "delta_no_conv_history": [R.delta(ff=None, conv=1, heads=4, kv_heads=2)],
    "delta_equal_heads_long_conv": [R.delta(ff=None, conv=6, heads=2, kv_heads=2, dim=64, vdim=72)],
    "latent": [R.latent(ff=None)],
    "latent_one_head": [R.latent(ff=None, heads=1, dim=40, rot_dim=8, vdim=8, kv_rank=16)],
    "feed_forward_beside_delta": [R.delta(ff=130, limit=0.4)],
    "feed_forward_beside_latent": [R.latent(ff=33, limit=3.0)],
}


@pytest.mark.parametrize("name", ALONE)
@pytest.mark.parametrize("dtype", [F32, BF16])
def test_mechanism_alone_residual_stream(name, dtype):
    cfg = R.config(ALONE[name])
    t = R.tensors(cfg, seed=3)
    toks = R.tokens(cfg, 70)
    trace = []
    O.Oracle(cfg, t).forward(toks, trace)
    eng = R.engine(cfg, t, dtype, rungs=(80,))
    eng.step([("a", toks)])
    b = next(iter(eng.model.buckets.values()))
    x = b.x[:70, : cfg["width"]].cpu().double()
    assert float((x - trace[0]).abs().max() / trace[0].abs().max()) < (1e-5 if dtype == F32 else 0.03)


@pytest.mark.parametrize("fuse", [True, False])
@pytest.mark.parametrize("M,N,K,splits", [(1, 40, 64, 1), (7, 520, 640, 5), (16, 256, 1024, 16), (130, 300, 192, 1), (300, 1000, 128, 1)])
def test_linear_project_and_stream(M, N, K, splits, fuse):
    """The bf16 linear by itself: projection with the row norm folded in, and the residual epilogue."""
    import ctypes as C
    from saber_engine_b200.models import stack_weights as SW
    from saber_engine_b200.ops import functional as F
    from saber_engine_b200.ops import layouts as L
    from saber_engine_b200.ops import native as NN
    g = torch.Generator().manual_seed(M + N)
    w = (torch.randn(N, K, generator=g) / K ** 0.5).bfloat16()
    a = torch.randn(M, K, generator=g).bfloat16()
    n_pad = L.round_up(N, 256)
    wp = torch.zeros(n_pad, K, dtype=BF16)
    wp[:N] = w
    lin = SW.pack_linear(wp.cuda(), BF16)
    m_pad = L.padded_rows(M)
    op = torch.zeros(K // 64, m_pad, 8, 8, dtype=BF16)                      # [k-block][row][16-byte chunk][8]
    rows, chunk = torch.arange(M)[:, None], torch.arange(8)[None, :]
    for kb in range(K // 64):
        op[kb, rows, chunk ^ (rows & 7)] = a[:, kb * 64:(kb + 1) * 64].reshape(M, 8, 8)
    op = op.cuda()
    sc = F.scratch("cuda")
    ss = torch.rand(m_pad, 3, generator=g).cuda() + 0.5
    ws = torch.zeros(M * n_pad + (1 << 22), dtype=F32, device="cuda")

    def run(e):
        p = NN.LinParams()
        p.w, p.a, p.err, p.ws, p.counters = lin.w.data_ptr(), op.data_ptr(), sc.err.data_ptr(), ws.data_ptr(), sc.counters.data_ptr()
        p.M, p.M_pad, p.N_pad, p.K, p.nt, p.splits, p.fp32, p.fuse = M, m_pad, n_pad, K, L.token_tile(M), splits, 0, int(fuse)
        p.mtiles = 2 if m_pad % 256 == 0 else 1
        p.e = e
        NN.check(NN.lib().saber_linear_launch(C.byref(p), NN.stream_handle()), "linear")
        torch.cuda.synchronize()
        sc.check()
    acc = a.double() @ w.double().T
    out = torch.full((M, L.round_up(N, 8) + 8), 7.0, dtype=F32, device="cuda")
    e = NN.LinEpi()
    e.ss, e.ss_n, e.inv_width, e.eps, e.out, e.ldo, e.n_plain, e.act_tile0 = ss.data_ptr(), 3, 0.25, 1e-3, out.data_ptr(), out.stride(0), N, n_pad // 256
    run(e)
    want = acc / torch.sqrt(ss[:M].cpu().double().sum(1) * 0.25 + 1e-3)[:, None]
    assert (out[:, :N].cpu().double() - want).abs().max() < 2e-5 * want.abs().max()
    assert torch.all(out[:, N:] == 7.0)
    ld = L.round_up(N, 32)
    x0 = torch.zeros(M, ld)
    x0[:, :N] = torch.randn(M, N, generator=g)
    x, bias, nw = x0.cuda(), torch.randn(N, generator=g).cuda(), torch.randn(N, generator=g).cuda()
    ko = L.round_up(N, 64)
    nxt = torch.zeros(ko // 64, m_pad, 8, 8, dtype=BF16, device="cuda")
    ss2 = torch.zeros(m_pad, (N + 127) // 128, dtype=F32, device="cuda")
    e = NN.LinEpi()
    e.stream, e.x, e.ldx, e.width, e.add, e.bias, e.norm_w = 1, x.data_ptr(), ld, N, 1, bias.data_ptr(), nw.data_ptr()
    e.op.p, e.op.M_pad, e.op.ld, e.op.fmt = nxt.data_ptr(), m_pad, ko, 0
    e.ss_out, e.ss_out_n = ss2.data_ptr(), ss2.shape[1]
    run(e)
    want = x0[:, :N].double() + acc + bias.cpu().double()
    assert (x[:, :N].cpu().double() - want).abs().max() < 2e-5 * want.abs().max()
    assert torch.allclose(ss2[:M].sum(1).cpu().double(), (want ** 2).sum(1), rtol=1e-4)
    got = torch.zeros(M, ko, dtype=BF16)
    nx = nxt.cpu()
    for kb in range(ko // 64):
        got[:, kb * 64:(kb + 1) * 64] = nx[kb, rows, chunk ^ (rows & 7)].reshape(M, 64)
    wo = want * nw.cpu().double()
    assert (got[:, :N].double() - wo).abs().max() < 0.01 * wo.abs().max()


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


def test_expanded_and_absorbed_prompts_agree():
    cfg = R.CASES["wide_heads"]
    t = R.tensors(cfg, seed=9)
    toks = R.tokens(cfg, 333)
    want = O.Oracle(cfg, t).forward(toks)
    for kw, form in (({}, 2), ({"attn_impl": "mma"}, 1), ({"expand_bytes": 0}, 0)):      # without the scratch pages prompts stay in the latent space
        eng = R.engine(cfg, t, BF16, **kw)
        assert eng.model._expanded(eng.model.cfg.layers[0].mixer, 256, False) == form
        assert R.error(R.feed(eng, "r", toks, [333]), want) < R.TOL[BF16]
        assert R.error(R.feed(eng, "r", toks, [70, 130, 2]), want) < R.TOL[BF16]


# ------------------------------------------------------------------------------ far keys, borders, long runs
def _needle(cfg: dict, seed: int):
    """Weights and tokens with a needle: one layer of latent attention whose query for the last token id meets the
    key of token id 1 with a score far above all others, wherever that token stands."""
    t = R.tensors(cfg, seed)
    W, m = cfg["width"], cfg["layers"][0]["mixer"]
    t["embed"][:, 0] = 0.0
    t["embed"][1, 0] = 6.0                                       # only the needle has this coordinate
    t["embed"][cfg["vocab"] - 1, 1] = 6.0
    t["l0.norm1"][:] = 1.0
    dkv = t["l0.mix.dkv"]
    dkv[0, :] = 0.0
    dkv[0, 0] = 8.0                                              # latent coordinate 0 <- needle
    t["l0.mix.dkv.norm"][:] = 1.0
    uk = t["l0.mix.uk"].view(m["heads"], m["dim"], m["kv_rank"])
    uk[:, 0, :] = 0.0
    uk[:, 0, 0] = 2.0
    q = t["l0.mix.q"].view(m["heads"], m["dim"] + m["rot_dim"], W)
    q[:, 0, :] = 0.0
    q[:, 0, 1] = 6.0                                             # the asking token's query along it
    return t


@pytest.mark.parametrize("dtype", [F32, BF16])
@pytest.mark.parametrize("place", [0, 1, 62, 63, 64, 65, 127, 128, 500])
def test_one_key_far_away_and_at_page_borders(dtype, place):
    cfg = R.config([R.latent(heads=3, dim=24, rot_dim=12, vdim=20, kv_rank=56, scale=0.4, ff=None)], vocab=131)
    t = _needle(cfg, 2)
    n = 520
    toks = [2 + x % 120 for x in R.tokens(cfg, n)]
    toks[place] = 1
    toks[-1] = cfg["vocab"] - 1
    orc = O.Oracle(cfg, t)
    want = orc.forward(toks)
    without = list(toks)
    without[place] = 2
    assert R.error(orc.forward(without)[-1:], want[-1:]) > 0.3   # the answer hangs on that one key
    eng = R.engine(cfg, t, dtype, rungs=(64, 256, 1024))
    tol = {F32: 5e-5, BF16: 0.08}[dtype]
    assert R.error(R.feed(eng, "r", toks, [n])[-1:], want[-1:]) < tol                   # asked in the prompt
    assert R.error(R.feed(eng, "r", toks, [n - 1, 1])[-1:], want[-1:]) < tol            # asked by a decoded token
    assert R.error(R.feed(eng, "r", toks, [place + 1, 1, 200, 255, 1])[-1:], want[-1:]) < tol


@pytest.mark.parametrize("scale", [0.05, 1.5])
@pytest.mark.parametrize("lens", [(300,), (129, 64, 1, 257), (128, 640)])
def test_prompt_attention_over_growing_scores(lens, scale):
    """Scores that rise along the keys (the running maximum moves in every block) and unequal prompts side by side."""
    cfg = R.config([R.latent(heads=3, dim=48, rot_dim=16, vdim=56, kv_rank=80, scale=scale, ff=None)], vocab=800)
    t = R.tensors(cfg, 5)
    t["embed"] = (t["embed"].float() * torch.linspace(0.2, 1.0, 800)[:, None]).bfloat16()
    toks = [sorted(R.tokens(cfg, n, seed=i)) for i, n in enumerate(lens)]
    orc = O.Oracle(cfg, t)
    for kw in ({}, {"attn_impl": "mma"}):
        eng = R.engine(cfg, t, BF16, rungs=(1024,), **kw)
        got = eng.step([(i, x) for i, x in enumerate(toks)])
        for g, x in zip(got, toks):
            assert R.error(g, orc.forward(x)) < 0.06 * max(1.0, scale)


def test_keys_reached_by_position_only():
    """Scores from the rotated part alone: a wrong position, frequency or pairing moves the peak."""
    cfg = R.config([R.latent(heads=2, dim=8, rot_dim=16, vdim=24, kv_rank=40, base=40.0, scale=1.0, ff=None)])
    t = R.tensors(cfg, 4)
    m = cfg["layers"][0]["mixer"]
    q = t["l0.mix.q"].view(2, m["dim"] + m["rot_dim"], cfg["width"])
    q[:, : m["dim"]] = 0.0
    q[:, m["dim"]:] *= 3.0
    t["l0.mix.dkv"][m["kv_rank"]:] *= 3.0
    toks = R.tokens(cfg, 400)
    want = O.Oracle(cfg, t).forward(toks)
    for dtype in (F32, BF16):
        eng = R.engine(cfg, t, dtype)
        # (the scores are in the tens: bf16 operands move them by tenths)
        assert R.error(R.feed(eng, "r", toks, [400]), want) < {F32: 1e-4, BF16: 0.3}[dtype]
        assert R.error(R.feed(eng, "r", toks, [390, 1]), want) < {F32: 1e-4, BF16: 0.3}[dtype]


def test_state_carries_far_and_a_lost_state_shows():
    """Slow decay: the first tokens' writes are still read hundreds of tokens later, over every cut."""
    cfg = R.config([R.delta(ff=None, dim=40, vdim=24)])
    t = R.tensors(cfg, 6)
    t["l0.mix.A_log"][:] = -6.0
    t["l0.mix.b"] *= 0.2
    toks = R.tokens(cfg, 300)
    orc = O.Oracle(cfg, t)
    want = orc.forward(toks)
    assert R.error(orc.forward(R.tokens(cfg, 20, 9) + toks[20:])[-1:], want[-1:]) > 0.01
    eng = R.engine(cfg, t, F32)
    for cuts in ([300], [255, 2, 43], [4, 3, 5, 1, 2, 6, 200, 1]):
        assert R.error(R.feed(eng, "r", toks, cuts), want) < 3e-5


@pytest.mark.parametrize("n", [1, 2, 3, 4, 5, 6])
def test_first_tokens(n):
    cfg = R.config([R.delta(conv=4), R.latent(), R.delta(conv=5, ff=None)], loop=(0, 1, 2))
    t = R.tensors(cfg, 8)
    toks = R.tokens(cfg, n)
    want = O.Oracle(cfg, t).forward(toks)
    for dtype in (F32, BF16):
        eng = R.engine(cfg, t, dtype)
        for cuts in ([n], [1], [2]):
            assert R.error(R.feed(eng, "r", toks, cuts), want) < R.TOL[dtype]


def test_long_decoding_over_page_borders():
    cfg = R.CASES["mixed_loop"]
    t = R.tensors(cfg, 10)
    toks = R.tokens(cfg, 330)
    want = O.Oracle(cfg, t).forward(toks)
    for dtype in (F32, BF16):
        eng = R.engine(cfg, t, dtype, capture=True)
        assert R.error(R.feed(eng, "r", toks, [10, 1]), want) < R.TOL[dtype]


def test_unfused_linears_agree():
    cfg = R.CASES["mixed_loop"]
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
    cfg = R.CASES["mixed_loop"]
    t = R.tensors(cfg, 12)
    m = R.model(cfg, t, F32, max_seqs=4, max_ctx=512)
    ex = HybridExecutor(m, decode_batches=(1, 2, 4), decode_widths=(1,), prefill_rungs=(32, 128))
    return cfg, O.Oracle(cfg, t), ex


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
    # sampled: top_k = 1 is greedy, a seed fixes the ids, the device draws what the host draws
    s = _sched(ex, prefix_cache=False)
    kw = dict(max_tokens=8, ignore_eos=True)
    subs = [s.submit(EngineRequest(p1, SamplingParams(temperature=1.0, top_k=1, seed=3, **kw))),
            s.submit(EngineRequest(p1, SamplingParams(temperature=1.3, seed=4, **kw))),
            s.submit(EngineRequest(p1, SamplingParams(temperature=1.3, seed=4, logprobs=2, **kw)))]
    s.run_until_idle()
    a, b, c = [_collect(x)[0] for x in subs]
    assert a == want[0] and b == c
    assert s.counters["sampled_steps_device_agrees"] == s.counters["sampled_steps"] > 0


def test_prompt_logprobs(served):
    cfg, orc, ex = served
    p = R.tokens(cfg, 150, seed=41)
    s = _sched(ex, prefix_cache=False)
    sub = s.submit(EngineRequest(p, SamplingParams(max_tokens=1, ignore_eos=True, prompt_logprobs=2)))
    s.run_until_idle()
    lps = _collect(sub)[1].prompt_logprobs
    want = torch.log_softmax(orc.forward(p), -1)
    assert len(lps) == 149
    for i, d in enumerate(lps):
        assert d["token_id"] == p[i + 1] and abs(d["logprob"] - float(want[i, p[i + 1]])) < 1e-3


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
    cfg = R.CASES["no_loop"]
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
