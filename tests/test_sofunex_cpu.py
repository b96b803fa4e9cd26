"""Sofunex without a GPU: descriptions, tensor layouts, plan and command line, the prompt scan's identities and the oracle's own laws."""
import math

import pytest
import torch

import oracle_sofunex as O
import sofunex_cases as R
from saber_engine_b200.cli.main import main as saber
from saber_engine_b200.models import config as MC
from saber_engine_b200.models import stack_config as SC
from saber_engine_b200.models import stack_weights as SW
from saber_engine_b200.plan import launch_plan as LP
from saber_engine_b200.runtime import bench_stack as B


def test_description_is_read_from_the_folder(tmp_path):
    cfg = R.CASES["every_kind"]
    t = R.tensors(cfg)
    R.write_model(tmp_path / "m", cfg, t)
    c = MC.by_name(str(tmp_path / "m"))
    assert (c.arch, c.vocab, c.width, c.eps, c.parallel, c.post_norms, c.token_shift) == ("Sofunex", 203, 104, 1e-5, False, True, True)
    assert (c.embed_scale, c.residual_mult, c.loop, c.loop_linear) == (3.0, 0.6, SC.LoopSpec(1, 3, 2), False)
    assert [type(l.mlp).__name__ for l in c.layers] == ["GatedUnit", "ExpertMix", "ExpertMix", "NoneType"] and [r.layer for r in c.runs] == [0, 1, 2, 1, 2, 3]
    a, d, m = c.layers[1].mixer.left, c.layers[1].mixer.right, c.layers[1].mixer
    assert (a.window, a.taps, a.out_bias, a.qk_norm, a.rot) == (9, 4, True, False, SC.Rotation(900.0, 16, False, 3.0))
    assert (d.heads, d.dim, m.left_scale, m.right_scale) == (3, 20, 0.7, 0.4)
    assert [l.mixer.right.rank for l in c.layers] == [9, 24, 1, 70]                 # from the tensors
    f = c.layers[1].mlp
    assert (f.experts, f.top, f.ff, f.groups, f.keep, f.shared, f.scale, f.gated, f.sigmoid) == (12, 3, 40, 4, 2, 56, 1.7, True, True)
    back = SW.read_safetensors(tmp_path / "m" / "model.safetensors")
    assert set(back) == set(SW.tensor_shapes(c)) and all(torch.equal(back[k], t[k]) for k in t)
    assert c.param_count() == sum(x.numel() for x in t.values())
    assert "loop.in" not in t and "l3.norm2" not in t and "l2.mlp.shared.up" not in t and "l1.mlp.shared.sg" not in t
    # a slot: state, convolution inputs and the last row of every layer run; pages: keys and values of every run
    states = [3 * 24 * 64, 3 * 24 * 64, 5 * 40 * 64] + [3 * 24 * 64, 5 * 40 * 64] + [3 * 24 * 64]
    conv = [3 * (8 * 24 + 2 * 40), 4 * (8 * 24 + 4 * 40), 3 * (8 * 24 + 2 * 40)]
    conv = conv + conv[1:] + [2 * (6 * 24 + 32)]
    assert c.slot_bytes() == 4 * (sum(states) + sum(conv) + 6 * 104)
    assert c.page_token_bytes() == 2 * (2 * 128 + 2 * (4 * 128 + 2 * 128) + (64 + 32))


def test_unknown_parts_are_refused():
    bad = R.config([R.layer()])
    bad["layers"][0]["type"] = "attention"
    with pytest.raises(ValueError):
        R.describe(bad)
    with pytest.raises(ValueError):
        R.describe(R.config([R.layer(mlp={"kind": "lookup"})]))
    with pytest.raises(ValueError, match="w1"):
        SC.from_json(R.config([R.layer()]), name="x")              # a description without its tensors
    for l in (R.layer(heads=5), R.layer(rot=26), R.layer(rot=7), R.layer(delta_dim=600), R.layer(mlp=R.moe(experts=10)), R.layer(mlp=R.moe(groups=(4, 5))),
              R.layer(mlp=R.moe(top=7)), R.layer(mlp=R.moe(2000, groups=None))):
        with pytest.raises(ValueError):
            R.describe(R.config([l]))
    with pytest.raises(ValueError):
        R.describe(R.config([R.layer()], loop=(0, 2, 1)))
    a = SC.GroupedMixer(2, 1, 16, 16, 1.0, qk_norm=False)
    side = SC.SideBySideMixer(a, SC.ChannelDeltaMixer(2, 16, 4))
    for mixer, kw in ((side, {}), (a, dict(post_norms=True)), (SC.ChannelDeltaMixer(2, 16, 4), dict(parallel=False)), (a, dict(parallel=False, token_shift=True)),
                      (SC.DeltaMixer(2, 1, 16, 16, 2), dict(parallel=False, post_norms=True))):
        with pytest.raises(ValueError):
            SC.StackConfig("x", "x", 64, 64, (SC.LayerSpec(mixer),), **kw)
    for mlp in (SC.SquaredRelu(64), SC.ExpertMix(4, 1, 64)):
        with pytest.raises(ValueError):
            SC.StackConfig("x", "x", 64, 64, (SC.LayerSpec(side, mlp),), parallel=False, post_norms=True)
    with pytest.raises(ValueError):
        SC.StackConfig("x", "x", 64, 64, (SC.LayerSpec(a, SC.GatedUnit(64)),), parallel=False)
    cfg = R.CASES["wide"]
    t = R.tensors(cfg)
    t["l1.mix.right.w2"] = t["l1.mix.right.w2"][:-1]
    with pytest.raises(ValueError, match="w2"):
        SW.build(R.describe(cfg), t.__getitem__, torch.float32, "cpu")


def _gated(rows, ff, W):
    """Gate and up rows of a stack of tiles."""
    x = rows.view(-1, 2, 128, rows.shape[-1])
    return x[:, 0].reshape(-1, rows.shape[-1])[:ff, :W], x[:, 1].reshape(-1, rows.shape[-1])[:ff, :W]


@pytest.mark.parametrize("name", list(R.CASES))
def test_packed_linears_hold_every_row_once(name):
    """fp32 layout: every tensor is found where the kernels read it, and nothing else is there."""
    cfg = R.CASES[name]
    t = R.tensors(cfg, 1)
    c = R.describe(cfg)
    w = SW.build(c, t.__getitem__, torch.float32, "cpu")
    W = c.width
    for i, (l, lw) in enumerate(zip(c.layers, w.layers)):
        p, f, got = f"l{i}.", l.mlp, 0.0
        for seg, n in l.mixer.segments():
            assert torch.equal(lw.proj.w[lw.off[seg]: lw.off[seg] + n, :W], t[f"{p}mix.{seg}"].float())
        for seg in ("left.q", "left.k", "left.v", "right.a"):
            n = t[f"{p}mix.{seg}.b"].numel()
            assert torch.equal(lw.bias[lw.off[seg]: lw.off[seg] + n], t[f"{p}mix.{seg}.b"].float())
        for side, n in (("left", l.mixer.left.out_features), ("right", l.mixer.right.out_features)):
            k0 = lw.mix_k0[side + "."]
            assert k0 % 64 == 0 and torch.equal(lw.out.w[:W, k0: k0 + n], t[f"{p}mix.{side}.o"].float())
        assert torch.allclose(lw.out_bias[:W], l.mixer.left_scale * t[p + "mix.left.o.b"].float()) and not lw.out_bias[W:].any()
        right, left = lw.part("right."), lw.part("left.")
        assert not right.extra["w2"][:, l.mixer.right.rank:].any() and torch.equal(left.extra["conv"].T, torch.cat([t[f"{p}mix.left.{n}.conv"] for n in "qkv"]).float())
        assert torch.equal(right.extra["w2"][:, : l.mixer.right.rank], t[p + "mix.right.w2"].float()) and set(left.off) == {"q", "k", "v"} and "conv" in left.extra
        for got_row, key in ((lw.norm, "norm1"), (lw.post1, "norm1b"), (lw.shift, "shift"), *(((lw.norm2, "norm2"), (lw.post2, "norm2b")) if f else ())):
            assert got_row.numel() % 8 == 0 and torch.equal(got_row[:W], t[p + key].float()) and not got_row[W:].any()
        got = sum(float(x.w.abs().sum()) for x in lw.linears())
        total = sum(float(x.float().abs().sum()) for k, x in t.items() if k.startswith(p) and x.dim() == 2 and ".conv" not in k and not k.endswith("right.w2"))
        assert abs(got - total) < 1e-3 * total
        if f is None:
            assert lw.up is None and lw.norm2 is None
            continue
        at = "" if isinstance(f, SC.GatedUnit) else "shared."
        if at:
            assert torch.equal(lw.up.w[: f.experts, :W], t[p + "mlp.router"].float()) and torch.equal(lw.correction, t[p + "mlp.correction"].float())
            eu, ed = (x.w.view(f.experts, x.N_pad, x.K) for x in (lw.experts_up, lw.experts_down))
            for e in range(f.experts):
                gate, up = _gated(eu[e], f.ff, W)
                assert torch.equal(gate, t[f"{p}mlp.e{e}.gate"].float()) and torch.equal(up, t[f"{p}mlp.e{e}.up"].float())
                assert torch.equal(ed[e, :W, : f.ff], t[f"{p}mlp.e{e}.down"].float())
        if f.inner:
            gate, up = _gated(lw.up.w[lw.up_tile0 * 256:], f.inner, W)
            assert torch.equal(gate, t[f"{p}mlp.{at}gate"].float()) and torch.equal(up, t[f"{p}mlp.{at}up"].float())
            assert torch.equal(lw.down.w[:W, : f.inner], t[f"{p}mlp.{at}down"].float())
        else:
            assert lw.down is None


def test_block_form_of_the_recurrence_equals_the_token_form():
    """The identities the prompt kernel rests on: four tokens from the state at their start, products of decays only."""
    g = torch.Generator().manual_seed(0)
    H, D, T = 2, 5, 12
    r, k, v = (torch.randn(T, H, D, generator=g).double() for _ in range(3))
    w, a = (torch.rand(T, H, D, generator=g).double() for _ in range(2))
    want, last = O.delta_states(r, k, v, w, a)
    u = k / torch.sqrt((k * k).sum(-1, keepdim=True) + 1e-6)
    b = -a * u
    S = torch.zeros(H, D, D).double()
    between = lambda i, j, at: torch.ones(H, D).double() if i <= j else between(i - 1, j, at) * w[at + i]      # noqa: E731  w_{j+1} .. w_i
    for at in range(0, T, 4):
        held = []
        for i in range(4):
            before, upto = between(i - 1, -1, at), between(i, -1, at)
            p = torch.einsum("hdv,hd->hv", S, u[at + i] * before)
            for j in range(i):
                d = between(i - 1, j, at)
                p = p + (u[at + i] * d * k[at + j]).sum(-1, keepdim=True) * v[at + j] + (u[at + i] * d * b[at + j]).sum(-1, keepdim=True) * held[j]
            held.append(p)
            o = torch.einsum("hdv,hd->hv", S, r[at + i] * upto)
            for j in range(i + 1):
                d = between(i, j, at)
                o = o + (r[at + i] * d * k[at + j]).sum(-1, keepdim=True) * v[at + j] + (r[at + i] * d * b[at + j]).sum(-1, keepdim=True) * held[j]
            assert torch.allclose(o, want[at + i])
        S = S * between(3, -1, at)[..., None] + sum((between(3, j, at) * k[at + j])[..., None] * v[at + j][:, None] + (between(3, j, at) * b[at + j])[..., None] * held[j][:, None]
                                                    for j in range(4))
    assert torch.allclose(S, last)


def test_oracle_laws():
    """A position's logits depend on earlier tokens only; a window's edge; an untouched blend; a key that is removed and written again."""
    cfg = R.CASES["every_kind"]
    t = R.tensors(cfg)
    o = O.Oracle(cfg, t)
    toks = R.tokens(cfg, 40)
    assert torch.allclose(o.forward(toks)[:27], o.forward(toks[:27]))
    g = torch.Generator().manual_seed(0)
    s = torch.randn(2, 9, 9, generator=g).double()
    p = O.window_weights(s, 4)
    assert torch.allclose(p.sum(-1), torch.ones(2, 9).double()) and int((p[0, 8] > 0).sum()) == 4 and p[0, 8, 5] > 0 and p[0, 8, 4] == 0
    assert torch.equal(O.window_weights(s, 9), O.window_weights(s, 0)) and int((p[0, 2] > 0).sum()) == 3
    h = torch.randn(6, 8, generator=g).double()
    assert torch.equal(O.shifted(h, torch.zeros(8)), h) and torch.allclose(O.shifted(h, torch.ones(8))[1:], h[:-1]) and not O.shifted(h, torch.ones(8))[0].any()
    u = torch.randn(6, 3, generator=g).double()
    assert torch.allclose(O.causal_conv(u, torch.tensor([[0.0, 0.0, 2.0]] * 3).double()), 2 * u) and torch.allclose(O.causal_conv(u, torch.tensor([[1.0, 0.0, 0.0]] * 3).double())[2:], u[:-2])
    # one key, no decay: removed at rate one it holds the last value only
    k = torch.tensor([1.0, 0.0]).double().expand(3, 1, 2)
    v = torch.randn(3, 1, 2, generator=g).double()
    out, _ = O.delta_states(k, k, v, torch.ones(3, 1, 2).double(), torch.ones(3, 1, 2).double())
    assert torch.allclose(out, v, atol=1e-5)
    decay, rate = O.channel_rates(h[:, :4], {"w1": torch.zeros(2, 4).double(), "w2": torch.zeros(3, 2).double(), "w0": torch.full((3,), 90.0).double(), "a": torch.zeros(3, 4).double(),
                                             "a.b": torch.zeros(3).double()}, 1)
    assert torch.allclose(decay, torch.full((6, 1, 3), math.exp(-math.exp(-0.5))).double()) and torch.allclose(rate, torch.full((6, 1, 3), 0.5).double())


def test_oracle_routing():
    s, none = [0.9, 0.1, 0.6, 0.55, 0.2, 0.85], [0.0] * 6
    pick = lambda *a: [e for e, _ in O.route(*a)]      # noqa: E731
    assert pick(s, none, 2, {"count": 1, "keep": 1}) == [0, 5]
    assert pick(s, none, 2, {"count": 3, "keep": 1}) == [2, 3]              # two good members beat one of the best
    shares = O.route(s, [0, 0.7, 0, 0, 0.7, 0], 2, {"count": 1, "keep": 1})
    assert sorted(e for e, _ in shares) == [0, 4] and math.isclose(dict(shares)[4], 0.2 / 1.1)      # chosen with the correction, weighted without


def test_plan_registry_and_command_line(capsys):
    man = LP.Manifest(model="sofunex-mini", max_ctx=2048, max_seqs=4, decode_batches=(1, 4), decode_widths=(1,), prefill_rows=(64,), budget_mib=12000)
    plan = LP.bind(LP.resolve(man))
    c = MC.by_name("sofunex-mini")
    assert plan.kv_blocks >= 2048 // 64 + 1 and plan.ledger.items["recurrent_state_slots"] == 5 * c.slot_bytes()
    assert plan.ledger.items["expert_rows"] == 2 * c.expert_row_bytes(64) > 0 and plan.ledger.items["weights"] == 2 * c.param_count()
    assert plan.ledger.items["scan_rows"] == c.scan_row_bytes(64) > 0
    man.decode_widths = (1, 5)
    with pytest.raises(LP.PlanError):
        LP.resolve(man)
    assert saber(["serve", "--model", "sofunex", "--random-init", "--print-argv"]) == 0
    assert "--engine-config sofunex-mini" in capsys.readouterr().out
    assert saber(["explain", "--model", "sofunex-mini"]) == 0


def test_bench_models_and_costs():
    cfg = MC.by_name("sofunex-4k")
    like = B.like_models(cfg)
    assert [x.name.split("-like")[0] for x in like] == ["fitatar", "renosun", "hybrid"]
    for M in (8, 2048):
        costs = B.stack_costs(cfg, M, 8, 8.0 * M, 4096.0)
        assert {"experts_up", "experts_down", "route", "up", "down", "up+experts", "down+experts", "mixer:attention", "mixer:channel_delta", "join"} <= set(costs)
        assert costs["experts_up"][1] == 4.0 * M * 6 * 1024 * 4096
