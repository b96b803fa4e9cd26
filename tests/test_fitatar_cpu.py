"""Fitatar without a GPU: descriptions, tensor layouts, plan and command line, and the oracle's own laws."""
import math

import pytest
import torch

import fitatar_cases as R
import oracle_fitatar as O
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
    assert (c.arch, c.vocab, c.width, c.eps, c.parallel, c.two_norms, c.logit_cap, c.embed_scale) == ("Fitatar", 203, 104, 1e-5, True, True, 8.0, 3.0)
    assert [type(l.mixer).__name__ for l in c.layers] == ["GroupedMixer", "LatentMixer", "GroupedMixer", "LatentMixer"]
    assert [type(l.mlp).__name__ for l in c.layers] == ["Gelu", "ExpertMix", "ExpertMix", "ExpertMix"]
    assert [c.pages_of(r) for r in c.runs] == [0, 1, 2, 1]
    a, la, f = c.layers[0].mixer, c.layers[1].mixer, c.layers[1].mlp
    assert (a.rot, a.sink, a.gate, a.qk_norm, a.bias) == (SC.Rotation(900.0, 16, False, 3.0), True, True, False, False)
    assert (la.rot, la.q_rank, la.gate_heads) == (SC.Rotation(700.0, 12, True, 2.5, (64.0, 20.0, 1.5)), 40, True)
    assert (f.experts, f.top, f.ff, f.groups, f.keep, f.shared) == (12, 3, 40, 4, 2, 56) and c.layers[2].mlp.shared == 0
    back = SW.read_safetensors(tmp_path / "m" / "model.safetensors")
    assert set(back) == set(SW.tensor_shapes(c)) and all(torch.equal(back[k], t[k]) for k in t)
    assert c.param_count() == sum(x.numel() for x in t.values())
    assert "l3.mix.dkv" not in t and "l3.mix.dkv.norm" not in t and "l2.mlp.shared.up" not in t
    # pages: keys and values of two layers, the latents and key parts of one
    assert c.page_token_bytes() == 2 * (2 * (64 + 64) + 2 * (64 + 64) + 64 + 16)


def test_unknown_parts_are_refused():
    bad = R.config([R.attention()])
    bad["layers"][0]["type"] = "conv"
    with pytest.raises(ValueError):
        SC.from_json(bad)
    bad = R.config([R.attention(mlp={"kind": "lookup"})])
    with pytest.raises(ValueError):
        SC.from_json(bad)
    for layers in ([R.attention(heads=5)], [R.attention(rot=26)], [R.attention(rot=7)], [R.latent(rot_dim=7)], [R.latent(kv_from=0)],
                   [R.attention(), R.latent(kv_from=0)], [R.latent(), R.latent(kv_rank=48, kv_from=0)], [R.latent(), R.latent(base=9.0, kv_from=0)],
                   [R.latent(), R.latent(kv_from=0), R.latent(kv_from=1)], [R.attention(mlp=R.moe(experts=10))], [R.attention(mlp=R.moe(keep=5))],
                   [R.attention(mlp=R.moe(top=7))], [R.attention(mlp=R.moe(experts=2000, groups=1, keep=1))]):
        with pytest.raises(ValueError):
            SC.from_json(R.config(layers), name="x")
    for mlp in (SC.Gelu(64), SC.ExpertMix(4, 1, 64)):
        with pytest.raises(ValueError):
            SC.StackConfig("x", "x", 64, 64, (SC.LayerSpec(SC.GroupedMixer(1, 1, 16, 16, 1.0), mlp),), parallel=False)
    cfg = R.CASES["all_equal_heads"]
    t = R.tensors(cfg)
    t["l1.mix.uq"] = t["l1.mix.uq"][:-1]
    with pytest.raises(ValueError, match="uq"):
        SW.build(SC.from_json(cfg, name="x"), t.__getitem__, torch.float32, "cpu")


@pytest.mark.parametrize("name", list(R.CASES))
def test_packed_linears_hold_every_row_once(name):
    """fp32 layout: every tensor is found where the kernels read it, and nothing else is there."""
    cfg = R.CASES[name]
    t = R.tensors(cfg, 1)
    c = SC.from_json(cfg, name="x")
    w = SW.build(c, t.__getitem__, torch.float32, "cpu")
    W = c.width
    for i, (l, lw) in enumerate(zip(c.layers, w.layers)):
        p, m, f, rows = f"l{i}.", l.mixer, l.mlp, dict(l.mixer.segments())
        for seg, n in rows.items():
            assert torch.equal(lw.proj.w[lw.off[seg]: lw.off[seg] + n, :W], t[f"{p}mix.{seg}"].float())
        assert torch.equal(lw.out.w[:W, : m.out_features], t[p + "mix.o"].float())
        if m.q_rank:
            assert lw.off["dq"] == 0 and lw.lat_tiles * 256 >= m.q_rank and min(lw.off[s] for s in rows if s != "dq") >= lw.lat_tiles * 256
            assert torch.equal(lw.carry.w[: m.query_rows, : m.q_rank], t[p + "mix.uq"].float())
        up = lw.proj.w[lw.act_tile0 * 256:]
        if f is None:
            assert up.numel() == 0 and lw.norm2 is None
            continue
        assert torch.equal(lw.norm2, t[p + "norm2"].float()) and max(lw.off[s] + n for s, n in rows.items()) <= lw.tile2 * 256
        if isinstance(f, SC.Gelu):
            assert torch.equal(up[: f.ff, :W], t[p + "mlp.up"].float()) and torch.equal(lw.act_bias[: f.ff], t[p + "mlp.up.b"].float())
            assert torch.equal(lw.out.w[:W, lw.act_k0: lw.act_k0 + f.ff], t[p + "mlp.down"].float()) and torch.equal(lw.out_bias, t[p + "mlp.down.b"].float())
            continue
        assert lw.off["router"] == lw.tile2 * 256 and torch.equal(lw.proj.w[lw.off["router"]:][: f.experts, :W], t[p + "mlp.router"].float())
        if f.shared:
            tiles = up.view(-1, 256, up.shape[1])
            assert torch.equal(tiles[:, :248].reshape(-1, up.shape[1])[: f.shared, :W], t[p + "mlp.shared.up"].float())
            assert all(torch.equal(x[248, :W], t[p + "mlp.shared.sg"][0].float()) for x in tiles)
            assert torch.equal(lw.out.w[:W, lw.act_k0: lw.act_k0 + f.shared], t[p + "mlp.shared.down"].float())
        eu, ed = (x.w.view(f.experts, x.N_pad, x.K) for x in (lw.experts_up, lw.experts_down))
        for e in range(f.experts):
            assert torch.equal(eu[e, : f.ff, :W], t[f"{p}mlp.e{e}.up"].float()) and torch.equal(ed[e, :W, : f.ff], t[f"{p}mlp.e{e}.down"].float())
        total = sum(float(x.float().abs().sum()) for k, x in t.items() if k.startswith(p) and x.dim() == 2 and k not in (p + "mix.uk", p + "mix.uv"))
        total += (f.tiles - 1) * float(t[p + "mlp.shared.sg"].float().abs().sum()) if f.shared else 0.0
        assert abs(float(sum(x.w.abs().sum() for x in lw.linears())) - total) < 1e-3 * total


@pytest.mark.parametrize("base,dims,yarn", [(700.0, 12, (2.5, 64, 20.0, 1.5)), (1e6, 64, (8.0, 4096, 32.0, 1.0)), (50.0, 32, (4.0, 1e5, 4.0, 2.0)),
                                            (1e6, 48, (4.0, 16, 64.0, 30.0)), (10000.0, 2, (2.0, 128, 32.0, 1.0))])
def test_rotations_agree_with_the_oracle(base, dims, yarn):
    s = dict(zip(("factor", "original", "fast", "slow"), yarn))
    for scaling in (s, {"factor": 3.0}, None):
        d = {"base": base, "dims": dims, **({"scaling": scaling} if scaling else {})}
        r = SC.Rotation.from_json(d)
        f, amp = O.frequencies(base, dims, scaling)
        assert torch.allclose(torch.tensor(r.frequencies(), dtype=torch.float64), f, rtol=1e-12) and math.isclose(r.amplitude, amp, rel_tol=1e-12)


def test_oracle_laws():
    """A position's logits depend on earlier tokens only; a rotation keeps scores of equal distances; a large sink empties a head."""
    cfg = R.CASES["every_kind"]
    o = O.Oracle(cfg, R.tensors(cfg))
    toks = R.tokens(cfg, 60)
    assert torch.allclose(o.forward(toks)[:37], o.forward(toks[:37]))
    g = torch.Generator().manual_seed(0)
    q, k = (torch.randn(1, 1, 16, generator=g).double().expand(40, 1, 16) for _ in range(2))
    for rot in ({"base": 30.0, "dims": 12, "scaling": {"factor": 2.0}}, {"base": 30.0, "dims": 16, "scaling": dict(factor=4.0, original=64, fast=8.0, slow=1.0)}):
        for interleaved in (True, False):
            s = O.rotate(q, rot, interleaved)[:, 0] @ O.rotate(k, rot, interleaved)[:, 0].T
            assert torch.allclose(s[5:, 5:], s[:-5, :-5]) and not torch.allclose(s[0], s[1])
    s = torch.randn(2, 4, 4, generator=g).double()
    assert torch.allclose(O.causal_weights(s).sum(-1), torch.ones(2, 4).double())
    w = O.causal_weights(s, torch.tensor([50.0, -50.0]).double())
    assert float(w[0].sum()) < 1e-12 and torch.allclose(w[1], O.causal_weights(s)[1])


def test_oracle_routing():
    groups = {"count": 3, "keep": 2}
    s = [0.05, 0.30, 0.01, 0.02, 0.28, 0.03, 0.04, 0.27]
    assert O.route(s + [0.0], 3, groups) == [1, 4, 0]                      # the third best stands in a group that is out
    assert O.route(s + [0.0], 2, {"count": 3, "keep": 1}) == [1, 0]
    assert O.route(s + [0.0], 3, {"count": 1, "keep": 1}) == [1, 4, 7]


def test_plan_registry_and_command_line(capsys):
    man = LP.Manifest(model="fitatar-mini", max_ctx=2048, max_seqs=4, decode_batches=(1, 4), decode_widths=(1,), prefill_rows=(64,), budget_mib=12000)
    plan = LP.bind(LP.resolve(man))
    assert plan.kv_blocks >= 2048 // 64 + 1 and plan.ledger.items["recurrent_state_slots"] == 0
    c = MC.by_name("fitatar-mini")
    assert plan.ledger.items["expert_rows"] == 2 * c.expert_row_bytes(64) > 0 and plan.ledger.items["weights"] == 2 * c.param_count()
    man.decode_widths = (1, 5)
    with pytest.raises(LP.PlanError):
        LP.resolve(man)
    assert saber(["serve", "--model", "fitatar", "--random-init", "--print-argv"]) == 0
    assert "--engine-config fitatar-mini" in capsys.readouterr().out
    assert saber(["explain", "--model", "fitatar-mini"]) == 0


def test_bench_models_and_costs():
    cfg = MC.by_name("fitatar-4k")
    like = B.like_models(cfg)
    assert [x.name.split("-like")[0] for x in like] == ["tepavik", "renosun", "hybrid"] and like[2].moe.n_experts == 64
    for M in (8, 2048):
        costs = B.stack_costs(cfg, M, 8, 8.0 * M, 4096.0)
        assert {"experts_up", "experts_down", "route", "carry", "mixer:attention", "mixer:latent_attention_shared_keys"} <= set(costs)
        assert costs["experts_up"][1] == 2.0 * M * 6 * 1536 * 4096
    assert B.hybrid_costs(like[2], 8, 8, 64.0, 4096.0)["experts"][0] > 0
