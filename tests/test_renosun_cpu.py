"""Renosun without a GPU: descriptions, tensor layouts, plan and command line, and the oracle's own laws."""
import pytest
import torch

import oracle_renosun as O
import renosun_cases as R
from saber_engine_b200.cli.main import main as saber
from saber_engine_b200.models import config as MC
from saber_engine_b200.models import stack_config as SC
from saber_engine_b200.models import stack_weights as SW
from saber_engine_b200.plan import launch_plan as LP


def test_description_is_read_from_the_folder(tmp_path):
    cfg = R.CASES["mixed_loop"]
    t = R.tensors(cfg)
    R.write_model(tmp_path / "m", cfg, t)
    c = MC.by_name(str(tmp_path / "m"))
    assert (c.arch, c.vocab, c.width, c.eps, c.embed_scale) == ("Renosun", 203, 104, 1e-5, 3.0)
    assert [r.layer for r in c.runs] == [0, 1, 2, 1, 2, 3] and [r.enter for r in c.runs] == [None, 0, None, 1, None, None]
    assert [(i, n) for i, n, _ in O.Oracle(cfg, t).order()] == [(r.layer, n) for r, n in zip(c.runs, (None, 0, 0, 1, 1, None))]
    back = SW.read_safetensors(tmp_path / "m" / "model.safetensors")
    assert set(back) == set(SW.tensor_shapes(c)) and all(torch.equal(back[k], t[k]) for k in t)
    assert c.param_count() == sum(x.numel() for x in t.values())


def test_unknown_parts_are_refused():
    bad = R.config([R.delta()])
    bad["layers"][0]["type"] = "conv"
    with pytest.raises(ValueError):
        SC.from_json(bad)
    with pytest.raises(KeyError):
        SC.from_json({"architecture": "Other"})
    with pytest.raises(ValueError):
        SC.from_json(R.config([R.delta(heads=3, kv_heads=2)]), name="x")
    with pytest.raises(ValueError):
        SC.from_json(R.config([R.delta()], loop=(0, 2, 1)), name="x")
    odd = R.config([R.latent()])
    odd["layers"][0]["mixer"]["rot"]["dims"] = 4
    with pytest.raises(ValueError):
        SC.from_json(odd, name="x")
    cfg = R.CASES["no_loop"]
    t = R.tensors(cfg)
    t["head"] = t["head"][:-1]
    with pytest.raises(ValueError, match="head"):
        SW.build(SC.from_json(cfg, name="x"), t.__getitem__, torch.float32, "cpu")


@pytest.mark.parametrize("name", list(R.CASES))
def test_packed_linears_hold_every_row_once(name):
    """fp32 layout: the projection's rows and the output's columns give back the tensors they were built from."""
    cfg = R.CASES[name]
    t = R.tensors(cfg, 1)
    c = SC.from_json(cfg, name="x")
    w = SW.build(c, t.__getitem__, torch.float32, "cpu")
    for i, (l, lw) in enumerate(zip(c.layers, w.layers)):
        for seg, n in l.mixer.segments():
            assert torch.equal(lw.proj.w[lw.off[seg]: lw.off[seg] + n, : c.width], t[f"l{i}.mix.{seg}"].float())
        assert torch.equal(lw.out.w[: c.width, : l.mixer.out_features], t[f"l{i}.mix.o"].float())
        if l.mlp:
            gu = lw.proj.w[lw.act_tile0 * 256:].view(-1, 2, 128, lw.proj.K)
            for half, key in enumerate(("gate", "up")):
                assert torch.equal(gu[:, half].reshape(-1, lw.proj.K)[: l.mlp.ff, : c.width], t[f"l{i}.mlp.{key}"].float())
            assert torch.equal(lw.out.w[: c.width, lw.act_k0: lw.act_k0 + l.mlp.ff], t[f"l{i}.mlp.down"].float())
        total = sum(float(x.float().abs().sum()) for k, x in t.items() if k.startswith(f"l{i}.") and x.dim() == 2 and ".conv" not in k
                    and not k.endswith((".uk", ".uv")))
        assert abs(float(lw.proj.w.abs().sum() + lw.out.w.abs().sum()) - total) < 1e-3 * total


def test_block_form_of_the_delta_rule_equals_the_token_form():
    """The identities the prompt kernel rests on: four tokens from the state at their start."""
    g = torch.Generator().manual_seed(0)
    H, D, V, T = 2, 5, 3, 8
    q, k = torch.randn(T, H, D, generator=g).double(), torch.randn(T, H, D, generator=g).double()
    v, beta, dec = torch.randn(T, H, V, generator=g).double(), torch.rand(T, H, generator=g).double(), torch.rand(T, H, generator=g).double()
    want = O.delta_rule(q, k, v, beta, dec)
    S = torch.zeros(H, D, V).double()
    for b in range(0, T, 4):
        G, u, D_ = torch.ones(H).double(), [], []
        for i in range(4):
            t = b + i
            G = G * dec[t]
            D_ = [d * dec[t] for d in D_]
            r = v[t] - G[:, None] * torch.einsum("hdv,hd->hv", S, k[t])
            for j in range(i):
                r = r - (D_[j] * (k[b + j] * k[t]).sum(-1))[:, None] * u[j]
            u.append(beta[t][:, None] * r)
            D_.append(torch.ones(H).double())
            o = G[:, None] * torch.einsum("hdv,hd->hv", S, q[t])
            for j in range(i + 1):
                o = o + (D_[j] * (k[b + j] * q[t]).sum(-1))[:, None] * u[j]
            assert torch.allclose(o, want[t])
        S = S * G[:, None, None] + sum(D_[j][:, None, None] * k[b + j][:, :, None] * u[j][:, None, :] for j in range(4))


def test_oracle_prefix_law():
    """A position's logits do not depend on later tokens."""
    cfg = R.CASES["no_loop"]
    o = O.Oracle(cfg, R.tensors(cfg))
    toks = R.tokens(cfg, 30)
    assert torch.allclose(o.forward(toks)[:17], o.forward(toks[:17]))


def test_plan_registry_and_command_line(capsys):
    man = LP.Manifest(model="renosun-mini", max_ctx=2048, max_seqs=4, decode_batches=(1, 4), decode_widths=(1,), prefill_rows=(64,), budget_mib=12000)
    plan = LP.bind(LP.resolve(man))
    assert plan.kv_blocks >= 2048 // 64 + 1 and plan.ledger.items["recurrent_state_slots"] == 5 * MC.by_name("renosun-mini").slot_bytes()
    man.decode_widths, man.tp = (1, 5), 2
    with pytest.raises(LP.PlanError) as ei:
        LP.resolve(man)
    assert len(ei.value.problems) == 2
    assert saber(["serve", "--model", "renosun", "--random-init", "--print-argv"]) == 0
    assert "--engine-config renosun-mini" in capsys.readouterr().out
    assert saber(["explain", "--model", "renosun-mini"]) == 0
    assert saber(["pack", "build", "--model", "renosun-mini"]) == 2
