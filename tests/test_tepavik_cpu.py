"""Tepavik without a GPU: descriptions, tensor layouts, plan and command line, and the oracle's own laws."""
import pytest
import torch

import oracle_tepavik as O
import tepavik_cases as R
from saber_engine_b200.cli.main import main as saber
from saber_engine_b200.models import config as MC
from saber_engine_b200.models import stack_config as SC
from saber_engine_b200.models import stack_weights as SW
from saber_engine_b200.plan import launch_plan as LP


def test_description_is_read_from_the_folder(tmp_path):
    cfg = R.CASES["every_kind"]
    t = R.tensors(cfg)
    R.write_model(tmp_path / "m", cfg, t)
    c = MC.by_name(str(tmp_path / "m"))
    assert (c.arch, c.vocab, c.width, c.eps, c.parallel, c.norm_offset) == ("Tepavik", 203, 104, 1e-5, False, 1.0)
    assert [type(l.mixer).__name__ for l in c.layers] == ["OuterMixer", "GroupedMixer", "OuterMixer", "GroupedMixer"]
    assert [c.pages_of(r) for r in c.runs] == [0, 1, 2, 1]
    assert c.layers[2].mixer.decay == (0.5, 0.93, 0.998) and c.layers[3].mixer.chunk == 96
    back = SW.read_safetensors(tmp_path / "m" / "model.safetensors")
    assert set(back) == set(SW.tensor_shapes(c)) and all(torch.equal(back[k], t[k]) for k in t)
    assert c.param_count() == sum(x.numel() for x in t.values())
    # only the layer with keys of its own holds pages
    assert c.page_token_bytes() == 2 * 2 * (64 + 64)


def test_unknown_parts_are_refused():
    bad = R.config([R.lightning()])
    bad["layers"][0]["type"] = "conv"
    with pytest.raises(ValueError):
        SC.from_json(bad)
    for layers in ([R.mamba(heads=6, groups=4)], [R.mamba(heads=5, groups=1, norm_groups=3)], [R.lightning(heads=4)], [R.attention(heads=3)],
                   [R.attention(kv_from=0)], [R.mamba(), R.attention(kv_from=0)], [R.attention(), R.attention(dim=16, kv_from=0)],
                   [R.attention(), R.attention(kv_from=0), R.attention(kv_from=1)]):
        with pytest.raises(ValueError):
            SC.from_json(R.config(layers), name="x")
    cfg = R.CASES["equal_heads"]
    t = R.tensors(cfg)
    t["l1.mix.conv"] = t["l1.mix.conv"][:-1]
    with pytest.raises(ValueError, match="conv"):
        SW.build(SC.from_json(cfg, name="x"), t.__getitem__, torch.float32, "cpu")


@pytest.mark.parametrize("name", list(R.CASES))
def test_packed_linears_hold_every_row_once(name):
    """fp32 layout: projection rows, biases and output columns give back the tensors they were built from."""
    cfg = R.CASES[name]
    t = R.tensors(cfg, 1)
    c = SC.from_json(cfg, name="x")
    w = SW.build(c, t.__getitem__, torch.float32, "cpu")
    for i, (l, lw) in enumerate(zip(c.layers, w.layers)):
        p, rows = f"l{i}.mix.", dict(l.mixer.segments())
        for seg, tensor, first in l.mixer.sources():
            assert torch.equal(lw.proj.w[lw.off[seg]: lw.off[seg] + rows[seg], : c.width], t[p + tensor][first: first + rows[seg]].float())
            if l.mixer.biases():
                assert torch.equal(lw.bias[lw.off[seg]: lw.off[seg] + rows[seg]], t[f"{p}{tensor}.b"].float())
        assert torch.equal(lw.out.w[: c.width, : l.mixer.out_features], t[p + "o"].float())
        assert torch.equal(lw.norm, 1 + t[f"l{i}.norm1"].float())
        if l.mlp:
            assert torch.equal(lw.up.w[: l.mlp.ff, : c.width], t[f"l{i}.mlp.up"].float()) and torch.equal(lw.norm2, 1 + t[f"l{i}.norm2"].float())
            assert torch.equal(lw.down.w[: c.width, : l.mlp.ff], t[f"l{i}.mlp.down"].float())
        else:
            assert lw.up is None and f"l{i}.norm2" not in t
        total = sum(float(x.float().abs().sum()) for k, x in t.items() if k.startswith(f"l{i}.") and x.dim() == 2 and ".conv" not in k)
        assert abs(float(sum(x.w.abs().sum() for x in (lw.proj, lw.out, lw.up, lw.down) if x is not None)) - total) < 1e-3 * total


def test_mamba_rows_and_channels():
    """One packed tensor: gate | values | keys | queries | steps; the convolution's channels follow the values-first order."""
    cfg = R.config([R.mamba(heads=2, groups=1, state=3, vdim=4, conv=2, norm_groups=1, ff=None)], width=8)
    t = R.tensors(cfg)
    t["l0.mix.in"] = torch.arange(24.0)[:, None].expand(-1, 8).bfloat16()
    t["l0.mix.conv"] = torch.arange(14.0)[:, None].expand(-1, 2).bfloat16()
    t["l0.mix.conv.b"] = torch.arange(14.0).bfloat16()
    lw = SW.build(SC.from_json(cfg, name="x"), t.__getitem__, torch.float32, "cpu").layers[0]
    col = lambda seg, n: lw.proj.w[lw.off[seg]: lw.off[seg] + n, 0].tolist()     # noqa: E731
    assert (col("g", 8), col("v", 8), col("k", 3), col("q", 3), col("dt", 2)) == \
        ([*range(8)], [*range(8, 16)], [16, 17, 18], [19, 20, 21], [22, 23])
    assert lw.extra["conv_b"].tolist() == [11, 12, 13, 8, 9, 10, *range(8)] and lw.extra["conv"][:, 1].tolist() == lw.extra["conv_b"].tolist()


def _random_outer(T=128, H=2, N=5, V=3, strong=False):
    g = torch.Generator().manual_seed(0)
    q, k, v = (torch.randn(T, H, n, generator=g).double() for n in (N, N, V))
    la = -torch.rand(T, H, generator=g).double() * (12 if strong else 0.3)
    return q, k, v, la, O.decayed_outer_products(q, k, v, torch.exp(la))


@pytest.mark.parametrize("strong", [False, True])
def test_chunk_form_of_the_decayed_outer_products(strong):
    """The identity the chunk kernels rest on: products inside a chunk of 64, the state at its start for the rest.  Decays
    are exponentials of sums over the tokens between, never quotients."""
    q, k, v, la, want = _random_outer(strong=strong)
    S = torch.zeros(2, 5, 3).double()
    for c in range(0, 128, 64):
        L, Q, K, Vv = (x[c:c + 64] for x in (la, q, k, v))
        cum = torch.cumsum(L, 0)
        D = torch.exp(cum[:, None] - cum[None]).masked_fill(torch.ones(64, 64).triu(1).bool()[..., None], 0.0)
        P = torch.einsum("ihn,jhn->ijh", Q, K) * D
        o = torch.einsum("ijh,jhv->ihv", P, Vv) + torch.exp(cum)[..., None] * torch.einsum("ihn,hnv->ihv", Q, S)
        assert torch.allclose(o, want[c:c + 64], rtol=1e-9, atol=1e-11)
        S = torch.exp(cum[-1])[:, None, None] * S + torch.einsum("jhn,jhv->hnv", K * torch.exp(cum[-1] - cum)[..., None], Vv)


def test_oracle_laws():
    """A position's logits depend on earlier tokens only, and an attention layer's on its own chunk."""
    cfg = R.CASES["every_kind"]
    o = O.Oracle(cfg, R.tensors(cfg))
    toks = R.tokens(cfg, 60)
    assert torch.allclose(o.forward(toks)[:37], o.forward(toks[:37]))
    one = R.config([R.attention(chunk=20)])
    o = O.Oracle(one, R.tensors(one))
    a, b = R.tokens(one, 45), R.tokens(one, 45, seed=1)
    assert torch.allclose(o.forward(a[:40] + b[40:])[40:], o.forward(b)[40:])
    assert not torch.allclose(o.forward(a[:41] + b[41:])[41:], o.forward(b)[41:])


def test_plan_registry_and_command_line(capsys):
    man = LP.Manifest(model="tepavik-mini", max_ctx=2048, max_seqs=4, decode_batches=(1, 4), decode_widths=(1,), prefill_rows=(64,), budget_mib=12000)
    plan = LP.bind(LP.resolve(man))
    assert plan.kv_blocks >= 2048 // 64 + 1 and plan.ledger.items["recurrent_state_slots"] == 5 * MC.by_name("tepavik-mini").slot_bytes()
    man.decode_widths = (1, 5)
    with pytest.raises(LP.PlanError):
        LP.resolve(man)
    assert saber(["serve", "--model", "tepavik", "--random-init", "--print-argv"]) == 0
    assert "--engine-config tepavik-mini" in capsys.readouterr().out
    assert saber(["explain", "--model", "tepavik-mini"]) == 0
