"""Small Sofunex configurations and random weights for the tests (sizes chosen to be awkward)."""
from __future__ import annotations

import torch

from renosun_cases import TOL, error, feed, tokens, write_model  # noqa: F401  (any layer-by-layer model)
from saber_engine_b200.models import stack_config as SC
from saber_engine_b200.models import stack_weights as SW


def dense(ff=72):
    return {"kind": "dense", "ff": ff}


def moe(experts=12, top=3, ff=40, groups=(4, 2), shared=56, scale=1.7):
    d = {"kind": "moe", "expert": {"ff": ff}, "router": {"experts": experts, "top": top, "scale": scale}}
    if groups:
        d["router"]["groups"] = dict(zip(("count", "keep"), groups))
    if shared:
        d["shared"] = {"ff": shared}
    return d


def layer(heads=6, kv_heads=2, dim=24, vdim=40, conv=3, window=50, rot=16, base=900.0, factor=3.0, scale=0.3, delta_heads=3, delta_dim=20,
          left=0.7, right=0.4, mlp=None):
    r = {"base": base, "dims": rot}
    if factor:
        r["scaling"] = {"factor": factor}
    a = dict(heads=heads, kv_heads=kv_heads, dim=dim, vdim=vdim, conv=conv, mask={"size": window}, rot=r, scale=scale)
    return {"type": "parallel", "mlp": mlp, "mixer": {"left": a, "left_scale": left, "right": {"heads": delta_heads, "dim": delta_dim}, "right_scale": right}}


def config(layers, width=104, vocab=203, loop=None, eps=1e-5, scale=3.0, mult=0.6):
    d = {"architecture": "Sofunex", "embedding": {"scale": scale}, "layers": layers, "norm": {"eps": eps}, "residual_mult": mult, "vocab": vocab, "width": width}
    if loop is not None:
        d["loop"] = dict(zip(("start", "stop", "times"), loop))
    return d


CASES = {
    "every_kind": config([layer(mlp=dense()), layer(heads=4, kv_heads=4, window=9, conv=4, mlp=moe()), layer(delta_heads=5, delta_dim=33, mlp=moe(8, 2, groups=(2, 1), shared=0)),
                          layer(heads=5, kv_heads=1, vdim=32, conv=2, window=70, scale=0.2, left=0.3, right=0.9)], loop=(1, 3, 2)),
    "loop_first_to_last": config([layer(window=1, mlp=dense(200)), layer(conv=1, mlp=moe(6, 1, groups=None))], width=72, loop=(0, 2, 3)),
    "no_loop_all_ones": config([layer(heads=1, kv_heads=1, dim=8, vdim=8, conv=1, rot=2, factor=None, scale=1.0, delta_heads=1, delta_dim=8, left=1.0, right=1.0, mlp=dense(8))],
                               vocab=97, mult=1.0, scale=1.0),
    "wide": config([layer(heads=8, kv_heads=1, dim=136, vdim=160, rot=136, window=64, delta_heads=2, delta_dim=130, mlp=dense(300)),
                    layer(heads=3, kv_heads=3, dim=72, vdim=100, rot=40, window=128, delta_heads=4, delta_dim=72, mlp=moe(40, 6, 264, (5, 3), 520))], width=264, loop=(1, 2, 2)),
    "many_heads": config([layer(heads=36, kv_heads=2, dim=16, vdim=24, rot=8, window=33, delta_heads=40, delta_dim=8, mlp=moe(64, 9, 24, (8, 8), 8)),
                          layer(heads=66, kv_heads=1, dim=16, vdim=16, rot=16, conv=5, window=65, delta_heads=11, delta_dim=16)], width=320, vocab=700),
    "groups_of_one": config([layer(window=1000, mlp=moe(7, 4, 130, (7, 4), 249)), layer(mlp=moe(6, 6, 8, (3, 3), 0, scale=0.5))], width=91, loop=(1, 2, 1)),
}


def shapes(cfg: dict) -> dict:
    """The size that a description leaves to its tensors: values that a layer's decays pass through."""
    return {f"l{i}.mix.right.w1": ((9, 24, 1, 70)[i % 4], cfg["width"]) for i in range(len(cfg["layers"]))}


def describe(cfg: dict) -> SC.StackConfig:
    return SC.from_json(cfg, name="t", shapes=shapes(cfg))


def _choice(z, corr, r):
    """(chosen experts, smallest distance to another choice) of router logits z [E]."""
    c, g = torch.sigmoid(z) + corr, r.get("groups") or {"count": 1, "keep": 1}
    n, gap = len(c) // g["count"], 9.0
    strength = c.view(g["count"], n).sort(-1, descending=True).values[:, :2].sum(-1)
    order = strength.argsort(descending=True)
    if g["keep"] < g["count"]:
        gap = float(strength[order[g["keep"] - 1]] - strength[order[g["keep"]]]) / 2
    left = [e for k in order[: g["keep"]].tolist() for e in range(k * n, (k + 1) * n)]
    best = sorted(left, key=lambda e: -float(c[e]))
    if r["top"] < len(best):
        gap = min(gap, float(c[best[r["top"] - 1]] - c[best[r["top"]]]))
    return set(best[: r["top"]]), gap


def tensors(cfg: dict, seed: int = 0, code: int = 10) -> dict:
    """Random bf16 tensors by name, norms, biases, blends and corrections away from their trivial values.  Routers read the first `code`
    coordinates of the stream, which no layer writes, and every token's are drawn until its choices are the same, and far from ties, at every size
    that the stream's other coordinates may give their norm: they do not change with rounding."""
    g = torch.Generator().manual_seed(seed)
    out = {}
    for name, shape in SW.tensor_shapes(describe(cfg)).items():
        leaf = name.rsplit(".", 1)[-1]
        r = torch.randn(shape, generator=g)
        if leaf in ("norm", "norm1", "norm2", "norm1b", "norm2b"):
            t = 1.0 + 0.3 * r
        elif leaf == "shift":
            t = torch.rand(shape, generator=g)
        elif leaf == "b":
            t = 0.3 * r
        elif leaf == "w0":
            t = 1.5 * r - 1.0
        elif leaf == "conv":
            t = 0.5 * r
        elif leaf == "correction":
            t = 0.3 * r
        elif name == "embed":
            t = r
        elif name == "loop.step":
            t = 0.5 * r
        elif name == "head":
            t = r / 4
        elif leaf == "router":
            t = torch.zeros(shape)
            t[:, :code] = r[:, :code]
        else:
            t = r * (1.3 / shape[-1] ** 0.5)
        if leaf in ("norm1b", "norm2b"):
            t[:code] = 0.0
        elif name == "loop.step":
            t[:, :code] = 0.0
        out[name] = t.to(torch.bfloat16)
    routers = [(out[f"l{i}.mlp.router"].double()[:, :code] * out[f"l{i}.norm2"].double()[:code], out[f"l{i}.mlp.correction"].double(), l["mlp"]["router"])
               for i, l in enumerate(cfg["layers"]) if l["mlp"] and l["mlp"]["kind"] == "moe"]

    def settled(v) -> bool:
        for w, corr, r in routers:
            z, chosen = w @ out["embed"][v, :code].double(), None
            for c in (0.5, 0.65, 0.8, 1.0, 1.3):                       # (the scale of the embedding over the root mean square of the stream)
                ids, gap = _choice(c * z, corr, r)
                if gap < 0.012 or (chosen is not None and ids != chosen):
                    return False
                chosen = ids
        return True
    for v in range(cfg["vocab"] if routers else 0):
        for _ in range(3000):
            if settled(v):
                break
            out["embed"][v, :code] = torch.randn(code, generator=g).to(torch.bfloat16)
        else:
            raise AssertionError(f"no settled choice for token {v}")
    return out


def model(cfg: dict, t: dict, dtype=torch.float32, max_seqs=4, max_ctx=1024, kv_blocks=None, **kw):
    from saber_engine_b200.models.stack import StackModel
    c = describe(cfg)
    return StackModel(c, max_seqs=max_seqs, max_ctx=max_ctx, kv_blocks=kv_blocks, dtype=dtype, weights=SW.build(c, t.__getitem__, dtype, "cuda"), **kw)


def engine(cfg: dict, t: dict, dtype=torch.float32, rungs=(16, 64, 256, 1024), capture=False, **kw):
    from saber_engine_b200.runtime.trace_run import TraceEngine
    return TraceEngine(model(cfg, t, dtype, **kw), prefill_rungs=rungs, capture=capture)
