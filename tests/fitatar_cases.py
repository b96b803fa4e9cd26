"""Small Fitatar configurations and random weights for the tests (sizes chosen to be awkward)."""
from __future__ import annotations

import torch

from renosun_cases import TOL, engine, error, feed, model, tokens, write_model  # noqa: F401  (any layer-by-layer model)
from saber_engine_b200.models import stack_config as SC
from saber_engine_b200.models import stack_weights as SW


def dense(ff=72):
    return {"kind": "dense", "ff": ff}


def moe(experts=12, top=3, ff=40, groups=4, keep=2, shared=56):
    d = {"kind": "moe", "expert": {"ff": ff}, "router": {"experts": experts, "top": top, "groups": {"count": groups, "keep": keep}}}
    if shared:
        d["shared"] = {"ff": shared}
    return d


def attention(heads=6, kv_heads=2, dim=24, vdim=40, rot=16, base=900.0, factor=3.0, scale=0.3, mlp=None):
    return {"type": "attention", "mlp": mlp, "mixer": dict(heads=heads, kv_heads=kv_heads, dim=dim, vdim=vdim, scale=scale,
                                                           rot={"base": base, "dims": rot, "scaling": {"factor": factor}})}


def latent(heads=3, dim=24, rot_dim=12, vdim=20, kv_rank=56, q_rank=40, base=700.0, scale=0.21, yarn=(2.5, 64, 20.0, 1.5), kv_from=None, mlp=None):
    """yarn: factor, original, fast, slow."""
    m = dict(heads=heads, dim=dim, rot_dim=rot_dim, vdim=vdim, kv_rank=kv_rank, q_rank=q_rank, scale=scale,
             rot={"base": base, "dims": rot_dim, "scaling": dict(zip(("factor", "original", "fast", "slow"), yarn))})
    if kv_from is not None:
        m["kv_from"] = kv_from
    return {"type": "latent_attention", "mixer": m, "mlp": mlp}


def config(layers, width=104, vocab=203, eps=1e-5, scale=3.0, cap=8.0):
    return {"architecture": "Fitatar", "embedding": {"scale": scale}, "layers": layers, "norm": {"eps": eps}, "logit_softcap": cap, "vocab": vocab,
            "width": width}


CASES = {
    "every_kind": config([attention(mlp=dense()), latent(mlp=moe()), attention(heads=4, mlp=moe(experts=8, top=2, groups=2, keep=1, shared=0)),
                          latent(heads=5, vdim=32, kv_from=1, scale=0.3, mlp=moe())]),
    "all_equal_heads": config([attention(heads=3, kv_heads=3, dim=16, vdim=16, rot=16, factor=1.0, mlp=moe(groups=1, keep=1, top=1)),
                               latent(heads=1, dim=16, rot_dim=2, vdim=40, kv_rank=24, q_rank=16, mlp=dense(200))], width=200),
    "no_feed_forwards": config([latent(heads=2), attention(heads=1, kv_heads=1, dim=8, vdim=8, rot=2), latent(heads=3, kv_from=0)], width=72, vocab=97),
    "wide": config([attention(heads=8, kv_heads=1, dim=136, vdim=160, rot=136, mlp=dense(300)),
                    latent(heads=18, dim=72, rot_dim=32, vdim=100, kv_rank=264, q_rank=300, mlp=moe(experts=40, top=6, ff=264, groups=5, keep=3, shared=520)),
                    latent(heads=4, dim=48, rot_dim=32, vdim=136, kv_rank=264, q_rank=130, kv_from=1, mlp=moe(ff=130, shared=250))], width=264),
    "many_heads": config([latent(heads=40, dim=8, rot_dim=4, vdim=8, kv_rank=72, q_rank=64, mlp=dense(40)), attention(heads=66, kv_heads=1, dim=16, vdim=24, rot=8),
                          attention(heads=36, kv_heads=2, dim=32, vdim=32, rot=20, mlp=moe(experts=64, top=9, groups=8, keep=8, shared=8))], width=320, vocab=700),
    "every_expert": config([latent(mlp=moe(experts=6, top=6, groups=3, keep=3, ff=8)), latent(kv_from=0, mlp=moe(experts=3, top=1, groups=3, keep=1, ff=200)),
                            attention(mlp=moe(experts=33, top=5, groups=11, keep=2, ff=72))], width=136),
}


def _chosen_apart(z, f, margin):
    """Whether the expert choice of router logits z [E] would survive a disturbance of `margin` of the largest of them."""
    r = f["router"]
    g, size = r["groups"]["count"], r["experts"] // r["groups"]["count"]
    m = margin * float(z.abs().max())
    best = z.view(g, size).max(1).values
    order = torch.argsort(best, descending=True)
    if r["groups"]["keep"] < g and best[order[r["groups"]["keep"] - 1]] - best[order[r["groups"]["keep"]]] < m:
        return False
    left = torch.cat([z.view(g, size)[i] for i in order[: r["groups"]["keep"]]]).sort(descending=True).values
    return r["top"] == len(left) or bool(left[r["top"] - 1] - left[r["top"]] >= m)


def tensors(cfg: dict, seed: int = 0, code: int = 12) -> dict:
    """Random bf16 tensors by name, norms, sinks and biases away from their trivial values.  Routers read the first `code` coordinates of
    the stream, which no layer writes, and every token's are drawn until its choices are far from ties: they do not change with rounding."""
    g = torch.Generator().manual_seed(seed)
    out = {}
    for name, shape in SW.tensor_shapes(SC.from_json(cfg, name="t")).items():
        leaf = name.rsplit(".", 1)[-1]
        r = torch.randn(shape, generator=g)
        if leaf in ("norm", "norm1", "norm2"):
            t = 1.0 + 0.3 * r
        elif leaf == "sink":
            t = 1.0 + r
        elif leaf == "b":
            t = 0.3 * r
        elif name == "embed":
            t = r
        elif name == "head":
            t = r / 4
        elif leaf == "router":
            t = torch.zeros(shape)
            t[:, :code] = r[:, :code]
        else:
            t = r * (1.3 / shape[-1] ** 0.5)
        if leaf in ("o", "down") or name.endswith("down.b"):
            t[:code] = 0.0
        out[name] = t.to(torch.bfloat16)
    routers = [(out[f"l{i}.mlp.router"].double()[:, :code] * out[f"l{i}.norm2"].double()[:code], l["mlp"]) for i, l in enumerate(cfg["layers"])
               if l["mlp"] and l["mlp"]["kind"] == "moe"]
    for v in range(cfg["vocab"] if routers else 0):
        while not all(_chosen_apart(w @ out["embed"][v, :code].double(), f, 0.02) for w, f in routers):
            out["embed"][v, :code] = torch.randn(code, generator=g).to(torch.bfloat16)
    return out
