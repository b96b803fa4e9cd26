"""Small Tepavik configurations and random weights for the tests (sizes chosen to be awkward)."""
from __future__ import annotations

import torch

from renosun_cases import TOL, engine, error, feed, model, tokens, write_model  # noqa: F401  (any layer-by-layer model)
from saber_engine_b200.models import stack_config as SC
from saber_engine_b200.models import stack_weights as SW


def _layer(kind, mixer, ff):
    return {"type": kind, "mixer": mixer, "mlp": None if ff is None else {"kind": "dense", "ff": ff}}


def mamba(heads=6, groups=3, state=24, vdim=20, conv=4, norm_groups=2, ff=72):
    return _layer("mamba2", dict(heads=heads, groups=groups, state=state, vdim=vdim, conv=conv, norm_groups=norm_groups), ff)


def lightning(heads=3, dim=40, vdim=24, decay=(0.5, 0.93, 0.998), ff=72):
    return _layer("lightning", dict(heads=heads, dim=dim, vdim=vdim, decay=list(decay)), ff)


def attention(heads=6, kv_heads=2, dim=24, vdim=40, chunk=50, scale=0.3, softcap=6.0, kv_from=None, ff=72):
    m = dict(heads=heads, kv_heads=kv_heads, dim=dim, vdim=vdim, mask={"size": chunk}, scale=scale, softcap=softcap)
    if kv_from is not None:
        m["kv_from"] = kv_from
    return _layer("attention", m, ff)


def config(layers, width=104, vocab=203, eps=1e-5):
    return {"architecture": "Tepavik", "layers": layers, "norm": {"eps": eps}, "vocab": vocab, "width": width}


CASES = {
    "every_kind": config([mamba(), attention(), lightning(), attention(kv_from=1, chunk=96, scale=0.2)]),
    "equal_heads": config([attention(heads=2, kv_heads=2, dim=16, vdim=16, chunk=128, ff=40), mamba(heads=4, groups=4, norm_groups=4, conv=2),
                           lightning(heads=1, dim=64, vdim=72, decay=(0.99,), ff=200)], width=200),
    "one_of_each_size": config([mamba(heads=5, groups=1, state=8, vdim=8, conv=1, norm_groups=1, ff=None), lightning(ff=None),
                                attention(heads=1, kv_heads=1, dim=8, vdim=8, chunk=7, ff=None)], width=72, vocab=97),
    "wide_heads": config([attention(heads=8, kv_heads=1, dim=136, vdim=160, chunk=1000, ff=300), mamba(heads=3, groups=1, state=136, vdim=64, norm_groups=3, ff=130),
                          attention(heads=5, kv_heads=1, dim=136, vdim=160, chunk=80, kv_from=0, ff=300)], width=264),
    "many_query_heads": config([attention(heads=36, kv_heads=2, dim=32, vdim=32, chunk=65), attention(heads=66, kv_heads=1, dim=16, vdim=24, chunk=300),
                                lightning(heads=7, dim=72, vdim=40, decay=(0.0, 0.2, 0.5, 0.8, 0.95, 0.999, 1.0))], width=320, vocab=700),
    "two_readers": config([attention(chunk=64), attention(chunk=33, kv_from=0, scale=0.5), mamba(conv=5, heads=8, groups=2, vdim=12, norm_groups=3),
                           attention(chunk=20, kv_heads=3, softcap=2.0), attention(heads=3, chunk=500, kv_heads=3, kv_from=3)], width=136),
}


def tensors(cfg: dict, seed: int = 0) -> dict:
    """Random bf16 tensors by name; norms, decays, biases and skips away from their trivial values."""
    g = torch.Generator().manual_seed(seed)
    out = {}
    for name, shape in SW.tensor_shapes(SC.from_json(cfg, name="t")).items():
        leaf = name.rsplit(".", 1)[-1]
        r = torch.randn(shape, generator=g)
        if leaf == "norm" and ".mix." in name:
            t = 1.0 + 0.3 * r
        elif leaf in ("norm", "norm1", "norm2", "b"):
            t = 0.3 * r
        elif leaf == "A_log":
            t = 0.8 * r - 0.5
        elif leaf == "dt_bias":
            t = 0.7 * r - 1.5
        elif leaf == "D":
            t = r
        elif leaf == "conv":
            t = 0.5 * r
        elif name == "embed":
            t = 2.0 * r
        elif name == "head":
            t = r / 4
        else:
            t = r * (1.3 / shape[-1] ** 0.5)
        out[name] = t.to(torch.bfloat16)
    return out
