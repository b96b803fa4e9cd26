"""Small Renosun configurations and random weights for the tests (sizes chosen to be awkward)."""
from __future__ import annotations

import json
import struct

import torch

from saber_engine_b200.models import stack_config as SC
from saber_engine_b200.models import stack_weights as SW


def delta(heads=3, kv_heads=1, dim=40, vdim=24, conv=4, ff=72, limit=1.5):
    return {"type": "delta", "mixer": dict(heads=heads, kv_heads=kv_heads, dim=dim, vdim=vdim, conv=conv),
            "mlp": None if ff is None else {"kind": "dense", "ff": ff, "limit": limit}}


def latent(heads=3, dim=24, rot_dim=12, vdim=20, kv_rank=56, base=700.0, scale=0.21, ff=72, limit=1.5):
    return {"type": "latent_attention", "mixer": dict(heads=heads, dim=dim, rot_dim=rot_dim, vdim=vdim, kv_rank=kv_rank, scale=scale,
                                                      rot={"base": base, "dims": rot_dim}),
            "mlp": None if ff is None else {"kind": "dense", "ff": ff, "limit": limit}}


def config(layers, width=104, vocab=203, loop=None, eps=1e-5, scale=3.0):
    d = {"architecture": "Renosun", "embedding": {"scale": scale}, "layers": layers, "norm": {"eps": eps}, "vocab": vocab, "width": width}
    if loop is not None:
        d["loop"] = dict(zip(("start", "stop", "times"), loop))
    return d


CASES = {
    "mixed_loop": config([latent(), delta(), latent(heads=5, kv_rank=48), delta(heads=4, kv_heads=4, conv=2)], loop=(1, 3, 2)),
    "loop_first_to_last": config([delta(conv=5), latent(ff=None)], width=72, loop=(0, 2, 3)),
    "loop_once_at_end": config([latent(ff=40), delta(ff=200, limit=0.7, dim=128, vdim=136, heads=2, kv_heads=2)], loop=(1, 2, 1), width=200),
    "no_loop": config([delta(conv=1, heads=6, kv_heads=3, dim=16, vdim=8), latent(heads=1, dim=16, rot_dim=2, vdim=40, kv_rank=24), delta(ff=None, conv=3)],
                      width=136, vocab=97),
    "many_heads": config([latent(heads=40, dim=8, rot_dim=4, vdim=8, kv_rank=72), delta(heads=12, kv_heads=4, dim=72, vdim=40)], width=320, vocab=700),
    "wide_heads": config([latent(heads=18, dim=72, rot_dim=32, vdim=100, kv_rank=264), delta(heads=2, kv_heads=1, dim=200, vdim=64)], width=264, loop=(0, 1, 2)),
}


def tensors(cfg: dict, seed: int = 0) -> dict:
    """Random bf16 tensors by name; norms, decays and biases away from their trivial values."""
    g = torch.Generator().manual_seed(seed)
    out = {}
    for name, shape in SW.tensor_shapes(SC.from_json(cfg, name="t")).items():
        leaf = name.rsplit(".", 1)[-1]
        r = torch.randn(shape, generator=g)
        if leaf in ("norm", "norm1"):
            t = 1.0 + 0.3 * r
        elif leaf == "A_log":
            t = 0.7 * r - 1.0
        elif leaf == "dt_bias":
            t = 0.7 * r - 2.0
        elif leaf == "conv":
            t = 0.5 * r
        elif name == "embed":
            t = r
        elif name == "loop.step":
            t = 0.5 * r
        elif name == "head":
            t = r / 4
        else:
            t = r * (1.3 / shape[-1] ** 0.5)
        out[name] = t.to(torch.bfloat16)
    return out


def tokens(cfg: dict, n: int, seed: int = 0) -> list:
    return torch.randint(0, cfg["vocab"], (n,), generator=torch.Generator().manual_seed(1000 + seed)).tolist()


def write_model(path, cfg: dict, t: dict) -> None:
    path.mkdir(parents=True, exist_ok=True)
    (path / "config.json").write_text(json.dumps(cfg))
    head, blob = {}, b""
    for name, x in t.items():
        raw = x.contiguous().view(torch.uint8).numpy().tobytes()
        head[name] = {"dtype": "BF16", "shape": list(x.shape), "data_offsets": [len(blob), len(blob) + len(raw)]}
        blob += raw
    h = json.dumps(head).encode()
    (path / "model.safetensors").write_bytes(struct.pack("<Q", len(h)) + h + blob)


def model(cfg: dict, t: dict, dtype=torch.float32, max_seqs=4, max_ctx=1024, kv_blocks=None, **kw):
    from saber_engine_b200.models.stack import StackModel
    c = SC.from_json(cfg, name="t")
    return StackModel(c, max_seqs=max_seqs, max_ctx=max_ctx, kv_blocks=kv_blocks, dtype=dtype, weights=SW.build(c, t.__getitem__, dtype, "cuda"), **kw)


def engine(cfg: dict, t: dict, dtype=torch.float32, rungs=(16, 64, 256, 1024), capture=False, **kw):
    from saber_engine_b200.runtime.trace_run import TraceEngine
    return TraceEngine(model(cfg, t, dtype, **kw), prefill_rungs=rungs, capture=capture)


def feed(eng, rid, toks, cuts) -> torch.Tensor:
    """One request in portions of the given sizes (the last size repeats); logits of every position."""
    out, at, k = [], 0, 0
    while at < len(toks):
        n = min(cuts[min(k, len(cuts) - 1)], len(toks) - at)
        out.append(eng.step([(rid, toks[at:at + n])])[0])
        at, k = at + n, k + 1
    eng.end(rid)
    return torch.cat(out)


def error(got, want) -> float:
    """Largest difference of a position's logits (mean taken off) over the root mean square of all logits."""
    d = got.double() - want.double()
    d = d - d.mean(-1, keepdim=True)
    return float(d.pow(2).mean(-1).sqrt().max() / want.double().pow(2).mean().sqrt())


TOL = {torch.float32: 2e-5, torch.bfloat16: 0.06}
