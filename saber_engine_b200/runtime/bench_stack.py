"""Throughput of a layer-by-layer model beside its closest relatives at equal layer sizes: Renosun beside the int4
hybrid decoder, Tepavik beside Renosun and the hybrid decoder, Fitatar beside Tepavik (grouped-query attention), Renosun (latent
attention) and the hybrid decoder with a mixture of experts, Sofunex beside Fitatar (grouped-query attention, experts), Renosun (delta
rule) and the hybrid decoder with a mixture of experts.

Prefill: a cold prompt in portions of one rung (device-timed).  Decode: `streams` sequences at the prompt's length,
one row each (no drafter on either side).  Then every group of launches of one step on its own: the group's
launches between two events after an L2 flush (a write of 256 MB), the median over repetitions, and the fraction
of its roofline: the slower of algorithmic bytes / measured copy bandwidth and FLOPs / measured bf16 GEMM rate.
"""
from __future__ import annotations

import json
import os
import statistics

import torch

from ..models import config as C
from ..models.hybrid import HybridModel
from ..models.stack import StackModel
from ..models.stack_config import (ChannelDeltaMixer, ClampedGlu, DeltaMixer, Gelu, GroupedMixer, ExpertMix, LatentMixer, LayerSpec, OuterMixer, Rotation,
                                   SideBySideMixer, SquaredRelu, StackConfig)
from ..models.step import SeqStep, run_bucket

SIZES = ("renosun-2k", "renosun-4k", "renosun-5k", "tepavik-2k", "tepavik-4k", "tepavik-5k", "fitatar-2k", "fitatar-4k", "fitatar-5k", "sofunex-2k",
         "sofunex-4k", "sofunex-5k")


def peaks() -> tuple:
    path = os.path.join(os.path.dirname(os.path.abspath(__file__)), "..", "..", "MEASURED_PEAKS.json")
    if os.path.exists(path):
        d = json.load(open(path))
        return d["hbm_gbs"] * 1e9, d["bf16_tflops"] * 1e12
    return 6.65e12, 1.59e15


def like_models(cfg: StackConfig) -> list:
    makers = {"Renosun": [like_hybrid], "Tepavik": [like_renosun, like_hybrid], "Fitatar": [like_tepavik, like_renosun, like_hybrid],
              "Sofunex": [like_fitatar, like_renosun, like_hybrid]}[cfg.arch]
    return [make(cfg) for make in makers]


def experts_of(cfg: StackConfig):
    return next((l.mlp for l in cfg.layers if isinstance(l.mlp, ExpertMix)), None)


def mixer_of(cfg: StackConfig, *kinds):
    return next((m for m in cfg.mixers() if isinstance(m, kinds)), None)


def like_fitatar(cfg: StackConfig) -> StackConfig:
    """Fitatar with the same attention heads, a layer for every layer run, and feed-forwards of the same bytes: its matrices are two, half as
    wide again, where the other has three."""
    a, layers = mixer_of(cfg, GroupedMixer), []
    m = GroupedMixer(a.heads, a.kv_heads, a.dim, a.vdim, a.scale, qk_norm=False, bias=False, rot=a.rot, sink=True, gate=True)
    for r in cfg.runs:
        f = cfg.layers[r.layer].mlp
        layers.append(LayerSpec(m, ExpertMix(f.experts, f.top, f.ff * 3 // 2, f.groups, f.keep, f.shared * 3 // 2) if isinstance(f, ExpertMix) else Gelu(f.ff * 3 // 2)))
    return StackConfig(f"fitatar-like-{cfg.name}", "Fitatar", vocab=cfg.vocab, width=cfg.width, layers=tuple(layers), two_norms=True, max_ctx=cfg.max_ctx)


def like_tepavik(cfg: StackConfig) -> StackConfig:
    """Tepavik attention layers only, over every earlier key, with the same heads; the feed-forward as wide as what a token meets."""
    a = next(l.mixer for l in cfg.layers if isinstance(l.mixer, GroupedMixer))
    f = experts_of(cfg)
    l = LayerSpec(GroupedMixer(a.heads, a.kv_heads, a.dim, a.vdim, a.scale, 30.0, 0), SquaredRelu(f.top * f.ff + f.shared))
    return StackConfig(f"tepavik-like-{cfg.name}", "Tepavik", vocab=cfg.vocab, width=cfg.width, layers=(l,) * len(cfg.layers), parallel=False,
                       norm_offset=1.0, max_ctx=cfg.max_ctx)


def like_renosun(cfg: StackConfig) -> StackConfig:
    """Renosun with the same width, vocabulary, layers of each sort and attention heads; its gated feed-forward has three
    matrices where the other has two."""
    a = mixer_of(cfg, GroupedMixer)
    if cfg.arch == "Sofunex":                                  # delta layers only, as many key heads as value heads; gated units on both sides
        c = mixer_of(cfg, ChannelDeltaMixer)
        d = LayerSpec(DeltaMixer(c.heads, c.heads, c.dim, c.dim, 4), ClampedGlu(cfg.layers[0].mlp.ff, 7.0))
        return StackConfig(f"renosun-like-{cfg.name}", "Renosun", vocab=cfg.vocab, width=cfg.width, layers=(d,) * len(cfg.runs), max_ctx=cfg.max_ctx)
    mlp = ClampedGlu(cfg.layers[0].mlp.ff * 2 // 3 // 128 * 128, 7.0)
    d = LayerSpec(DeltaMixer(a.heads, a.heads // 2, 128, 128, 4), mlp)
    la = LayerSpec(LatentMixer(a.heads, 128, 64, 128, 512, 192 ** -0.5, Rotation(1e6, 64)), mlp)
    return StackConfig(f"renosun-like-{cfg.name}", "Renosun", vocab=cfg.vocab, width=cfg.width,
                       layers=tuple(la if isinstance(l.mixer, LatentMixer if cfg.arch == "Fitatar" else GroupedMixer) else d for l in cfg.layers),
                       max_ctx=cfg.max_ctx)


def like_hybrid(cfg: StackConfig) -> C.HybridConfig:
    """The hybrid decoder with the same width, feed-forward or experts, recurrent heads of 128 and number of layer runs; its gated GQA
    attention has the same query width in heads of 256 and a quarter as many key heads."""
    a, d = mixer_of(cfg, LatentMixer, GroupedMixer), mixer_of(cfg, DeltaMixer)
    kh, vh, ff = (d.kv_heads, d.heads, cfg.layers[0].mlp.ff) if d else (a.heads // 2, a.heads, cfg.layers[0].mlp.ff * 2 // 3 // 256 * 256)
    nq, f = max(4, a.heads * a.dim // 256), experts_of(cfg)
    return C.HybridConfig(name=f"hybrid-like-{cfg.name}", n_layers=len(cfg.runs), hidden=cfg.width, n_q_heads=nq, n_kv_heads=max(1, nq // 4),
                          head_dim=256, ffn_inter=ff, vocab=cfg.vocab, gdn_k_heads=kh, gdn_v_heads=vh,
                          gdn_head_dim=128, max_ctx=cfg.max_ctx, moe=None if f is None else C.MoEConfig(f.experts, f.top, f.ff, f.shared, True))


def mixer_name(m) -> str:
    if isinstance(m, OuterMixer):
        return "state_space" if m.decay is None else "linear_attention"
    return m.kind + ("_shared_keys" if m.kv_from is not None else "")


def _groups(model, b) -> dict:
    """Launch ranges per group, by tag.  A layer-by-layer model: (group, mixer) of every layer run, "mixer" its kernels."""
    tags = b.program.tags()
    out = {}
    if isinstance(model, StackModel):
        for i, t in enumerate(tags):
            part = t.split(".")
            if part[0][0] == "R" and part[0][1:].isdigit() and part[-1] != "digest":
                spec = model.cfg.layers[int(part[1][1:])]
                alone = ("loop_in", "carry", "route", "experts_up", "experts_down", "join", "end", "up", "down")
                label = part[2] if part[2] in ("project", "out", *alone) else "mixer"
                if isinstance(spec.mixer, SideBySideMixer):
                    tail = "+experts" if isinstance(spec.mlp, ExpertMix) and label in ("up", "down", "end") else ""
                    out.setdefault(f"mixer:{part[2]}" if label == "mixer" else label + tail, []).append((i, i + 1))
                    continue
                key = label if label in alone else f"{label}:{mixer_name(spec.mixer)}" + ("+experts" if label != "mixer" and isinstance(spec.mlp, ExpertMix) else "")
                out.setdefault(key, []).append((i, i + 1))
            elif t == "lm_head":
                out["lm_head"] = [(i, i + 1)]
        return out
    layers = sorted({int(t[1:].split(".")[0]) for t in tags if t[0] == "L" and t[1].isdigit()})
    span = lambda li, keys: [i for i, t in enumerate(tags) if t.startswith(f"L{li}.") and any(k in t for k in keys)]   # noqa: E731
    moe = model.cfg.moe is not None
    spec = {"delta": ("gdn.conv", "gdn.rec", "gdn.norm", "gdn.step"), "attention": ("attn.rope", "attn.core", "attn.gate", "attn.quant"),
            "linears": ("in_norm", "in_proj", "attn.qkv", "out_proj", "o_proj", "post_norm", *(() if moe else ("mlp",)))}
    if moe:
        spec["experts"] = (".moe.",)
    for g, keys in spec.items():
        out[g] = []
        for li in layers:
            idx = span(li, keys)
            runs = []
            for i in idx:
                if runs and runs[-1][1] == i:
                    runs[-1][1] = i + 1
                else:
                    runs.append([i, i + 1])
            if runs:
                out[g].append([tuple(r) for r in runs])
    out["linears"] = [r for r in out["linears"] if r]
    return out


def _time(model, b, ranges, flush, reps: int = 7) -> float:
    """Median microseconds of the launches in `ranges`."""
    st, res = model.stream, []
    with torch.cuda.stream(st):
        for k in range(reps + 2):
            flush.zero_()
            tot = []
            for lo, hi in ranges:
                e0, e1 = torch.cuda.Event(enable_timing=True), torch.cuda.Event(enable_timing=True)
                e0.record(st)
                b.program.run(st, lo, hi)
                e1.record(st)
                tot.append((e0, e1))
            st.synchronize()
            if k >= 2:
                res.append(sum(a.elapsed_time(c) for a, c in tot) * 1e3)
    return statistics.median(res)


def _roof(nbytes: float, flops: float) -> float:
    hbm, mm = peaks()
    return max(nbytes / hbm, flops / mm) * 1e6


def stack_costs(cfg: StackConfig, M: int, nseq: int, ctx_pairs: float, ctx_tokens: float) -> dict:
    """Algorithmic (bytes, FLOPs) per launch group.  ctx_pairs: visible (row, key) pairs; ctx_tokens: keys read."""
    if cfg.post_norms:
        return joined_costs(cfg, M, nseq, ctx_pairs, ctx_tokens)
    W, head_rows = cfg.width, min(M, 8)
    out = {"loop_in": (4 * cfg.width ** 2 + M * 10 * cfg.width, 4.0 * M * cfg.width ** 2)}
    for l in cfg.layers:
        m, ff, f = l.mixer, l.mlp.inner, l.mlp
        name, mix = mixer_name(m), isinstance(f, ExpertMix)
        tail = "+experts" if mix else ""
        segs = sum(n for _, n in m.segments()) + (f.experts if mix else 0)
        up_rows = ff * (2 if isinstance(f, ClampedGlu) else 1)
        n, k = (segs + up_rows, m.out_features + ff) if cfg.parallel else (segs, m.out_features)
        ops = 2 if cfg.two_norms else 1                        # operands of the stream
        out[f"project:{name}{tail}"] = (2 * n * W + M * (2 * W * ops + 4 * segs + (2 * ff if cfg.parallel else 0)), 2.0 * M * n * W)
        out[f"out:{name}{tail}"] = (2 * k * W + M * (2 * k + 8 * W + 2 * W * ops + (2 * f.top * W if mix else 0)), 2.0 * M * k * W)
        if mix:
            routes, met = M * f.top, f.experts * (1 - (1 - f.top / f.experts) ** M)       # experts that some token chooses, choices alike
            out["route"] = (M * (4 * f.experts + 16 * f.top), 0.0)
            out["experts_up"] = (2 * met * f.ff * W + M * 2 * W + routes * 2 * f.ff, 2.0 * routes * f.ff * W)
            out["experts_down"] = (2 * met * f.ff * W + routes * 2 * (f.ff + W), 2.0 * routes * f.ff * W)
        if m.q_rank:
            out["carry"] = (2 * m.q_rank * m.query_rows + M * (2 * m.q_rank + 4 * m.query_rows), 2.0 * M * m.q_rank * m.query_rows)
        out["up"] = (2 * ff * W + M * (2 * W + 2 * ff), 2.0 * M * ff * W)
        out["down"] = (2 * ff * W + M * (2 * ff + 8 * W + 2 * W), 2.0 * M * ff * W)
        if isinstance(m, (DeltaMixer, OuterMixer)):
            out[f"mixer:{name}"] = (2 * 4 * nseq * m.heads * m.dim * m.vdim + M * (4 * segs + 2 * m.out_features),
                                    M * m.heads * m.dim * m.vdim * (8.0 if isinstance(m, DeltaMixer) else 4.0))
        elif isinstance(m, GroupedMixer):
            out[f"mixer:{name}"] = (2 * ctx_tokens * m.kv_heads * (m.dim + m.vdim) + M * (4 * segs + 2 * m.out_features),
                                    ctx_pairs * 2.0 * m.heads * (m.dim + m.vdim))
        else:
            pair = 2.0 * m.heads * (m.dim + m.rot_dim + m.vdim)
            carry = 2.0 * ctx_tokens * m.heads * (m.dim + m.vdim) * m.kv_rank if M > 64 else 2.0 * M * m.heads * (m.dim + m.vdim) * m.kv_rank
            if M <= 64:
                pair = 2.0 * m.heads * (2 * m.kv_rank + m.rot_dim)
            out[f"mixer:{name}"] = (2 * ctx_tokens * (m.kv_rank + m.rot_dim) + 2 * m.heads * (m.dim + m.vdim) * m.kv_rank
                                    + M * (4 * m.heads * (m.dim + m.rot_dim + m.vdim) + 2 * m.heads * m.vdim), ctx_pairs * pair + carry)
    out["lm_head"] = (2 * cfg.vocab * W, 2.0 * head_rows * cfg.vocab * W)
    return out


def joined_costs(cfg: StackConfig, M: int, nseq: int, ctx_pairs: float, ctx_tokens: float) -> dict:
    """The same for layers whose sublayers' results are normed ahead of the stream."""
    W, head_rows = cfg.width, min(M, 8)
    out = {"lm_head": (2 * cfg.vocab * W, 2.0 * head_rows * cfg.vocab * W)}
    lin = lambda n, k, stored: (2 * n * k + M * (2 * k + stored), 2.0 * M * n * k)       # noqa: E731  (bytes a row leaves with)
    for l in cfg.layers:
        f, segs = l.mlp, sum(n for _, n in l.mixer.segments())
        out["project"], out["out"] = lin(segs, W, 4 * segs), lin(W, sum(n for _, n, _ in l.mixer.out_tensors()), 4 * W)
        out["join"] = out["end"] = (M * 14 * W, 0.0)                                     # result, stream, stream, operand
        for _, m, _ in l.mixer.parts():
            rows = sum(n for _, n in m.segments())
            if isinstance(m, ChannelDeltaMixer):
                out["mixer:channel_delta"] = (2 * 4 * nseq * m.heads * m.dim ** 2 + M * (4 * rows + 2 * m.out_features), M * m.heads * m.dim ** 2 * 9.0)
            else:
                part = min(1.0, m.window * nseq / max(ctx_tokens, 1)) if m.window else 1.0
                out["mixer:attention"] = (2 * part * ctx_tokens * m.kv_heads * (m.dim + m.vdim) + M * (4 * rows + 2 * m.out_features),
                                          part * ctx_pairs * 2.0 * m.heads * (m.dim + m.vdim))
        if isinstance(f, ExpertMix):
            routes, met = M * f.top, f.experts * (1 - (1 - f.top / f.experts) ** M)       # experts that some token chooses, choices alike
            out["route"] = (M * (4 * f.experts + 16 * f.top), 0.0)
            out["experts_up"] = (4 * met * f.ff * W + M * 2 * W + routes * 2 * f.ff, 4.0 * routes * f.ff * W)
            out["experts_down"] = (2 * met * f.ff * W + routes * 2 * (f.ff + W), 2.0 * routes * f.ff * W)
            out["up+experts"], out["down+experts"] = lin(f.experts + 2 * f.shared, W, 4 * f.experts + 2 * f.shared), lin(W, f.shared, 4 * W)
            out["end+experts"] = (M * (14 * W + 2 * f.top * W), 0.0)
        elif f is not None:
            out["up"], out["down"] = lin(2 * f.ff, W, 2 * f.ff), lin(W, f.ff, 4 * W)
    return out


def hybrid_costs(cfg: C.HybridConfig, M: int, nseq: int, ctx_pairs: float, ctx_tokens: float) -> dict:
    sh = C.shard(cfg, 1, 0)
    H, D = cfg.hidden, 128
    lin = H * (sh.gdn_in_n + 2 * sh.ffn_inter) + H * (sh.gdn_out_k + sh.ffn_inter)
    out = {"linears": (0.5 * lin + M * (2 * sh.gdn_in_n + sh.gdn_out_k + sh.ffn_inter + 12 * H), 2.0 * M * lin)}
    out["delta"] = (2 * 4 * nseq * sh.gdn_v_heads * D * D + M * (2 * sh.gdn_in_n + sh.gdn_out_k), M * sh.gdn_v_heads * D * D * 8.0)
    if cfg.moe is not None:
        f = cfg.moe
        met, mats = f.n_experts * (1 - (1 - f.top_k / f.n_experts) ** M), 3 * f.expert_inter * H
        lin -= 3 * H * sh.ffn_inter
        out["linears"] = (0.5 * lin + M * (2 * sh.gdn_in_n + sh.gdn_out_k + 12 * H), 2.0 * M * lin)
        out["experts"] = (0.5 * (met * mats + 3 * f.shared_inter * H) + f.n_experts * H + M * f.top_k * (2 * H + 2 * 4 * f.expert_inter + 2 * H) + M * 4 * H,
                          2.0 * M * (f.top_k * mats + 3 * f.shared_inter * H))
    out["attention"] = (2 * ctx_tokens * sh.n_kv_heads * cfg.head_dim + M * (2 * sh.qkv_n + sh.o_k), ctx_pairs * 4.0 * sh.n_q_heads * cfg.head_dim)
    return out


def measure(cfg, prompt: int, streams: int, rung: int, steps: int, warmup: int, detail: bool) -> dict:
    stack = isinstance(cfg, StackConfig)
    ctx = prompt + 64 * ((steps + warmup) // 64 + 4)
    if stack:
        model = StackModel(cfg, max_seqs=streams, max_ctx=ctx, seed=5)
    else:
        model = HybridModel(cfg, max_seqs=streams, max_ctx=ctx, max_width=1, seed=5, use_drafter=False)
    page = cfg.page_tokens
    per = (ctx + page - 1) // page
    g = torch.Generator().manual_seed(3)
    toks = torch.randint(0, cfg.vocab, (streams, prompt), generator=g).tolist()
    blocks = [list(range(1 + j * per, 1 + (j + 1) * per)) for j in range(streams)]
    pb = model.build_bucket("prefill", 1, rung)
    ms, last = [], [0] * streams
    for j in range(streams):
        model.reset_slot(j + 1)
        torch.cuda.synchronize()
        e0, e1 = torch.cuda.Event(enable_timing=True), torch.cuda.Event(enable_timing=True)
        e0.record(model.stream)
        for pos in range(0, prompt, rung):
            r = run_bucket(model, pb, [SeqStep(toks[j][pos:pos + rung], pos, j + 1, 0, blocks[j])])
        e1.record(model.stream)
        torch.cuda.synchronize()
        last[j] = r.tokens[0][0]
        ms.append(e0.elapsed_time(e1))
    model.scratch.check()
    flush = torch.empty(256 << 20, dtype=torch.uint8, device="cuda")
    res = {"prefill_ms": statistics.median(ms), "prefill_tok_s": prompt / statistics.median(ms) * 1e3, "prefill_launches": pb.n_launches}
    if detail:      # the last portion again, group by group (the tables of that step are still on the device)
        lo = prompt - rung
        costs = (stack_costs if stack else hybrid_costs)(cfg, rung, 1, rung * lo + rung * (rung + 1) / 2.0, prompt)
        res["prefill_groups"] = _detail(model, pb, costs, flush)
    db = model.build_bucket("decode", streams, 1)
    pos = prompt

    def step():
        nonlocal pos, last
        r = run_bucket(model, db, [SeqStep([last[j]], pos, j + 1, 1 if (pos > prompt and not stack) else 0, blocks[j], uid=j, step_no=pos,
                                           blocks_key=("b", j)) for j in range(streams)])
        last = [t[0] for t in r.tokens]
        pos += 1
    for _ in range(warmup):
        step()
    torch.cuda.synchronize()
    e0, e1 = torch.cuda.Event(enable_timing=True), torch.cuda.Event(enable_timing=True)
    e0.record(model.stream)
    for _ in range(steps):
        step()
    e1.record(model.stream)
    torch.cuda.synchronize()
    model.scratch.check()
    t = e0.elapsed_time(e1) / steps
    res.update(decode_ms_per_step=t, decode_tok_s=streams / t * 1e3, decode_launches=db.n_launches)
    if detail:
        costs = (stack_costs if stack else hybrid_costs)(cfg, streams, streams, streams * pos, streams * pos)
        res["decode_groups"] = _detail(model, db, costs, flush)
    res["state_bytes"] = model.state_bytes()
    return res


def _detail(model, b, costs: dict, flush) -> dict:
    out = {}
    for g, ranges in _groups(model, b).items():
        if not ranges:
            continue
        one = ranges[len(ranges) // 2]
        us = _time(model, b, one if isinstance(one, list) else [one], flush)
        nb, fl = costs.get(g, (0, 0))
        roof = _roof(nb, fl)
        out[g] = {"us": round(us, 1), "roofline_us": round(roof, 1), "of_roofline": round(roof / us, 3), "per_step": len(ranges)}
    return out


def run(args) -> dict:
    names = SIZES if args.stack == "all" else tuple(args.stack.split(","))
    out = {"metric": "layer_stack_prefill_decode_tok_s", "n_gpus": 1, "data": "synthetic", "dtype": "bf16", "steps": args.steps,
           "config": {"prompt": args.prompt, "streams": args.streams, "rung": args.rung, "l2": "flushed between group timings; weights of a step exceed L2"},
           "models": {}}
    for n in names:
        cfg = C.by_name(n)
        for c in (cfg, *like_models(cfg)):
            out["models"][c.name] = measure(c, args.prompt, args.streams, args.rung, args.steps, args.warmup, True)
            torch.cuda.empty_cache()
    return out
