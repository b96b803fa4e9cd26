"""Trace replay: token ids in, logits out, nothing sampled.

    bin/trace_run --model DIR --dtype bfloat16|float32 --out DIR --max-tokens N

Standard input carries one JSON object a line:

    {"step": 0, "entries": [{"id": "a", "tokens": [5, 17, 3], "want": [0, 2]}], "end": []}

`entries` are the next tokens of each request (all entries of a step are one batch: portions of prompts of any
length beside single decoded tokens), `want` the places among them whose logits are asked for, `end` the
requests whose pages and slot are given back after the step.  A step that wants logits writes DIR/<step>.f32
(little-endian fp32, [wanted, vocab], in the order of the entries); every step prints `done <step>`.

The engine's own parts do the work: the model class its config.json names, the page and slot allocators of
the scheduler with a pool for N tokens and four slots, and the executor's step.
"""
from __future__ import annotations

import argparse
import json
import os
import sys
from dataclasses import dataclass, field

MAX_LIVE = 4
PREFILL_RUNGS = (16, 64, 256, 1024, 2048)


@dataclass
class _Request:
    slot: int
    key: tuple
    blocks: list = field(default_factory=list)
    pos: int = 0


class TraceEngine:
    """Replay over one model: its executor, and the scheduler's allocators for its pages and slots."""

    def __init__(self, model, prefill_rungs: tuple = PREFILL_RUNGS, capture: bool = True):
        from ..sched.alloc import Arenas, GdnStateAllocator, PagedKvAllocator
        from .hybrid_executor import HybridExecutor
        self.model = model
        self.ex = HybridExecutor(model, decode_batches=tuple(range(1, model.max_seqs + 1)), decode_widths=(1,), prefill_rungs=prefill_rungs,
                                 prefill_pack=model.max_seqs, capture=capture)
        self.arenas = Arenas(PagedKvAllocator(model.kv_blocks, model.cfg.page_tokens), GdnStateAllocator(model.max_seqs + 1))
        self.live: dict = {}
        self.admitted = 0

    @staticmethod
    def open(model_dir: str, dtype: str, max_tokens: int) -> "TraceEngine":
        import torch
        from ..models import config as MC
        from ..models.stack import StackModel
        cfg = MC.by_name(model_dir)
        pages = (max_tokens + cfg.page_tokens - 1) // cfg.page_tokens
        return TraceEngine(StackModel(cfg, device="cuda", max_seqs=MAX_LIVE, max_ctx=max(1, pages) * cfg.page_tokens, kv_blocks=pages + 1,
                                      dtype=getattr(torch, dtype)))      # block 0 is the null block

    def _admit(self, rid) -> _Request:
        self.admitted += 1
        r = _Request(self.arenas.gdn.allocate(), ("trace", self.admitted))
        self.ex.reset_slot(r.slot)
        self.live[rid] = r
        return r

    def step(self, entries: list):
        """[(request id, tokens)] -> logits of all their rows, entry by entry."""
        import torch
        from ..sched.executor import SeqRun
        parts = []
        for rid, toks in entries:
            r = self.live.get(rid) or self._admit(rid)
            bad = [t for t in toks if not 0 <= t < self.ex.vocab]
            if bad:
                raise ValueError(f"request {rid!r}: token {bad[0]} is outside the vocabulary")
            need = self.arenas.kv.blocks_for(r.pos + len(toks)) - len(r.blocks)
            if need > 0:
                r.blocks = r.blocks + self.arenas.kv.allocate(need)
            parts.append([r, list(toks), []])
        top = max(self.ex.prefill_rungs)
        todo = [p for p in parts if p[1]]
        while todo:                       # more rows than the largest bucket: the batch runs in pieces
            runs, took, room = [], [], top
            for p in todo:
                n = min(len(p[1]), room)
                if n == 0:
                    break
                r = p[0]
                runs.append(SeqRun(0, p[1][:n], r.pos, r.slot, 0, r.blocks, last_chunk=False, blocks_key=r.key))
                took.append((p, n))
                room -= n
            logits = self.ex.forward_logits(runs)
            at = 0
            for p, n in took:
                p[2].append(logits[at:at + n])
                p[1] = p[1][n:]
                p[0].pos += n
                at += n
            todo = [p for p in todo if p[1]]
        self.model.scratch.check()
        return [torch.cat(p[2]) if p[2] else torch.zeros(0, self.ex.vocab) for p in parts]

    def end(self, rid) -> None:
        r = self.live.pop(rid)
        self.arenas.release(r.blocks, r.slot)


def main(argv=None) -> int:
    ap = argparse.ArgumentParser(prog="trace_run", description="replay a trace of token ids and write logits")
    ap.add_argument("--model", required=True, help="folder with config.json and model.safetensors")
    ap.add_argument("--dtype", required=True, choices=["bfloat16", "float32"])
    ap.add_argument("--out", required=True)
    ap.add_argument("--max-tokens", type=int, required=True, help="tokens that live requests hold at most (sizes the page pool)")
    a = ap.parse_args(argv)
    import torch
    eng = TraceEngine.open(a.model, a.dtype, a.max_tokens)
    for line in sys.stdin:
        if not line.strip():
            continue
        s = json.loads(line)
        rows = eng.step([(e["id"], e["tokens"]) for e in s["entries"]])
        want = [r[e["want"]] for r, e in zip(rows, s["entries"]) if e["want"]]
        if want:
            part = os.path.join(a.out, f".{s['step']}.part")
            with open(part, "wb") as f:
                f.write(torch.cat(want).contiguous().numpy().astype("<f4").tobytes())
            os.replace(part, os.path.join(a.out, f"{s['step']}.f32"))
        for rid in s["end"]:
            eng.end(rid)
        print(f"done {s['step']}", flush=True)
    return 0
