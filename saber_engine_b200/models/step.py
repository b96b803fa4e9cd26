"""One planned step shape: the index tables of a step, the bucket (program + tables + read-backs) built for
it, and the step function that fills the tables, runs the program and parses what comes back.  Shared by
every model class: `models.hybrid.HybridModel` and `models.stack.StackModel`.

Parity: the index tables of `crates/saber-exec/src/forward.rs:587-860` (slot 0 is the null slot; padding
rows carry slot_map -1).
"""
from __future__ import annotations

from dataclasses import dataclass, field
from typing import Optional

import torch

from ..ops import native as N


@dataclass
class BlobLayout:
    """Offsets (in int32 words) of the per-step index tables inside a bucket's index blob."""
    M: int
    nseq: int
    max_blocks: int
    ids: int = 0
    pos: int = 0
    slot_map: int = 0
    cu_rows: int = 0
    slots: int = 0
    shift: int = 0
    kv_len: int = 0
    seq_uid: int = 0
    step_no: int = 0
    last_rows: int = 0
    temps: int = 0
    next_ids: int = 0          # per row: the token that follows it in its prompt (-1: none), for prompt log-probabilities
    samp: int = 0              # per HEAD row: fp32 {temperature, top_k, top_p, min_p} (temperature 0: keep the greedy pick)
    samp_u: int = 0            # per HEAD row: the uniform number of the draw (fp32)
    block_table: int = 0
    words: int = 0

    @staticmethod
    def make(M: int, nseq: int, max_blocks: int) -> "BlobLayout":
        b = BlobLayout(M, nseq, max_blocks)
        off = 0
        def take(n):
            nonlocal off
            o = off
            off += (n + 3) // 4 * 4          # keep every table 16-byte aligned
            return o
        b.ids = take(M)
        b.pos = take(3 * M)
        b.slot_map = take(M)
        b.cu_rows = take(nseq + 1)
        b.slots = take(nseq)
        b.shift = take(nseq)
        b.kv_len = take(nseq)
        b.seq_uid = take(nseq)
        b.step_no = take(nseq)
        b.last_rows = take(nseq)
        b.temps = take(M)
        b.next_ids = take(M)
        b.samp = take(4 * M)
        b.samp_u = take(M)
        b.block_table = take(nseq * max_blocks)
        b.words = off
        return b

    @property
    def header_words(self) -> int:
        return self.block_table


@dataclass
class Bucket:
    """One planned shape: its program, blob layout, output tensors."""
    kind: str                 # "decode" | "prefill"
    nseq: int
    width: int                # rows per sequence (decode) or rung rows (prefill, nseq sequences packed)
    M: int
    layout: BlobLayout
    program: N.Program
    blob_dev: torch.Tensor    # int32 [words]
    blob_host: torch.Tensor   # pinned int32 [words]
    out_dev: torch.Tensor     # int32: n_commit[nseq] | out_tokens[nseq*W] | drafts[nseq*block] | picks[M]
    out_host: torch.Tensor    # pinned mirror
    captured: bool = False
    n_launches: int = 0
    logits: Optional[torch.Tensor] = None
    keep: list = field(default_factory=list)
    bt_rows: dict = field(default_factory=dict)    # row j -> (blocks_key, n blocks) of the block-table row the device holds
    last_h2d_bytes: int = 0                        # index-table bytes the last step copied to the device
    arenas: list = field(default_factory=list)     # pure activation buffers: written before read in every step
    digests: Optional[torch.Tensor] = None         # int64 [n_layers + 1] stage digests (race_check = "shadow")
    sp: bool = False                               # prefill on several ranks: the sequence-parallel chain (rows owned by ranks)
    seam_dev: Optional[torch.Tensor] = None        # int32 blob: ids [Mh*64] | values [Mh*64] fp32 bits | lse [Mh*2] (seam buckets)
    seam_host: Optional[torch.Tensor] = None       # pinned mirror
    plp_dev: Optional[torch.Tensor] = None         # int32 blob of a prompt-log-probability bucket (every row: candidates, lse, next-token logit)
    plp_host: Optional[torch.Tensor] = None


def head_outputs(nseq: int, W: int, block: int, Mh: int, dev) -> tuple:
    """The int32 blob a step reads back: n_commit[nseq] | out_tokens[nseq * W] | drafts[nseq * block] | picks[Mh]."""
    nd = nseq * max(block, 1)
    out = torch.zeros(nseq + nseq * W + nd + Mh, dtype=torch.int32, device=dev)
    return out, out[:nseq], out[nseq:nseq + nseq * W], out[nseq + nseq * W + nd:]


def seam_outputs(Mh: int, dev) -> tuple:
    """One int32 blob so that the read-back is one copy: ids | values (fp32 bits) | log-sum-exp pairs."""
    d = torch.zeros(Mh * (2 * N.SEAM_K + 2), dtype=torch.int32, device=dev)
    k = Mh * N.SEAM_K
    return d, d[:k], d[k: 2 * k].view(torch.float32), d[2 * k:].view(torch.float32)


def plp_outputs(M: int, dev) -> tuple:
    """ids [M*K] | values [M*K] | lse [M*2] | logit of the next prompt token [M]."""
    d = torch.zeros(M * (2 * N.SEAM_K + 3), dtype=torch.int32, device=dev)
    k = M * N.SEAM_K
    return d, d[:k], d[k: 2 * k].view(torch.float32), d[2 * k: 2 * k + 2 * M].view(torch.float32), d[2 * k + 2 * M:].view(torch.float32)


def finish_bucket(model, prog: N.Program, key, kind, nseq, width, M, lay, blob, blob_host, keep, capture: bool, head: dict) -> Bucket:
    """Pinned mirrors of the outputs, one eager walk and the graph capture; registers the bucket with the model."""
    out = head["out"]
    pinned = lambda t: None if t is None else torch.zeros(t.numel(), dtype=torch.int32).pin_memory()   # noqa: E731
    prog.keep(*[k for k in keep if k is not None], model.w)
    b = Bucket(kind, nseq, width, M, lay, prog, blob, blob_host, out, pinned(out), n_launches=prog.declared_launches,
               logits=head["logits"], keep=keep)
    b.W, b.block, b.Mh = head["W"], head["block"], head["Mh"]
    b.seam_dev, b.plp_dev = head.get("seam"), head.get("plp")
    b.plp_logits = head.get("plp_logits") if b.plp_dev is not None else None
    b.plp_host, b.seam_host = pinned(b.plp_dev), pinned(b.seam_dev)
    if capture:
        # the bucket's buffers were zeroed on the current stream; one eager walk first: sets function
        # attributes and warms lazy module loading
        model.stream.wait_stream(torch.cuda.current_stream())
        with torch.cuda.stream(model.stream):
            prog.run(model.stream)
            model.stream.synchronize()
            model.scratch.check()
            prog.capture(model.stream)
        model.stream.synchronize()
        b.captured = True
    else:
        torch.cuda.current_stream().synchronize()
    model.buckets[key] = b
    return b


@dataclass
class SeqStep:
    """What one sequence contributes to a step."""
    tokens: list              # token ids of this step's rows (decode: [last committed, drafts...])
    pos0: int                 # position of the first row
    slot: int                 # GDN state slot (>= 1)
    shift: int                # rows of the previous decode step that were committed (0 after prefill)
    blocks: list              # physical KV block ids covering positions [0, pos0 + len(tokens))
    uid: int = 0
    step_no: int = 0
    rope_pos: Optional[object] = None   # int [3, rows]: three-axis rotary positions of the rows (prompts with images)
    rope_delta: int = 0       # added to the index of every row for the rotary position (after an image)
    next_token: int = -1      # the prompt token after this chunk's last row (-1: none), for prompt log-probabilities
    sampling: Optional[tuple] = None   # (temperature, top_k, top_p, min_p) of a sampled sequence the device may draw for
    uniforms: Optional[list] = None    # one uniform number per head row of this step (decode: every row; prefill: the last)
    blocks_key: Optional[object] = None   # identity of `blocks` (same key = same list contents): the block table row is then uploaded once


@dataclass
class StepResult:
    n_commit: list            # per sequence: tokens committed (decode) / 1 (prefill last chunk)
    tokens: list              # per sequence: committed token ids
    drafts: list              # per sequence: next block of draft tokens
    picks: list


def fill_blob(b: Bucket, seqs: list, page_tokens: int = 16) -> list:
    """Write the index tables of one step into the bucket's pinned blob.  Returns the word ranges
    [(first, count), ...] that have to reach the device: the header (every per-row and per-sequence
    table) and the block-table rows that changed.  A sequence's KV blocks are allocated up front
    and never change, so a row whose `blocks_key` is the one the device already holds is skipped:
    in steady-state decode no block-table byte crosses the bus (the reference sends the table only
    on page-crossing steps, `crates/saber-engine/src/tp2.rs:1897`)."""
    import numpy as np
    lay = b.layout
    a = b.blob_host.numpy()
    M, nseq = lay.M, lay.nseq
    hdr = lay.header_words
    a[:hdr] = 0
    a[lay.slot_map:lay.slot_map + M] = -1
    a[lay.next_ids:lay.next_ids + M] = -1
    a[lay.slots:lay.slots + nseq] = -1
    ranges = [(0, hdr)]
    row = 0
    for j, s in enumerate(seqs):
        n = len(s.tokens)
        a[lay.ids + row: lay.ids + row + n] = s.tokens
        a[lay.next_ids + row: lay.next_ids + row + n] = list(s.tokens[1:]) + [s.next_token]
        if s.sampling is not None and s.uniforms:
            hr0, hn = (row, n) if b.kind == "decode" else (j, 1)      # head rows of this sequence
            fa = a.view(np.float32)
            for r in range(min(hn, len(s.uniforms))):
                fa[lay.samp + 4 * (hr0 + r): lay.samp + 4 * (hr0 + r) + 4] = s.sampling
                fa[lay.samp_u + hr0 + r] = s.uniforms[r]
        pos = np.arange(s.pos0, s.pos0 + n, dtype=np.int32)
        for ax in range(3):
            a[lay.pos + ax * M + row: lay.pos + ax * M + row + n] = \
                pos + s.rope_delta if s.rope_pos is None else np.asarray(s.rope_pos[ax], dtype=np.int32)[:n]
        nblk = len(s.blocks)
        first_page, last_page = s.pos0 // page_tokens, (s.pos0 + n - 1) // page_tokens
        touched = np.asarray(s.blocks[first_page:last_page + 1], dtype=np.int32)     # pages this step's rows write
        a[lay.slot_map + row: lay.slot_map + row + n] = touched[pos // page_tokens - first_page] * page_tokens + pos % page_tokens
        a[lay.cu_rows + j] = row
        a[lay.slots + j] = s.slot
        a[lay.shift + j] = s.shift
        a[lay.kv_len + j] = s.pos0 + n
        a[lay.seq_uid + j] = s.uid
        a[lay.step_no + j] = s.step_no
        a[lay.last_rows + j] = row + n - 1
        bt = lay.block_table + j * lay.max_blocks
        sig = (s.blocks_key, nblk) if s.blocks_key is not None else None
        held = getattr(b, "bt_rows", None)
        if sig is None or held is None or held.get(j) != sig:
            a[bt: bt + nblk] = np.asarray(s.blocks, dtype=np.int32)
            ranges.append((bt, nblk))
            if held is not None:
                held[j] = sig
        row += n
    for j in range(len(seqs), nseq + 1):
        a[lay.cu_rows + j] = row
    assert row <= M, (row, M)
    return ranges


def run_bucket(model, b: Bucket, seqs: list, eager: bool = False) -> StepResult:
    """One step: index tables host->device (pinned; only what changed), the program (graph replay
    or eager walk), results device->host, then parse."""
    ranges = fill_blob(b, seqs, model.cfg.page_tokens)
    st = model.stream
    with torch.cuda.stream(st):
        nbytes = 0
        for first, count in ranges:
            if count > 0:
                b.blob_dev[first:first + count].copy_(b.blob_host[first:first + count], non_blocking=True)
                nbytes += 4 * count
        b.last_h2d_bytes = nbytes
        if b.captured and not eager:
            b.program.replay(st)
        else:
            b.program.run(st)
        b.out_host.copy_(b.out_dev, non_blocking=True)
        if getattr(b, "seam_dev", None) is not None:
            b.seam_host.copy_(b.seam_dev, non_blocking=True)
        if getattr(b, "plp_dev", None) is not None:
            b.plp_host.copy_(b.plp_dev, non_blocking=True)
    # bounded: a step that never completes (a kernel wait that did not run out, a lost peer) raises,
    # and the scheduler's fatal law ends the engine instead of leaving this thread blocked
    from ..runtime.device_rt import bounded_wait
    bounded_wait(st, model.step_timeout_s, f"the {b.kind} step")
    return parse_result(b, len(seqs))


def parse_result(b: Bucket, n_live: int) -> StepResult:
    o = b.out_host.numpy()
    nseq, W, block, Mh = b.nseq, b.W, b.block, b.Mh
    o_commit = o[:nseq]
    o_tokens = o[nseq:nseq + nseq * W].reshape(nseq, W)
    nd = max(block, 1)
    o_drafts = o[nseq + nseq * W: nseq + nseq * W + nseq * nd].reshape(nseq, nd)
    o_picks = o[nseq + nseq * W + nseq * nd:]
    if b.kind == "decode":
        n_commit = [int(o_commit[j]) for j in range(n_live)]
        tokens = [o_tokens[j, :n_commit[j]].tolist() for j in range(n_live)]
    else:
        n_commit = [1] * n_live
        tokens = [[int(o_picks[j])] for j in range(n_live)]
    drafts = [o_drafts[j, :block].tolist() for j in range(n_live)]
    return StepResult(n_commit, tokens, drafts, o_picks.tolist())
