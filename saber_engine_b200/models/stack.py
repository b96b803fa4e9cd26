"""A decoder assembled from a list of layers (`models.stack_config.StackConfig`) as native step programs.

The residual stream stays fp32; a linear that ends a sublayer adds its result to it and leaves the next linear's operand
(norm weight times x) with the row's partial sums of squares, so that no normalisation, activation or addition needs a
launch of its own.
  parallel    x <- x + mixer(norm(x)) + ff(norm(x)): two linears around the mixer's kernels.  Two norms: the same, the rows of the
              feed-forward multiply a second operand
  sequential  x <- x + mixer(norm1(x)); x <- x + ff(norm2(x)): two linears around the mixer, two for the feed-forward
  joined      x <- x + c norm(mixer(blend of norm(x) with the token before)); x <- x + c norm(ff(norm(x))): a sublayer's result is whole
              rows ahead of the stream, so that a row kernel stands between the linears (`join.cu`): it norms the result, adds it, norms
              the stream and, ahead of a mixer, blends.  Mixers may stand side by side between the same two linears
Launches of a mixer in decoding (of mixers side by side, the first on a stream of its own): delta rule 1, decayed outer products 1, grouped-query attention 1 (2 behind a convolution), latent attention 5 (6 where
queries come from a latent of their own); a pass of a looped block adds one linear, routed experts add 3 (routing and two grouped
products: the output linear's epilogue adds the experts' rows to the stream).

Every row of every bucket is committed (no drafter): a decode bucket is one row per sequence, a prefill bucket
is `width` ragged rows of up to `nseq` sequences, single decoded tokens beside portions of prompts included.
Caches and states belong to a layer RUN: the pages of an attention run (a run may read those of an earlier one), the
slots of a recurrent run, of a convolution's inputs and of the last token's row where tokens are blended.
"""
from __future__ import annotations

import ctypes as C
from typing import Optional

import torch

from ..ops import functional as F
from ..ops import layouts as L
from ..ops import native as N
from . import stack_weights as SW
from .stack_config import ChannelDeltaMixer, DeltaMixer, ExpertMix, GroupedMixer, LatentMixer, OuterMixer, StackConfig
from .step import BlobLayout, Bucket, finish_bucket, head_outputs, plp_outputs, seam_outputs


class StackModel:
    def __init__(self, cfg: StackConfig, device="cuda", max_seqs: int = 8, max_ctx: Optional[int] = None, kv_blocks: Optional[int] = None,
                 weights: Optional[SW.StackWeights] = None, seed: int = 0, dtype: torch.dtype = torch.bfloat16, fuse: bool = True,
                 expand_bytes: int = 24 << 30, race_check: str = "off", attn_impl: str = "tc", side_stream: bool = True):
        if dtype not in (torch.bfloat16, torch.float32):
            raise ValueError("dtype must be bfloat16 or float32")
        if attn_impl not in ("tc", "mma"):
            raise ValueError("attn_impl must be 'tc' or 'mma'")
        # side_stream: mixers side by side run beside each other in decoding (in prompts each fills the SMs, and the scan's few warps
        # would wait for the other's)
        self.attn_impl, self.side_stream = attn_impl, side_stream
        if race_check not in ("off", "shadow"):
            raise ValueError("race_check must be 'off' or 'shadow'")
        self.cfg, self.tp, self.rank, self.comm = cfg, 1, 0, None
        self.dtype, self.f32 = dtype, dtype == torch.float32
        self.device = torch.device(device)
        self.max_seqs, self.max_width = max_seqs, 1
        self.max_ctx = max_ctx or cfg.max_ctx
        self.max_blocks = (self.max_ctx + cfg.page_tokens - 1) // cfg.page_tokens
        self.kv_blocks = kv_blocks if kv_blocks is not None else max_seqs * self.max_blocks + 1
        self.fuse, self.race_check, self.image_rows = bool(fuse), race_check, 0
        self.step_timeout_s = 120.0
        self.scratch = F.scratch(self.device)
        dev = self.device
        if weights is not None:
            self.w = weights
        elif cfg.source is not None:
            self.w = SW.load(cfg, cfg.source, dtype, dev)
        else:
            self.w = SW.random_init(cfg, dtype, dev, seed)
        self.n_slots = max_seqs + 1                       # slot 0 is the null slot
        self.kv, self.state, self.hist, self.before = {}, {}, {}, {}
        for r in cfg.runs:
            if cfg.token_shift:
                self.before[r.index] = torch.zeros(self.n_slots, cfg.width, dtype=torch.float32, device=dev)
            for pre, m, _ in cfg.layers[r.layer].mixer.parts():
                key = self._key(r, pre)
                if isinstance(m, LatentMixer):
                    if m.kv_from is None:
                        self.kv[key] = torch.zeros(self.kv_blocks, cfg.page_tokens, m.rank_pad + m.rot_pad, dtype=dtype, device=dev)
                    continue
                if isinstance(m, GroupedMixer):
                    if m.kv_from is None:                 # the padding of a page stays zero: the kernels multiply it
                        self.kv[key] = torch.zeros(self.kv_blocks, m.kv_heads, cfg.page_tokens * (m.key_pad + m.vdim_pad), dtype=dtype, device=dev)
                else:
                    self.state[key] = torch.zeros(self.n_slots, m.heads, m.vdim_pad, m.dim_pad, dtype=torch.float32, device=dev)
                if m.taps:
                    self.hist[key] = torch.zeros(self.n_slots, m.taps, m.channels, dtype=torch.float32, device=dev)
        # expanded keys / values of the pages a prompt portion sees: scratch of one layer run at a time, in
        # physical page order (absent when it would not fit its budget: the absorbed form serves then)
        self.k_exp = self.v_exp = None
        lat = [m for m in cfg.mixers() if isinstance(m, LatentMixer)]
        tokens = self.kv_blocks * cfg.page_tokens
        if lat and not self.f32 and tokens * cfg.expanded_token_bytes() <= expand_bytes:
            self.k_exp = torch.zeros(tokens * max(m.heads * m.key_tile for m in lat), dtype=dtype, device=dev)
            self.v_exp = torch.zeros(tokens * max(m.heads * m.vdim_pad for m in lat), dtype=dtype, device=dev)
        self.buckets: dict = {}
        self.stream = torch.cuda.Stream(device=dev)
        torch.cuda.synchronize(dev)                       # buckets run on a stream of their own

    # ------------------------------------------------------------------------------ state
    @staticmethod
    def _key(run, prefix: str):
        """Name of a mixer's caches and states: the layer run, and the part where mixers stand side by side."""
        return run.index if not prefix else f"{run.index}.{prefix[:-1]}"

    def reset_slot(self, slot: int) -> None:
        with torch.cuda.stream(self.stream):
            for t in self.slot_tensors().values():
                t[slot].zero_()

    def page_pools(self) -> dict:
        return {f"kv.{i}": t for i, t in self.kv.items()}

    def slot_tensors(self) -> dict:
        return {f"{name}.{i}": t for name, d in (("state", self.state), ("hist", self.hist), ("before", self.before)) for i, t in d.items()}

    def snapshot_views(self, slot: int) -> dict:
        return {k: t[slot] for k, t in self.slot_tensors().items()}

    def state_bytes(self) -> dict:
        size = lambda d: sum(t.numel() * t.element_size() for t in d.values())    # noqa: E731
        exp = 0 if self.k_exp is None else (self.k_exp.numel() + self.v_exp.numel()) * 2
        return {"weights": self.w.nbytes(), "kv_pool": size(self.kv), "state": size(self.state) + size(self.hist) + size(self.before),
                "expanded_kv_scratch": exp}

    # ------------------------------------------------------------------------------ builders
    def _operand(self, t: torch.Tensor, M: int, K: int) -> N.Operand:
        o = N.Operand()
        o.p, o.M_pad, o.ld, o.fmt = t.data_ptr(), L.padded_rows(M), K, int(self.f32)
        return o

    def _operand_buf(self, M: int, K: int) -> torch.Tensor:
        """Zeroed storage of a [M, K] operand: padding rows and columns stay zero."""
        return torch.zeros(L.padded_rows(M) * L.round_up(K, 64), dtype=self.dtype, device=self.device)

    def _linear(self, prog: N.Program, lin: SW.Linear, a: torch.Tensor, M: int, e: N.LinEpi, ws: Optional[torch.Tensor], tag: str,
                second: Optional[tuple] = None) -> None:
        """second: (operand, first weight tile that reads it)."""
        p = N.LinParams()
        if second is not None:
            p.a2, p.a2_tile0 = second[0].data_ptr(), second[1]
        sc = self.scratch
        p.w, p.a, p.err = lin.w.data_ptr(), a.data_ptr(), sc.err.data_ptr()
        p.ws, p.counters = (ws if ws is not None else sc.ws).data_ptr(), sc.counters.data_ptr()
        p.M, p.M_pad, p.N_pad, p.K = M, L.padded_rows(M), lin.N_pad, lin.K
        p.nt, p.fp32, p.fuse, p.splits, p.mtiles = L.token_tile(M), int(self.f32), int(self.fuse), 1, 1
        if not self.f32:
            tiles, kb = lin.N_pad // 256 * ((M + p.nt - 1) // p.nt), lin.K // 64
            p.splits = F.stream_splits(tiles, kb)
            p.mtiles = 2 if (M > 128 and tiles > F.device_sms() and p.M_pad % 256 == 0) else 1
        p.e = e
        prog.linear(p, tag=tag)

    def _grouped_linear(self, prog: N.Program, lin: SW.Linear, a: torch.Tensor, a_rows: int, ew: dict, gather: bool, e: N.LinEpi,
                        ws: Optional[torch.Tensor], tag: str) -> None:
        """The routed rows of a step against the stack of experts.  gather: the operand's rows are tokens."""
        p, sc = N.LinParams(), self.scratch
        p.w, p.a, p.err, p.counters = lin.w.data_ptr(), a.data_ptr(), sc.err.data_ptr(), sc.counters.data_ptr()
        p.ws = (ws if ws is not None else sc.ws).data_ptr()
        p.M, p.M_pad, p.N_pad, p.K, p.splits, p.mtiles = ew["rows"], a_rows, lin.N_pad, lin.K, 1, ew["mtiles"]
        p.nt, p.fp32, p.fuse = ew["nt"], int(self.f32), int(self.fuse)
        p.group_tiles, p.group_ntiles, p.group_rows, p.group_max = (*(ew[k].data_ptr() for k in ("tiles", "ntiles", "src_row")), ew["max_tiles"])
        p.src_row = ew["src_row"].data_ptr() if gather else None
        p.group_w_stride = lin.N_pad * lin.K * lin.w.element_size() if self.f32 else lin.N_pad * lin.K * 2
        p.e = e
        prog.linear(p, tag=tag)

    def _row_norm(self, e: N.LinEpi, ss: torch.Tensor) -> None:
        """The operand's rows were left undivided: scale the product by the row's reciprocal root mean square."""
        e.ss, e.ss_n = ss.data_ptr(), ss.shape[1]
        e.inv_width, e.eps = 1.0 / self.cfg.width, self.cfg.eps

    def _stream_epi(self, x: torch.Tensor, add: bool, target: tuple, bias: Optional[torch.Tensor] = None) -> N.LinEpi:
        """target: (operand, first column, norm weight or None, sums of squares or None) of the next linear, and the same stream's
        second operand with its norm weight (or None)."""
        e = N.LinEpi()
        op, k0, norm_w, ss, op2, norm_w2 = target
        if norm_w2 is not None:
            e.op2, e.norm_w2 = op2, norm_w2.data_ptr()
        e.stream, e.x, e.ldx, e.width, e.add = 1, x.data_ptr(), x.stride(0), self.cfg.width, int(add)
        e.bias, e.norm_w = N.ptr(bias), N.ptr(norm_w)
        e.op, e.op_k0 = op, k0
        if ss is not None:
            e.ss_out, e.ss_out_n = ss.data_ptr(), ss.shape[1]
        return e

    def build_bucket(self, kind: str, nseq: int, width: int, capture: bool = True, seam: bool = False, plp: bool = False) -> Bucket:
        """kind = 'decode': one row of each of nseq sequences.  kind = 'prefill': up to nseq sequences packed in
        `width` rows.  seam: the best candidates of every head row for the host sampler.  plp: the head over
        EVERY row, with the candidates and the logit of the row's successor."""
        key = ((kind, nseq, width, "seam") if seam else (kind, nseq, width))
        if plp:
            if kind != "prefill":
                raise ValueError("prompt log-probabilities: prefill buckets only")
            key = key + ("plp",)
        if key in self.buckets:
            return self.buckets[key]
        decode = kind == "decode"
        if decode and width != 1:
            raise ValueError("this model has no drafter: decode width 1 only")
        cfg, dev, w = self.cfg, self.device, self.w
        M = nseq if decode else width
        W, KW = cfg.width, L.round_up(cfg.width, 64)
        lay = BlobLayout.make(M, nseq, self.max_blocks)
        blob = torch.zeros(lay.words, dtype=torch.int32, device=dev)
        blob_host = torch.zeros(lay.words, dtype=torch.int32).pin_memory()
        at = lambda off: blob.data_ptr() + 4 * off      # noqa: E731
        f32 = lambda *s: torch.zeros(*s, dtype=torch.float32, device=dev)   # noqa: E731
        prog = N.Program(f"{kind}-b{nseq}-w{width}")

        # ---- activation buffers
        x = f32(M, L.round_up(W, 32))
        ss = f32(L.padded_rows(M), (W + 127) // 128) if not cfg.post_norms else None
        h = self._operand_buf(M, KW)
        h2 = self._operand_buf(M, KW) if cfg.two_norms else None
        loop_op = self._operand_buf(M, 2 * KW) if cfg.loop is not None and cfg.loop_linear else None
        mid = self._operand_buf(M, max(l.out.K for l in w.layers))
        ups = [l for l in w.layers if l.down is not None]
        ff = self._operand_buf(M, max(l.down.K for l in ups)) if ups else None
        ldp = max(L.round_up(l.n_plain, 8) for l in w.layers)
        proj = f32(M, ldp)
        work = self._mixer_scratch(M, nseq, decode)
        experts = self._expert_scratch(M)
        big = max([x.N_pad for l in w.layers for x in (l.proj, l.out, l.up, l.carry) if x is not None] + [w.head.N_pad]) * M
        if experts:
            big = max([big] + [x.N_pad * experts["rows"] for l in w.layers for x in (l.experts_up, l.experts_down) if x is not None])
        ws = None
        if self.f32 or not self.fuse:                    # product rows (and, behind them, the split parts)
            ws = torch.empty(big + (0 if self.f32 else self.scratch.capacity // 4), dtype=torch.float32, device=dev)
        keep = [blob, x, ss, h, h2, loop_op, mid, ff, proj, ws, work, experts]
        digests = None
        if self.race_check == "shadow":
            digests = torch.zeros(len(cfg.runs) + 1, dtype=torch.int64, device=dev)
            prog.digest_clear(digests, len(cfg.runs) + 1, tag="digest.clear")

        if cfg.post_norms:
            arenas = dict(x=x, h=h, mid=mid, ff=ff, proj=proj, work=work, experts=experts, ws=ws, digests=digests)
            x = self._joined_layers(prog, M, nseq, decode, lay, at, arenas)
            keep.append(arenas)
            b = self._head(prog, key, kind, nseq, width, M, lay, at, blob, blob_host, x, h, None, ws, keep + [digests], seam, plp, capture)
            b.arenas = [a for a in (arenas["x"], arenas["x2"], arenas["y"], h, mid, ff, proj) if a is not None]
            b.digests, b.x = digests, x
            return b

        h_op = self._operand(h, M, KW)
        h2_op = self._operand(h2, M, KW) if h2 is not None else None
        l_op = self._operand(loop_op, M, 2 * KW) if loop_op is not None else None

        def target(run) -> tuple:
            """What the linear ahead of a run (None: ahead of the head) leaves for it."""
            if run is None:
                return h_op, 0, w.final_norm, ss, None, None
            if run.enter is not None:
                return l_op, 0, None, None, None, None
            lw = w.layers[run.layer]
            return h_op, 0, lw.norm, ss, h2_op, lw.norm2 if cfg.two_norms else None

        # ---- embedding
        runs = cfg.runs
        ep = N.StreamEmbedParams()
        ep.table, ep.table_f32, ep.vocab, ep.ids = w.embed.data_ptr(), int(self.f32), cfg.vocab, at(lay.ids)
        ep.M, ep.width, ep.scale, ep.x = M, W, cfg.embed_scale, x.data_ptr()
        ep.x0_k0 = -1
        if loop_op is not None:
            ep.x0, ep.x0_k0 = l_op, KW
        op, k0, norm_w, s0, op2, norm_w2 = target(runs[0])
        ep.op, ep.op_k0, ep.norm_w = op, k0, N.ptr(norm_w)
        if norm_w2 is not None:
            ep.op2, ep.norm_w2 = op2, norm_w2.data_ptr()
        ep.ss_out, ep.ss_out_n = N.ptr(s0), ss.shape[1]
        prog.stream_embed(ep, tag="embed")

        # ---- layers
        for i, run in enumerate(runs):
            lw, spec, t = w.layers[run.layer], cfg.layers[run.layer], f"R{run.index}.L{run.layer}"
            if run.enter is not None:                    # x <- W_in [x; x0] + step
                e = self._stream_epi(x, False, (h_op, 0, lw.norm, ss, None, None), bias=w.loop_step[run.enter])
                self._linear(prog, w.loop_in, loop_op, M, e, ws, f"{t}.loop_in")
            m_op = self._operand(mid, M, lw.out.K)
            e = N.LinEpi()
            self._row_norm(e, ss)
            e.out, e.ldo, e.n_plain, e.act_tile0 = proj.data_ptr(), ldp, lw.n_plain, lw.act_tile0
            e.bias = N.ptr(lw.bias)
            if spec.mlp is not None and cfg.parallel:
                e.act, e.act_k0, e.act_kind, e.limit, e.alpha = m_op, lw.act_k0, spec.mlp.act_kind, spec.mlp.limit, spec.mlp.alpha
                e.act_bias = N.ptr(lw.act_bias)
            if lw.lat_tiles:
                e.lat_tiles, e.lat_n, e.lat, e.lat_w = lw.lat_tiles, spec.mixer.q_rank, self._operand(work["lat"], M, lw.carry.K), lw.extra["dq_norm"].data_ptr()
                e.lat_ss, e.lat_ss_n = work["lat_ss"].data_ptr(), 2 * lw.lat_tiles
            self._linear(prog, lw.proj, h, M, e, ws, f"{t}.project", second=(h2, lw.tile2) if cfg.two_norms and spec.mlp is not None else None)
            if lw.experts_up is not None:
                self._experts(prog, lw, spec.mlp, h2, ss, proj.data_ptr() + 4 * lw.off["router"], proj.stride(0), M, at(lay.cu_rows + nseq), experts, ws, t)
            if lw.carry is not None:
                self._carry_queries(prog, lw, spec.mixer, work, M, ws, f"{t}.carry")
            self._mixers(prog, run, lw, spec.mixer, proj, m_op, M, nseq, lay, at, work, decode, t)
            nxt = runs[i + 1] if i + 1 < len(runs) else None
            tgt = target(nxt)
            if lw.up is None:
                e = self._stream_epi(x, True, tgt, bias=lw.out_bias)
                if lw.experts_up is not None:
                    e.y, e.slot_of, e.route_w = (experts[k].data_ptr() for k in ("y", "slot_of", "topk_w"))
                    e.routes, e.ldy, e.y_f32 = spec.mlp.top, L.round_up(W, 8), int(self.f32)
                self._linear(prog, lw.out, mid, M, e, ws, f"{t}.out")
            else:
                self._linear(prog, lw.out, mid, M, self._stream_epi(x, True, (h_op, 0, lw.norm2, ss, None, None)), ws, f"{t}.out")
                e = N.LinEpi()
                self._row_norm(e, ss)
                e.act, e.act_kind = self._operand(ff, M, lw.down.K), 1         # (squared ReLU)
                self._linear(prog, lw.up, h, M, e, ws, f"{t}.up")
                self._linear(prog, lw.down, ff, M, self._stream_epi(x, True, tgt), ws, f"{t}.down")
            if digests is not None:
                prog.digest(x, x.numel() * 4, digests.data_ptr() + 8 * run.index, tag=f"{t}.digest")
        b = self._head(prog, key, kind, nseq, width, M, lay, at, blob, blob_host, x, h, ss, ws, keep + [digests], seam, plp, capture)
        b.arenas = [a for a in (x, ss, h, h2, loop_op, mid, ff, proj) if a is not None]
        b.digests, b.x = digests, x
        return b

    def _mixers(self, prog, run, lw, mixer, proj, m_op, M, nseq, lay, at, work, decode, t: str) -> None:
        for pre, m, scale in mixer.parts():
            part, key, k0 = lw.part(pre), self._key(run, pre), lw.mix_k0[pre]
            if isinstance(m, DeltaMixer):
                prog.delta(self._delta_params(run, lw, m, proj, m_op, M, nseq, lay, at, work), decode, tag=f"{t}.delta")
            elif isinstance(m, ChannelDeltaMixer):
                prog.cdelta(self._cdelta_params(key, part, m, proj, m_op, k0, scale, M, nseq, lay, at, work), decode, tag=f"{t}.channel_delta")
            elif isinstance(m, OuterMixer):
                prog.ssd(self._outer_params(run, lw, m, proj, m_op, M, nseq, lay, at, work, decode), decode, tag=f"{t}.outer")
            elif isinstance(m, GroupedMixer):
                cache = self.kv[key if pre else self.cfg.pages_of(run)]
                prog.gqa(self._gqa_params(key, cache, part, m, proj, m_op, k0, scale, M, nseq, lay, at, work, decode), tag=f"{t}.attention")
            else:
                prog.mla(self._mla_params(run, lw, m, proj, m_op, M, nseq, lay, at, work, decode), tag=f"{t}.latent_attention")

    def _joined_layers(self, prog, M: int, nseq: int, decode: bool, lay, at, ar: dict) -> torch.Tensor:
        """Layers whose sublayers' results are normed ahead of the stream; returns the stream's buffer behind the last.  A row kernel
        that blends tokens reads the stream of neighbouring rows, so it writes another buffer than it reads."""
        cfg, w, dev = self.cfg, self.w, self.device
        W, KW, wide = cfg.width, L.round_up(cfg.width, 64), L.round_up(cfg.width, 8)
        x, ws, live = ar["x"], ar["ws"], at(lay.cu_rows + nseq)
        ar["x2"] = other = torch.zeros_like(x) if cfg.token_shift else x
        ar["y"] = y = torch.zeros(M, wide, dtype=torch.float32, device=dev)
        E = max([l.up_plain for l in w.layers], default=0)
        ar["logits"] = logits = torch.zeros(M, max(8, E), dtype=torch.float32, device=dev)
        h_op, experts = self._operand(ar["h"], M, KW), ar["experts"]

        def plain(out: torch.Tensor, n: int, lin: SW.Linear, bias=None) -> N.LinEpi:
            e = N.LinEpi()
            e.out, e.ldo, e.n_plain, e.act_tile0, e.bias = out.data_ptr(), out.stride(0), n, lin.N_pad // 256, N.ptr(bias)
            return e

        def join(tag: str, norm_w, result=None, run=None) -> None:
            """result: (post norm, whether `y` holds product rows, feed-forward with routed rows or None).  run: the layer run that
            reads the row (None: a feed-forward or the head)."""
            nonlocal x, other
            p = N.JoinParams()
            p.M, p.width, p.ldx, p.rows, p.nseq, p.n_slots = M, W, x.stride(0), self._join_rows(M, decode), nseq, self.n_slots
            if result is None:
                p.table, p.table_f32, p.vocab, p.ids, p.embed_scale = w.embed.data_ptr(), int(self.f32), cfg.vocab, at(lay.ids), cfg.embed_scale
            else:
                post, product, f = result
                p.post_w, p.mult = post.data_ptr(), cfg.residual_mult
                if product:
                    p.y, p.ldy = y.data_ptr(), y.stride(0)
                if f is not None:
                    p.routed, p.slot_of, p.route_w = (experts[k].data_ptr() for k in ("y", "slot_of", "topk_w"))
                    p.routes, p.ldr, p.routed_f32 = f.top, wide, int(self.f32)
            p.norm_w, p.op, p.eps, p.err = norm_w.data_ptr(), h_op, cfg.eps, self.scratch.err.data_ptr()
            p.x = p.x_out = x.data_ptr()
            p.cu_rows, p.slots, p.pos = at(lay.cu_rows), at(lay.slots), at(lay.pos)
            if run is not None:
                if run.enter is not None:
                    p.step = w.loop_step[run.enter].data_ptr()
                if cfg.token_shift:
                    p.shift, p.state, p.x_out = w.layers[run.layer].shift.data_ptr(), self.before[run.index].data_ptr(), other.data_ptr()
                    x, other = other, x
            prog.join(p, tag=tag)

        runs = cfg.runs
        join("embed", w.layers[runs[0].layer].norm, run=runs[0])
        for i, run in enumerate(runs):
            lw, spec, t = w.layers[run.layer], cfg.layers[run.layer], f"R{run.index}.L{run.layer}"
            e = plain(ar["proj"], lw.n_plain, lw.proj, lw.bias)
            self._linear(prog, lw.proj, ar["h"], M, e, ws, f"{t}.project")
            at0 = prog.num_ops
            self._mixers(prog, run, lw, spec.mixer, ar["proj"], self._operand(ar["mid"], M, lw.out.K), M, nseq, lay, at, ar["work"], decode, t)
            mixers = prog.num_ops - at0
            self._linear(prog, lw.out, ar["mid"], M, plain(y, wide, lw.out, lw.out_bias), ws, f"{t}.out")
            if decode and self.side_stream and mixers == 2:    # (they read the same rows and write columns of their own)
                prog.beside(at0, at0 + 1, at0 + 2)
            result, f = (lw.post1, True, None), spec.mlp
            if f is not None:
                join(f"{t}.join", lw.norm2, result)
                e = N.LinEpi()
                e.out, e.ldo, e.n_plain, e.act_tile0 = logits.data_ptr(), logits.stride(0), lw.up_plain, lw.up_tile0
                if lw.down is not None:
                    e.act, e.act_kind = self._operand(ar["ff"], M, lw.down.K), f.act_kind
                self._linear(prog, lw.up, ar["h"], M, e, ws, f"{t}.up")
                mix = f if isinstance(f, ExpertMix) else None
                if mix is not None:
                    self._experts(prog, lw, mix, ar["h"], None, logits.data_ptr() + 4 * lw.up_off["router"], logits.stride(0), M, live, experts, ws, t)
                if lw.down is not None:
                    self._linear(prog, lw.down, ar["ff"], M, plain(y, wide, lw.down), ws, f"{t}.down")
                result = (lw.post2, lw.down is not None, mix)
            nxt = runs[i + 1] if i + 1 < len(runs) else None
            join(f"{t}.{'end' if f is not None else 'join'}", w.final_norm if nxt is None else w.layers[nxt.layer].norm, result, nxt)
            if ar["digests"] is not None:
                prog.digest(x, x.numel() * 4, ar["digests"].data_ptr() + 8 * run.index, tag=f"{t}.digest")
        return x

    def _join_rows(self, M: int, decode: bool) -> int:
        """Rows of a CTA of the row kernel: several share the row ahead of them, while its rows fit."""
        if decode or M < 256:
            return 1
        return next((r for r in (4, 2) if (r + 2) * L.round_up(self.cfg.width, 4) * 4 <= 110 << 10), 1)

    # ---- routed experts
    def _expert_scratch(self, M: int) -> dict:
        """Routing tables and routed rows of a bucket, sized for the largest mixture.  Every expert's rows start at a multiple of 16."""
        ms = [l.mlp for l in self.cfg.layers if isinstance(l.mlp, ExpertMix)]
        if not ms:
            return {}
        dev, W = self.device, self.cfg.width
        i32 = lambda *s: torch.zeros(*s, dtype=torch.int32, device=dev)       # noqa: E731
        nt, mtiles = 64 if self.f32 else L.token_tile(M), 1
        if nt == 128 and M * max(f.top for f in ms) > 96 * max(f.experts for f in ms):     # a weight tile for 256 rows
            mtiles = 2
        tile = nt * mtiles
        per = [(M * f.top, min(f.experts, M * f.top)) for f in ms]            # routes, experts that can have one
        rows = L.round_up(max(r + 15 * e for r, e in per), 16)
        pad = L.round_up(rows, 128)
        top, E, ff = max(f.top for f in ms), max(f.experts for f in ms), max(L.round_up(f.ff, f.k_step) for f in ms)
        most = max(e + r // tile for r, e in per)
        return {"nt": nt, "mtiles": mtiles, "rows": rows, "pad": pad, "max_tiles": most, "tiles": i32(most, 4),
                "ntiles": i32(2), "src_row": i32(pad), "topk_id": i32(M * top), "slot_of": i32(M * top), "counts": i32(E), "offsets": i32(E + 1), "cursors": i32(E),
                "topk_w": torch.zeros(M * top, dtype=torch.float32, device=dev), "act": torch.zeros(pad * ff, dtype=self.dtype, device=dev),
                "y": torch.zeros(rows * L.round_up(W, 8), dtype=self.dtype, device=dev)}

    def _experts(self, prog, lw, f: ExpertMix, h2, ss, logits: int, ld: int, M: int, live, ew: dict, ws, tag: str) -> None:
        """Routes of the step, then the experts' rows; their weighted sum is left to the output linear or the row kernel.
        ss: sums of squares of the operand's rows (None: they are divided already)."""
        p = N.MoeRouteParams()
        p.logits_f32, p.ld, p.M, p.E, p.top_k = logits, ld, M, f.experts, f.top
        p.sigmoid, p.correction, p.scale = int(f.sigmoid), N.ptr(lw.correction), f.scale
        p.topk_id, p.topk_w, p.counts, p.offsets, p.cursors, p.tiles, p.ntiles, p.src_row, p.slot_of = \
            (ew[k].data_ptr() for k in ("topk_id", "topk_w", "counts", "offsets", "cursors", "tiles", "ntiles", "src_row", "slot_of"))
        p.nt, p.rows_cap, p.e_lo, p.e_n, p.live, p.groups, p.keep = ew["nt"] * ew["mtiles"], ew["src_row"].numel(), 0, f.experts, live, f.groups, f.keep
        prog.add_moe_route(p, tag=f"{tag}.route")
        e = N.LinEpi()
        if ss is not None:
            self._row_norm(e, ss)
        e.act, e.act_kind = N.Operand(ew["act"].data_ptr(), ew["pad"], lw.experts_down.K, int(self.f32)), f.expert_act_kind
        self._grouped_linear(prog, lw.experts_up, h2, L.padded_rows(M), ew, True, e, ws, f"{tag}.experts_up")
        e = N.LinEpi()
        e.out, e.ldo, e.n_plain, e.act_tile0 = ew["y"].data_ptr(), L.round_up(self.cfg.width, 8), L.round_up(self.cfg.width, 8), lw.experts_down.N_pad // 256
        e.out_bf16 = int(not self.f32)
        self._grouped_linear(prog, lw.experts_down, ew["act"], ew["pad"], ew, False, e, ws, f"{tag}.experts_down")

    # ---- mixers
    def _carry_queries(self, prog, lw, m: LatentMixer, wk: dict, M: int, ws, tag: str) -> None:
        """Queries from their normed latent (its rows were left undivided, like the stream's)."""
        e = N.LinEpi()
        e.ss, e.ss_n, e.inv_width, e.eps = wk["lat_ss"].data_ptr(), 2 * lw.lat_tiles, 1.0 / m.q_rank, self.cfg.eps
        e.out, e.ldo, e.n_plain, e.act_tile0 = wk["queries"].data_ptr(), wk["queries"].stride(0), m.query_rows, lw.carry.N_pad // 256
        self._linear(prog, lw.carry, wk["lat"], M, e, ws, tag)

    def _mixer_scratch(self, M: int, nseq: int, decode: bool) -> dict:
        """Scratch shared by the layers of a bucket, sized for the largest of them."""
        f32 = lambda n: torch.zeros(max(1, n), dtype=torch.float32, device=self.device)   # noqa: E731
        ms = self.cfg.mixers()
        de, la = [m for m in ms if isinstance(m, (DeltaMixer, OuterMixer))], [m for m in ms if isinstance(m, LatentMixer)]
        outer, gr = [m for m in ms if isinstance(m, OuterMixer)], [m for m in ms if isinstance(m, GroupedMixer)]
        mx = lambda it: max(it, default=0)    # noqa: E731
        wk = {"splits": self._splits(M, decode)}
        if not decode:
            floats = {id(m): self._chunk_floats(m, M, nseq) for m in outer}
            scan = [m for m in de if not floats.get(id(m))]
            blk = M // 4 + nseq                           # blocks of four tokens
            wk["kq"] = f32(blk * mx(m.kv_heads * (8 * m.dim_pad + 16) for m in scan))
            wk["vb"] = f32(blk * mx(m.heads * ((m.vdim_pad + 15) // 16) * 72 for m in scan))
            wk["o"] = f32(M * mx(m.heads * m.vdim_pad for m in de))
            wk["chunk"] = f32(mx(floats.values()))
        elif outer:
            wk["o"] = f32(M * mx(m.heads * m.vdim_pad for m in outer))
        cd, conv = [m for m in ms if isinstance(m, ChannelDeltaMixer)], [m for m in gr if m.taps]
        if cd and not decode:
            blk = M // 4 + nseq
            wk["cd_rec"] = f32(blk * mx(m.heads * (17 * m.dim_pad + 64) for m in cd))
            wk["cd_v"] = f32(blk * mx(m.heads * ((m.vdim_pad + 31) // 32) * 128 for m in cd))
            wk["cd_o"] = f32(M * mx(m.heads * m.vdim_pad for m in cd))
        if conv:
            wk["conv_x"], wk["conv_ss"] = f32(M * mx(self._conv_width(m) for m in conv)), f32(M * mx(self._conv_parts(m) for m in conv))
        if outer or gr:                                   # arrivals at the end of a row: zero between launches
            wk["counters"] = torch.zeros(max(nseq * mx(m.norm_groups for m in outer), M * mx(m.kv_heads for m in gr)), dtype=torch.int32, device=self.device)
        if gr:
            split = [m for m in gr if self._gqa_form(m, M, decode) == 1]
            sp = {id(m): self._gqa_splits(m, M) for m in split}
            wk["gqa_q"] = torch.zeros(max(1, M * mx(m.heads * m.score_dim for m in gr if self._gqa_form(m, M, decode) == 2)), dtype=self.dtype,
                                      device=self.device)
            wk["gqa_o"] = f32(M * mx(m.heads * m.vdim_pad * sp[id(m)] for m in split))
            wk["gqa_ml"] = f32(M * mx(2 * m.heads * sp[id(m)] for m in split))
        carried = [m for m in la if m.q_rank]
        if carried:
            wk["lat"] = self._operand_buf(M, max(m.q_rank for m in carried))
            wk["lat_ss"] = f32(L.padded_rows(M) * 2 * mx((m.q_rank + 255) // 256 for m in carried))
            wk["queries"] = f32(M * mx(L.round_up(m.query_rows, 8) for m in carried)).view(M, -1)
        wk["q_eff"] = torch.zeros(max(1, M * mx(m.heads * (max(m.rank_pad, m.dim_pad) + m.rot_pad) for m in la)), dtype=self.dtype, device=self.device)
        absorbed = [m for m in la if not self._expanded(m, M, decode)]
        if absorbed:
            wk["o_part"] = f32(M * wk["splits"] * mx(m.heads * m.rank_pad for m in absorbed))
            wk["ml"] = f32(M * wk["splits"] * mx(2 * m.heads for m in absorbed))
        return wk

    def _expanded(self, m: LatentMixer, M: int, decode: bool) -> int:
        """Prompt portions attend over expanded keys and values; decoding, short portions and fp32 in the latent space."""
        if decode or M < 64 or self.k_exp is None:
            return 0
        p = N.MlaParams()
        p.f32, p.page, p.VP, p.DP, p.RP, p.CP, p.scale = int(self.f32), self.cfg.page_tokens, m.vdim_pad, m.dim_pad, m.rot_pad, m.rank_pad, m.scale
        form = N.lib().saber_mla_expand_ok(C.byref(p))       # 2: tcgen05, 1: mma.sync, 0: neither takes these sizes
        return form if self.attn_impl == "tc" else min(form, 1)

    def _splits(self, M: int, decode: bool) -> int:
        """Key splits of the absorbed attention: fill the SMs once."""
        return max(1, min(32, F.device_sms() // max(1, M))) if decode or M < 64 else 1

    def _chunk_floats(self, m: OuterMixer, M: int, nseq: int) -> int:
        """Scratch of the chunk form for prompt portions (0: the scan serves: fp32, or sizes it does not take)."""
        if self.f32:
            return 0
        p = N.SsdParams()
        p.M, p.nseq, p.H, p.HK, p.N, p.DP, p.V, p.VP, p.taps = M, nseq, m.heads, m.kv_heads, m.dim, m.dim_pad, m.vdim, m.vdim_pad, m.taps
        return N.lib().saber_ssd_chunk_floats(C.byref(p))

    def _gqa_sizes(self, m: GroupedMixer) -> N.GqaParams:
        p = N.GqaParams()
        p.H, p.G, p.D, p.DK, p.KP, p.V, p.VP = m.heads, m.kv_heads, m.dim, m.score_dim, m.key_pad, m.vdim, m.vdim_pad
        p.page, p.f32, p.scale, p.softcap = self.cfg.page_tokens, int(self.f32), m.scale, m.softcap
        if m.rot is not None:
            p.rot, p.rot_amp = m.rot.dims, m.rot.amplitude
        return p

    def _gqa_form(self, m: GroupedMixer, M: int, decode: bool) -> int:
        """2: tcgen05 (prompt portions), 1: split keys on mma.sync, 0: any size on the CUDA cores."""
        form = N.lib().saber_gqa_form(C.byref(self._gqa_sizes(m)))
        return min(form, 2 if (self.attn_impl == "tc" and not decode and M >= 64) else 1)

    def _gqa_splits(self, m: GroupedMixer, M: int) -> int:
        """Key splits: fill the SMs twice, never more parts than pages a row can see."""
        part = m.chunk or m.window                        # keys a row sees at most
        span = self.max_ctx if part == 0 else min(self.max_ctx, part + self.cfg.page_tokens - 1)
        pages = (span + self.cfg.page_tokens - 1) // self.cfg.page_tokens
        return max(1, min(32, pages, 2 * F.device_sms() // max(1, M * m.kv_heads)))

    def _outer_params(self, run, lw, m: OuterMixer, proj, m_op, M, nseq, lay, at, wk, decode) -> N.SsdParams:
        p, x = N.SsdParams(), lw.extra
        p.x, p.ldx = proj.data_ptr(), proj.stride(0)
        p.q_off, p.k_off, p.v_off, p.g_off, p.dt_off = lw.off["q"], lw.off["k"], lw.off["v"], lw.off["g"], lw.off.get("dt", -1)
        p.conv_w, p.conv_b, p.decay, p.A_log, p.dt_bias, p.skip = (N.ptr(x.get(k)) for k in ("conv", "conv_b", "decay", "A_log", "dt_bias", "D"))
        p.norm_w, p.state, p.hist = x["norm"].data_ptr(), self.state[run.index].data_ptr(), N.ptr(self.hist.get(run.index))
        p.kq, p.vb, p.o, p.counters = N.ptr(wk.get("kq")), N.ptr(wk.get("vb")), wk["o"].data_ptr(), wk["counters"].data_ptr()
        if not decode and self._chunk_floats(m, M, nseq):
            p.chunk = wk["chunk"].data_ptr()
        p.cu_rows, p.slots, p.pos = at(lay.cu_rows), at(lay.slots), at(lay.pos)
        p.out, p.out_k0, p.M, p.nseq = m_op, 0, M, nseq
        p.H, p.HK, p.N, p.DP, p.V, p.VP, p.taps, p.n_slots = m.heads, m.kv_heads, m.dim, m.dim_pad, m.vdim, m.vdim_pad, m.taps, self.n_slots
        p.groups, p.gate_first, p.eps, p.err = m.norm_groups, int(m.gate_first), self.cfg.eps, self.scratch.err.data_ptr()
        return p

    @staticmethod
    def _conv_width(m: GroupedMixer) -> int:
        """Columns of the convolved rows: q | k | v, each from a multiple of 8 on."""
        return sum(L.round_up(n, 8) for name, n in m.segments() if name != "g")

    @staticmethod
    def _conv_parts(m: GroupedMixer) -> int:
        """Partial sums of squares of a convolved row: 256 columns of q, then of k."""
        return sum((n + 255) // 256 for name, n in m.segments() if name in ("q", "k"))

    def _cdelta_params(self, key, lw, m: ChannelDeltaMixer, proj, m_op, k0, scale, M, nseq, lay, at, wk) -> N.CdeltaParams:
        p, x = N.CdeltaParams(), lw.extra
        p.x, p.ldx = proj.data_ptr(), proj.stride(0)
        p.r_off, p.k_off, p.v_off, p.a_off, p.l_off, p.g_off = (lw.off[k] for k in ("r", "k", "v", "a", "w1", "g"))
        p.w2, p.w2_f32, p.rank, p.w0, p.norm_w = x["w2"].data_ptr(), int(self.f32), m.rank, x["w0"].data_ptr(), x["norm"].data_ptr()
        p.state = self.state[key].data_ptr()
        p.rec, p.vb, p.o = (N.ptr(wk.get(k)) for k in ("cd_rec", "cd_v", "cd_o"))
        p.cu_rows, p.slots, p.pos = at(lay.cu_rows), at(lay.slots), at(lay.pos)
        p.out, p.out_k0, p.out_scale, p.M, p.nseq = m_op, k0, scale, M, nseq
        p.H, p.D, p.DP, p.VP, p.n_slots = m.heads, m.dim, m.dim_pad, m.vdim_pad, self.n_slots
        p.eps, p.unit_eps, p.err = self.cfg.eps, m.unit_eps, self.scratch.err.data_ptr()
        return p

    def _gqa_params(self, key, cache, lw, m: GroupedMixer, proj, m_op, k0, scale, M, nseq, lay, at, wk, decode) -> N.GqaParams:
        p = self._gqa_sizes(m)
        p.x, p.ldx = proj.data_ptr(), proj.stride(0)
        p.q_off, p.k_off, p.v_off, p.g_off = lw.off["q"], lw.off.get("k", -1), lw.off.get("v", -1), lw.off.get("g", -1)
        p.freq, p.sink = N.ptr(lw.extra.get("freq")), N.ptr(lw.extra.get("sink"))
        p.cache, p.q = cache.data_ptr(), wk["gqa_q"].data_ptr()
        p.window, p.out_scale, p.taps = m.window, scale, m.taps
        if m.taps:
            p.conv_w, p.q_w, p.k_w = (lw.extra[k].data_ptr() for k in ("conv", "q_norm", "k_norm"))
            p.hist, p.slots, p.n_slots, p.v_norm = self.hist[key].data_ptr(), at(lay.slots), self.n_slots, 1
            p.cx, p.ldc, p.row_ss = wk["conv_x"].data_ptr(), self._conv_width(m), wk["conv_ss"].data_ptr()
        p.o_part, p.ml, p.counters = wk["gqa_o"].data_ptr(), wk["gqa_ml"].data_ptr(), wk["counters"].data_ptr()
        p.slot_map, p.pos, p.cu_rows, p.kv_len, p.block_table = (at(o) for o in (lay.slot_map, lay.pos, lay.cu_rows, lay.kv_len, lay.block_table))
        p.out, p.out_k0, p.M, p.nseq = m_op, k0, M, nseq
        p.n_blocks, p.max_blocks, p.max_rows = self.kv_blocks, self.max_blocks, 1 if decode else M
        p.form = self._gqa_form(m, M, decode)
        p.splits = self._gqa_splits(m, M) if p.form == 1 else 1
        p.qk_norm, p.chunk, p.eps, p.err = int(m.qk_norm), m.chunk, self.cfg.eps, self.scratch.err.data_ptr()
        return p

    def _delta_params(self, run, lw, m: DeltaMixer, proj, m_op, M, nseq, lay, at, wk) -> N.DeltaParams:
        p = N.DeltaParams()
        p.x, p.ldx = proj.data_ptr(), proj.stride(0)
        p.q_off, p.k_off, p.v_off, p.b_off, p.a_off, p.g_off = (lw.off[k] for k in ("q", "k", "v", "b", "a", "g"))
        p.conv_w, p.A_log, p.dt_bias, p.norm_w = (lw.extra[k].data_ptr() for k in ("conv", "A_log", "dt_bias", "norm"))
        p.hist, p.state = self.hist[run.index].data_ptr(), self.state[run.index].data_ptr()
        p.kq, p.vb, p.o = (N.ptr(wk.get(k)) for k in ("kq", "vb", "o"))
        p.cu_rows, p.slots, p.pos = at(lay.cu_rows), at(lay.slots), at(lay.pos)
        p.out, p.out_k0, p.M, p.nseq = m_op, 0, M, nseq
        p.H, p.HK, p.D, p.DP, p.V, p.VP, p.taps, p.n_slots = m.heads, m.kv_heads, m.dim, m.dim_pad, m.vdim, m.vdim_pad, m.taps, self.n_slots
        p.eps, p.unit_eps, p.q_scale = self.cfg.eps, m.unit_eps, m.dim ** -0.5
        p.err = self.scratch.err.data_ptr()
        return p

    def _mla_params(self, run, lw, m: LatentMixer, proj, m_op, M, nseq, lay, at, wk, decode) -> N.MlaParams:
        p = N.MlaParams()
        p.x, p.ldx = proj.data_ptr(), proj.stride(0)
        p.q_off, p.dkv_off, p.g_off, p.q, p.ldq = lw.off.get("q", 0), lw.off.get("dkv", -1), lw.off["g"], proj.data_ptr(), proj.stride(0)
        if m.q_rank:
            p.q, p.ldq = wk["queries"].data_ptr(), wk["queries"].stride(0)
        p.gate_heads, p.interleaved, p.rot_amp = int(m.gate_heads), int(m.rot.interleaved), m.rot.amplitude
        p.dkv_norm, p.freq, p.w_uk, p.w_uv = (N.ptr(lw.extra.get(k)) for k in ("dkv_norm", "freq", "uk", "uv"))
        p.cache, p.q_eff = self.kv[self.cfg.pages_of(run)].data_ptr(), wk["q_eff"].data_ptr()
        p.o_part, p.ml = N.ptr(wk.get("o_part")), N.ptr(wk.get("ml"))
        p.k_exp, p.v_exp = N.ptr(self.k_exp), N.ptr(self.v_exp)
        p.slot_map, p.pos, p.cu_rows, p.kv_len, p.block_table = (at(o) for o in (lay.slot_map, lay.pos, lay.cu_rows, lay.kv_len, lay.block_table))
        p.out, p.out_k0, p.M, p.nseq = m_op, 0, M, nseq
        p.H, p.D, p.R, p.V, p.C, p.CP, p.RP, p.DP, p.VP = m.heads, m.dim, m.rot_dim, m.vdim, m.kv_rank, m.rank_pad, m.rot_pad, m.dim_pad, m.vdim_pad
        p.page, p.n_blocks, p.max_blocks = self.cfg.page_tokens, self.kv_blocks, self.max_blocks
        p.splits, p.f32, p.expand, p.max_rows = wk["splits"], int(self.f32), self._expanded(m, M, decode), 1 if decode else M
        p.scale, p.eps, p.err = m.scale, self.cfg.eps, self.scratch.err.data_ptr()
        return p

    # ---- head and sampling
    def _head(self, prog, key, kind, nseq, width, M, lay, at, blob, blob_host, x, h, ss, ws, keep, seam, plp, capture) -> Bucket:
        cfg, dev, w = self.cfg, self.device, self.w
        decode = kind == "decode"
        Mh = M if decode else nseq
        KW, V = L.round_up(cfg.width, 64), cfg.vocab
        ldv = L.round_up(V, 8)
        out, o_commit, o_tokens, o_picks = head_outputs(nseq, 1, 0, Mh, dev)
        logits = torch.zeros(Mh, ldv, dtype=torch.float32, device=dev)
        pick_val = torch.zeros(Mh, dtype=torch.float32, device=dev)

        def head(a, rows, dst, normed: bool, tag):
            e = N.LinEpi()
            if not normed and ss is not None:            # (the row kernel has divided its rows already)
                self._row_norm(e, ss)
            e.out, e.ldo, e.n_plain, e.act_tile0, e.cap = dst.data_ptr(), dst.stride(0), V, w.head.N_pad // 256, cfg.logit_cap
            self._linear(prog, w.head, a, rows, e, ws, tag)

        if decode:
            head(h, M, logits, False, "lm_head")
        else:
            last = self._operand_buf(nseq, KW)
            np_ = N.StreamNormParams()
            np_.x, np_.ldx, np_.width, np_.n, np_.rows = x.data_ptr(), x.stride(0), cfg.width, nseq, at(lay.last_rows)
            np_.w, np_.eps, np_.op = w.final_norm.data_ptr(), cfg.eps, self._operand(last, nseq, KW)
            prog.stream_norm(np_, tag="final_norm.last_rows")
            head(last, nseq, logits, True, "lm_head")
            keep.append(last)
        prog.argmax(logits, Mh, ldv, V, 0, o_picks, pick_val, tag="argmax")
        seam_dev = None
        if seam:
            seam_dev, s_ids, s_vals, s_lse = seam_outputs(Mh, dev)
            prog.seam(logits, Mh, ldv, V, 0, None, s_ids, s_vals, s_lse, tag="topk_seam")
            prog.sample_seam(s_ids, s_vals, at(lay.samp), at(lay.samp_u), o_picks, Mh, tag="sample_seam")
        plp_dev = plp_logits = None
        if plp:
            plp_logits = torch.zeros(M, ldv, dtype=torch.float32, device=dev)
            plp_dev, p_ids, p_vals, p_lse, p_next = plp_outputs(M, dev)
            head(h, M, plp_logits, False, "plp.lm_head")
            if V >= N.SEAM_K:
                prog.seam(plp_logits, M, ldv, V, 0, None, p_ids, p_vals, p_lse, tag="plp.topk_seam")
            prog.logit_gather(plp_logits, M, ldv, V, 0, at(lay.next_ids), p_next, tag="plp.logit_gather")
        if decode:
            vp = N.VerifyParams()
            vp.draft, vp.target, vp.cu_rows = at(lay.ids), o_picks.data_ptr(), at(lay.cu_rows)
            vp.seq_uid, vp.step_no = at(lay.seq_uid), at(lay.step_no)
            vp.n_commit, vp.out_tokens = o_commit.data_ptr(), o_tokens.data_ptr()
            vp.accept_row, vp.bonus = None, None
            vp.nseq, vp.max_w, vp.oracle_p, vp.seed = nseq, 1, 0.0, 0
            prog.verify(vp, tag="commit")
        return finish_bucket(self, prog, key, kind, nseq, width, M, lay, blob, blob_host, keep + [pick_val], capture,
                             dict(out=out, logits=logits, W=1, block=0, Mh=Mh, seam=seam_dev, plp=plp_dev, plp_logits=plp_logits))
