"""Weights of a layer-by-layer decoder: the tensors by name and shape, the safetensors reader, and the device
layouts its kernels read.

Side by side (parallel residual), a layer needs two linears.  `proj` holds every row that reads the normed stream:
the mixer's segments (each starting at a multiple of 8 rows, the whole padded to 256; a latent that queries come from has
whole tiles of its own ahead of them), then the feed-forward's rows as tiles of 256: 128 gate and 128 up rows of the same
features, 256 up rows, or 248 up rows and the row of their gate.  `out` holds the mixer's output columns and the down
columns side by side, so that one product adds both sublayers to the stream.  Where the feed-forward reads a norm of its
own, its rows (a router's first) start at a tile of their own and multiply the second operand.  One after the other, `proj` and
`out` belong to the mixer alone and `up` and `down` to the feed-forward behind its own norm (a router's rows ahead of the shared
expert's).  Mixers side by side share `proj` and `out`, part after part.  The routed experts of a mixture are stacks of tiles,
expert after expert.
"""
from __future__ import annotations

import dataclasses
import json
import math
import mmap
import struct
from dataclasses import dataclass, field
from pathlib import Path
from typing import Callable, Optional

import torch

from ..ops import layouts as L
from .stack_config import ChannelDeltaMixer, ClampedGlu, DeltaMixer, ExpertMix, Gelu, GroupedMixer, LatentMixer, OuterMixer, StackConfig

_ST_DTYPES = {"BF16": torch.bfloat16, "F32": torch.float32, "F16": torch.float16, "I32": torch.int32, "I64": torch.int64}


def read_safetensors(path) -> dict:
    """Every tensor of a safetensors file (8-byte header length, JSON header, data), by name."""
    with open(path, "rb") as f:
        mm = mmap.mmap(f.fileno(), 0, access=mmap.ACCESS_READ)
    (n,) = struct.unpack("<Q", mm[:8])
    out = {}
    for name, d in json.loads(mm[8:8 + n]).items():
        if name == "__metadata__":
            continue
        if d["dtype"] not in _ST_DTYPES:
            raise ValueError(f"{path}: tensor {name!r} has dtype {d['dtype']}")
        lo, hi = d["data_offsets"]
        raw = bytearray(mm[8 + n + lo: 8 + n + hi])
        out[name] = torch.frombuffer(raw, dtype=_ST_DTYPES[d["dtype"]]).reshape(d["shape"]) if raw else \
            torch.zeros(d["shape"], dtype=_ST_DTYPES[d["dtype"]])
    return out


def tensor_shapes(cfg: StackConfig) -> dict:
    """Tensor names and shapes."""
    w, t = cfg.width, {"embed": (cfg.vocab, cfg.width)}
    if cfg.loop is not None:
        if cfg.loop_linear:
            t["loop.in"] = (w, 2 * w)
        t["loop.step"] = (cfg.loop.times, w)
    for i, l in enumerate(cfg.layers):
        p, m = f"l{i}.", l.mixer
        rows, bias = dict(m.segments()), m.biases()
        t[p + "norm1"] = (w,)
        if cfg.post_norms:
            t[p + "norm1b"] = (w,)
        if cfg.token_shift:
            t[p + "shift"] = (w,)
        for seg, tensor, first in m.sources():
            have = t.get(f"{p}mix.{tensor}", (0, w))[0]
            t[f"{p}mix.{tensor}"] = (max(have, first + rows[seg]), w)
            if seg in bias:
                t[f"{p}mix.{tensor}.b"] = (rows[seg],)
        for name, shape in m.extra_shapes().items():
            t[f"{p}mix.{name}"] = shape
        for name, features, has_bias in m.out_tensors():
            t[f"{p}mix.{name}"] = (w, features)
            if has_bias:
                t[f"{p}mix.{name}.b"] = (w,)
        if l.mlp is not None:
            if not cfg.parallel or cfg.two_norms:
                t[p + "norm2"] = (w,)
            if cfg.post_norms:
                t[p + "norm2b"] = (w,)
            t.update({f"{p}mlp.{name}": shape for name, shape in l.mlp.shapes(w).items()})
    t["final.norm"], t["head"] = (w,), (cfg.vocab, w)
    return t


def random_tensor(name: str, shape: tuple, g: torch.Generator, device, norm_offset: float = 0.0) -> torch.Tensor:
    leaf = name.rsplit(".", 1)[-1]
    if leaf in ("norm1", "norm2", "norm", "norm1b", "norm2b"):
        around = norm_offset if ".mix." not in name else 0.0            # (a mixer's own norm is stored plain)
        return torch.full(shape, 1.0 - around, dtype=torch.bfloat16, device=device)
    if leaf in ("D", "sink"):
        return torch.ones(shape, dtype=torch.bfloat16, device=device)
    if leaf in ("b", "correction"):
        return torch.zeros(shape, dtype=torch.bfloat16, device=device)
    if leaf == "shift":
        return torch.rand(shape, generator=g, device=device).bfloat16()
    if leaf == "w0":
        return (torch.rand(shape, generator=g, device=device) * 6 - 7).bfloat16()
    if leaf == "A_log":
        return torch.log(torch.rand(shape, generator=g, device=device) * 15 + 1).bfloat16()
    if leaf == "dt_bias":
        dt = torch.exp(torch.rand(shape, generator=g, device=device) * math.log(100.0) + math.log(1e-3))
        return torch.log(torch.expm1(dt)).bfloat16()
    std = 0.02 if name in ("embed", "loop.step") else 1.0 / math.sqrt(shape[-1])
    return (torch.randn(shape, generator=g, device=device) * std).bfloat16()


@dataclass
class Linear:
    """A weight in the order its kernel reads: bf16 tiles [N_pad/256][K/64][32 KiB] or fp32 rows [N_pad][K]."""
    w: torch.Tensor
    N_pad: int
    K: int

    def nbytes(self) -> int:
        return self.w.numel() * self.w.element_size()


@dataclass
class StackLayer:
    norm: torch.Tensor
    proj: Linear
    out: Linear
    off: dict                        # segment name -> first column of the projection
    n_plain: int                     # columns of the projection's stored part
    act_tile0: int                   # first feed-forward tile
    act_k0: int                      # first feed-forward column of `out`'s operand
    extra: dict = field(default_factory=dict)
    bias: Optional[torch.Tensor] = None     # fp32, of the projection's stored columns
    norm2: Optional[torch.Tensor] = None    # the feed-forward's own norm
    up: Optional[Linear] = None             # feed-forward behind the mixer: its linears
    down: Optional[Linear] = None
    tile2: int = 0                          # first tile of the rows behind norm2 (side by side)
    lat_tiles: int = 0                      # tiles of the latent that queries come from
    carry: Optional[Linear] = None          # the linear from that latent to the queries
    act_bias: Optional[torch.Tensor] = None # fp32, of the feed-forward's rows
    out_bias: Optional[torch.Tensor] = None # fp32, of `out`
    experts_up: Optional[Linear] = None     # stacks of routed experts: N_pad and K of one
    experts_down: Optional[Linear] = None
    up_off: dict = field(default_factory=dict)      # stored columns of `up` (a router's)
    up_plain: int = 0
    up_tile0: int = 0                       # first tile of its activations
    post1: Optional[torch.Tensor] = None    # norms of the sublayers' results (these and the rows below padded to 8)
    post2: Optional[torch.Tensor] = None
    shift: Optional[torch.Tensor] = None    # blend with the token before
    correction: Optional[torch.Tensor] = None
    mix_k0: dict = field(default_factory=dict)      # part of the mixer -> first column of `out`'s operand

    def part(self, prefix: str) -> "StackLayer":
        """One of the mixers side by side: its own names in `off` and `extra`."""
        if not prefix:
            return self
        own = lambda d: {k[len(prefix):]: v for k, v in d.items() if k.startswith(prefix)}     # noqa: E731
        return dataclasses.replace(self, off=own(self.off), extra=own(self.extra))

    def linears(self) -> list:
        return [x for x in (self.proj, self.out, self.up, self.down, self.carry, self.experts_up, self.experts_down) if x is not None]


@dataclass
class StackWeights:
    embed: torch.Tensor
    layers: list
    final_norm: torch.Tensor
    head: Linear
    loop_in: Optional[Linear] = None
    loop_step: Optional[torch.Tensor] = None

    def nbytes(self) -> int:
        tot = self.embed.numel() * self.embed.element_size() + self.head.nbytes() + (self.loop_in.nbytes() if self.loop_in else 0)
        for l in self.layers:
            tot += sum(x.nbytes() for x in l.linears()) + sum(t.numel() * t.element_size() for t in l.extra.values())
        return tot


def pack_linear(rows: torch.Tensor, dtype: torch.dtype) -> Linear:
    """rows [N_pad, K] (N_pad a multiple of 256, K of 64)."""
    n, k = rows.shape
    assert n % 256 == 0 and k % 64 == 0, (n, k)
    if dtype == torch.float32:
        return Linear(rows.float().contiguous(), n, k)
    return Linear(L.tile_weight_int8(rows.to(torch.bfloat16).contiguous().view(torch.int8).reshape(n, k * 2)), n, k)


def pack_experts(rows: torch.Tensor, dtype: torch.dtype) -> Linear:
    """rows [experts, N_pad, K]: one expert's tiles after the other's."""
    e, n, k = rows.shape
    return Linear(pack_linear(rows.reshape(e * n, k), dtype).w, n, k)


@dataclass
class ProjectLayout:
    off: dict            # segment -> first row
    n_plain: int         # rows whose results are stored
    tile2: int           # first tile behind the second norm
    tile0: int           # first feed-forward tile
    rows: int            # in all
    lat_tiles: int


def project_layout(mixer, mlp, two_norms: bool = False) -> ProjectLayout:
    """mlp: the feed-forward beside the mixer, or None."""
    off, n, lat = {}, 0, 0
    for i, (name, rows) in enumerate(mixer.segments()):
        off[name] = n
        n = (n + rows + 7) // 8 * 8
        if i == 0 and mixer.q_rank:
            n = L.round_up(n, 256)
            lat = n // 256
    tile2 = (n + 255) // 256
    if two_norms and isinstance(mlp, ExpertMix):
        off["router"] = tile2 * 256
        n = (off["router"] + mlp.experts + 7) // 8 * 8
    tile0 = (n + 255) // 256
    return ProjectLayout(off, n, tile2, tile0, (tile0 + (mlp.tiles if mlp is not None else 0)) * 256, lat)


def gated_rows(gate: torch.Tensor, up: torch.Tensor, KW: int) -> torch.Tensor:
    """gate, up [ff, width] -> [tiles * 256, KW]: tiles of 128 gate and 128 up rows of the same features."""
    ff, W = gate.shape
    out = torch.zeros(L.round_up(ff, 128), 2, KW, dtype=gate.dtype, device=gate.device)
    out[:ff, 0, :W], out[:ff, 1, :W] = gate, up
    return out.view(-1, 128, 2, KW).transpose(1, 2).reshape(-1, KW)


def build(cfg: StackConfig, get: Callable[[str], torch.Tensor], dtype: torch.dtype, device) -> StackWeights:
    """Device layouts from `get(name)` (a tensor of the shape in `tensor_shapes`)."""
    dev = torch.device(device)
    shapes = tensor_shapes(cfg)

    def t(name: str) -> torch.Tensor:
        x = get(name)
        if tuple(x.shape) != tuple(shapes[name]):
            raise ValueError(f"tensor {name!r} has shape {tuple(x.shape)}, expected {tuple(shapes[name])}")
        return x.to(dev)

    f32 = lambda name: t(name).float().contiguous()                    # noqa: E731
    norm = lambda name: (f32(name) + cfg.norm_offset).contiguous()    # noqa: E731
    W = cfg.width
    KW, NW = L.round_up(W, 64), L.round_up(W, 256)
    zeros = lambda n, k: torch.zeros(n, k, dtype=torch.bfloat16 if dtype != torch.float32 else torch.float32, device=dev)   # noqa: E731
    wide = L.round_up(W, 8)

    def row(name: str) -> torch.Tensor:
        """A vector of the stream's width, zeros up to a multiple of 8."""
        out = torch.zeros(wide, dtype=torch.float32, device=dev)
        out[:W] = f32(name)
        return out

    def experts(p: str, f: ExpertMix) -> tuple:
        """The stacks of a mixture's routed experts."""
        eu = zeros(f.experts, (L.round_up(f.ff, 128) * 2 if f.gated else L.round_up(f.ff, 256)) * KW).view(f.experts, -1, KW)
        ed = zeros(f.experts, NW * L.round_up(f.ff, f.k_step)).view(f.experts, NW, -1)
        for e in range(f.experts):
            if f.gated:
                eu[e] = gated_rows(t(f"{p}mlp.e{e}.gate").to(eu.dtype), t(f"{p}mlp.e{e}.up").to(eu.dtype), KW)
            else:
                eu[e, : f.ff, :W] = t(f"{p}mlp.e{e}.up")
            ed[e, :W, : f.ff] = t(f"{p}mlp.e{e}.down")
        return pack_experts(eu, dtype), pack_experts(ed, dtype)

    def mixer_tensors(m, p: str) -> tuple:
        """Tensors beside the projections as a mixer's kernels read them, and the linear from a query latent."""
        extra, carry = {}, None
        if isinstance(m, DeltaMixer):
            extra["conv"] = torch.cat([f32(f"{p}{n}.conv") for n in ("q", "k", "v")]).contiguous()
            for n in ("A_log", "dt_bias", "norm"):
                extra[n] = f32(f"{p}{n}")
        elif isinstance(m, OuterMixer):
            for n in ("norm", *(("A_log", "dt_bias", "D") if m.decay is None else ())):
                extra[n] = f32(f"{p}{n}")
            if m.decay is not None:
                extra["decay"] = torch.tensor(m.decay, dtype=torch.float32, device=dev)
            if m.taps:                                                 # stored v | k | q, read q | k | v
                kd, vd = m.kv_heads * m.dim, m.heads * m.vdim
                for n, key in (("conv", "conv"), ("conv.b", "conv_b")):
                    c = f32(f"{p}{n}")
                    extra[key] = torch.cat([c[vd + kd:], c[vd: vd + kd], c[:vd]]).contiguous()
        elif isinstance(m, LatentMixer):
            if m.kv_from is None:
                extra["dkv_norm"] = f32(p + "dkv.norm")
            if m.q_rank:
                extra["dq_norm"] = f32(p + "dq.norm")
                c = zeros(L.round_up(m.query_rows, 256), L.round_up(m.q_rank, 64))
                c[: m.query_rows, : m.q_rank] = t(p + "uq")
                carry = pack_linear(c, dtype)
            for n in ("uk", "uv"):                                     # row stride: the padded latent
                full = t(f"{p}{n}")
                extra[n] = torch.zeros(full.shape[0], m.rank_pad, dtype=dtype, device=dev)
                extra[n][:, : m.kv_rank] = full
        elif isinstance(m, GroupedMixer):
            if m.sink:
                extra["sink"] = f32(p + "sink")
            if m.taps:
                extra["conv"] = torch.cat([f32(f"{p}{n}.conv") for n in ("q", "k", "v")]).T.contiguous()     # [tap][channel]
                extra["q_norm"], extra["k_norm"] = f32(p + "q.norm"), f32(p + "k.norm")
        elif isinstance(m, ChannelDeltaMixer):
            extra["w2"] = torch.zeros(m.out_features, L.round_up(m.rank, 16), dtype=dtype, device=dev)
            extra["w2"][:, : m.rank] = t(p + "w2")
            extra["w0"], extra["norm"] = f32(p + "w0"), f32(p + "norm")
        if getattr(m, "rot", None) is not None:
            extra["freq"] = torch.tensor(m.rot.frequencies() or [1.0], dtype=torch.float32, device=dev)
        return extra, carry

    def gated_feed_forward(lw: StackLayer, p: str, f) -> None:
        """`up`: a router's rows as stored columns, then tiles of gate and up rows; `down`."""
        mix, at = isinstance(f, ExpertMix), "shared." if isinstance(f, ExpertMix) else ""
        if mix:
            lw.up_off, lw.up_plain = {"router": 0}, L.round_up(f.experts, 8)
            lw.experts_up, lw.experts_down = experts(p, f)
            lw.correction = f32(p + "mlp.correction") if f.sigmoid else None
        lw.up_tile0 = (lw.up_plain + 255) // 256
        u = zeros((lw.up_tile0 + (f.tiles if f.inner else 0)) * 256, KW)
        if mix:
            u[: f.experts, :W] = t(p + "mlp.router")
        if f.inner:
            u[lw.up_tile0 * 256:] = gated_rows(t(f"{p}mlp.{at}gate").to(u.dtype), t(f"{p}mlp.{at}up").to(u.dtype), KW)
            d = zeros(NW, L.round_up(f.inner, 128))
            d[:W, : f.inner] = t(f"{p}mlp.{at}down")
            lw.down = pack_linear(d, dtype)
        lw.up = pack_linear(u, dtype)

    layers = []
    for i, l in enumerate(cfg.layers):
        p, m = f"l{i}.", l.mixer
        beside = l.mlp if cfg.parallel else None
        lay = project_layout(m, beside, cfg.two_norms)
        off, n_plain, tile0 = lay.off, lay.n_plain, lay.tile0
        r, seg_rows, bias = zeros(lay.rows, KW), dict(m.segments()), None
        for name, tensor, first in m.sources():
            r[off[name]: off[name] + seg_rows[name], :W] = t(f"{p}mix.{tensor}")[first: first + seg_rows[name]]
        if m.biases():
            bias = torch.zeros(L.round_up(n_plain, 8), dtype=torch.float32, device=dev)
            for name, tensor, first in m.sources():
                if name in m.biases():
                    bias[off[name]: off[name] + seg_rows[name]] = f32(f"{p}mix.{tensor}.b")
        mix_k0, mix_k = {}, 0
        for (pre, _, _), (_, features, _) in zip(m.parts(), m.out_tensors()):
            mix_k0[pre] = mix_k
            mix_k += L.round_up(features, 64)
        ff_k = L.round_up(beside.inner, beside.k_step) if beside is not None else 0
        o = zeros(NW, mix_k + ff_k)
        act_bias = out_bias = ex_up = ex_down = None
        for (pre, _, scale), (name, features, has_bias) in zip(m.parts(), m.out_tensors()):
            o[:W, mix_k0[pre]: mix_k0[pre] + features] = t(f"{p}mix.{name}")
            if has_bias:                                               # (the parts' factors are on their results otherwise)
                out_bias = scale * row(f"{p}mix.{name}.b") + (0 if out_bias is None else out_bias)
        if isinstance(beside, ClampedGlu):
            r[tile0 * 256:] = gated_rows(t(p + "mlp.gate").to(r.dtype), t(p + "mlp.up").to(r.dtype), KW)
            o[:W, mix_k: mix_k + l.mlp.ff] = t(p + "mlp.down")
        elif isinstance(beside, ExpertMix):
            r[off["router"]: off["router"] + beside.experts, :W] = t(p + "mlp.router")
            if beside.shared:
                full = zeros(beside.tiles * beside.per_tile, KW)
                full[: beside.shared, :W] = t(p + "mlp.shared.up")
                tiles = r[tile0 * 256:].view(-1, 256, KW)
                tiles[:, : beside.per_tile] = full.view(-1, beside.per_tile, KW)
                tiles[:, beside.per_tile, :W] = t(p + "mlp.shared.sg")[0]
                o[:W, mix_k: mix_k + beside.shared] = t(p + "mlp.shared.down")
            ex_up, ex_down = experts(p, beside)
        elif beside is not None:
            r[tile0 * 256: tile0 * 256 + beside.ff, :W] = t(p + "mlp.up")
            o[:W, mix_k: mix_k + beside.ff] = t(p + "mlp.down")
            if isinstance(beside, Gelu):
                act_bias, out_bias = torch.zeros(beside.tiles * 256, dtype=torch.float32, device=dev), f32(p + "mlp.down.b")
                act_bias[: beside.ff] = f32(p + "mlp.up.b")
        extra, carry = {}, None
        for pre, m, _ in l.mixer.parts():
            own, carried = mixer_tensors(m, f"{p}mix.{pre}")
            extra.update({pre + k: v for k, v in own.items()})
            carry = carry or carried
        lw = StackLayer(row(p + "norm1") if cfg.post_norms else norm(p + "norm1"), pack_linear(r, dtype), pack_linear(o, dtype), off, n_plain, tile0, mix_k, extra, bias,
                        tile2=lay.tile2, lat_tiles=lay.lat_tiles, carry=carry, act_bias=act_bias, out_bias=out_bias, experts_up=ex_up, experts_down=ex_down, mix_k0=mix_k0)
        if beside is not None and cfg.two_norms:
            lw.norm2 = norm(p + "norm2")
        del r, o
        if cfg.post_norms:
            lw.post1 = row(p + "norm1b")
            lw.shift = row(p + "shift") if cfg.token_shift else None
            if l.mlp is not None:
                lw.norm2, lw.post2 = row(p + "norm2"), row(p + "norm2b")
                gated_feed_forward(lw, p, l.mlp)
        elif l.mlp is not None and not cfg.parallel:
            ff = l.mlp.ff
            u, d = zeros(L.round_up(ff, 256), KW), zeros(NW, L.round_up(ff, 64))
            u[:ff, :W], d[:W, :ff] = t(p + "mlp.up"), t(p + "mlp.down")
            lw.norm2, lw.up, lw.down = norm(p + "norm2"), pack_linear(u, dtype), pack_linear(d, dtype)
            del u, d
        layers.append(lw)
    head = zeros(L.round_up(cfg.vocab, 256), KW)
    head[: cfg.vocab, :W] = t("head")
    out = StackWeights(t("embed").to(dtype).contiguous(), layers, row("final.norm") if cfg.post_norms else norm("final.norm"), pack_linear(head, dtype))
    if cfg.loop is not None and not cfg.loop_linear:
        out.loop_step = torch.zeros(cfg.loop.times, wide, dtype=torch.float32, device=dev)
        out.loop_step[:, :W] = f32("loop.step")
    elif cfg.loop is not None:
        li = t("loop.in")
        r = zeros(NW, 2 * KW)
        r[:W, :W], r[:W, KW: KW + W] = li[:, :W], li[:, W:]
        out.loop_in, out.loop_step = pack_linear(r, dtype), f32("loop.step")
    return out


def load(cfg: StackConfig, model_dir, dtype: torch.dtype, device) -> StackWeights:
    tensors = read_safetensors(Path(model_dir) / "model.safetensors")
    missing = [n for n in tensor_shapes(cfg) if n not in tensors]
    if missing:
        raise ValueError(f"{model_dir}: {len(missing)} tensors are missing (first: {missing[0]!r})")
    return build(cfg, tensors.__getitem__, dtype, device)


def random_init(cfg: StackConfig, dtype: torch.dtype, device, seed: int = 0) -> StackWeights:
    g = torch.Generator(device=device).manual_seed(seed)
    shapes = tensor_shapes(cfg)
    return build(cfg, lambda n: random_tensor(n, shapes[n], g, device, cfg.norm_offset), dtype, device)
