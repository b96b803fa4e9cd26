"""Weights of a layer-by-layer decoder: the tensors by name and shape, the safetensors reader, and the device
layouts its kernels read.

Side by side (parallel residual), a layer needs two linears.  `proj` holds every row that reads the normed stream:
the mixer's segments (each starting at a multiple of 8 rows, the whole padded to 256), then the feed-forward's rows
as tiles of 128 gate and 128 up rows of the same features.  `out` holds the mixer's output columns and the down
columns side by side, so that one product adds both sublayers to the stream.  One after the other, `proj` and `out`
belong to the mixer alone and `up` and `down` to the feed-forward behind its own norm.
"""
from __future__ import annotations

import json
import math
import mmap
import struct
from dataclasses import dataclass, field
from pathlib import Path
from typing import Callable, Optional

import torch

from ..ops import layouts as L
from .stack_config import ClampedGlu, DeltaMixer, LatentMixer, OuterMixer, StackConfig

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
        t["loop.in"], t["loop.step"] = (w, 2 * w), (cfg.loop.times, w)
    for i, l in enumerate(cfg.layers):
        p, m = f"l{i}.", l.mixer
        rows, bias = dict(m.segments()), m.biases()
        t[p + "norm1"] = (w,)
        for seg, tensor, first in m.sources():
            have = t.get(f"{p}mix.{tensor}", (0, w))[0]
            t[f"{p}mix.{tensor}"] = (max(have, first + rows[seg]), w)
            if seg in bias:
                t[f"{p}mix.{tensor}.b"] = (rows[seg],)
        for name, shape in m.extra_shapes().items():
            t[f"{p}mix.{name}"] = shape
        t[p + "mix.o"] = (w, m.out_features)
        if l.mlp is not None:
            if not cfg.parallel:
                t[p + "norm2"] = (w,)
            for name in ("gate", "up") if isinstance(l.mlp, ClampedGlu) else ("up",):
                t[f"{p}mlp.{name}"] = (l.mlp.ff, w)
            t[p + "mlp.down"] = (w, l.mlp.ff)
    t["final.norm"], t["head"] = (w,), (cfg.vocab, w)
    return t


def random_tensor(name: str, shape: tuple, g: torch.Generator, device, norm_offset: float = 0.0) -> torch.Tensor:
    leaf = name.rsplit(".", 1)[-1]
    if leaf in ("norm1", "norm2", "norm"):
        around = norm_offset if ".mix." not in name else 0.0            # (a mixer's own norm is stored plain)
        return torch.full(shape, 1.0 - around, dtype=torch.bfloat16, device=device)
    if leaf == "D":
        return torch.ones(shape, dtype=torch.bfloat16, device=device)
    if leaf == "b":
        return torch.zeros(shape, dtype=torch.bfloat16, device=device)
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
    act_tile0: int                   # first gate | up tile
    act_k0: int                      # first feed-forward column of `out`'s operand
    extra: dict = field(default_factory=dict)
    bias: Optional[torch.Tensor] = None     # fp32, of the projection's stored columns
    norm2: Optional[torch.Tensor] = None    # feed-forward behind the mixer: its norm and linears
    up: Optional[Linear] = None
    down: Optional[Linear] = None


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
            tot += sum(x.nbytes() for x in (l.proj, l.out, l.up, l.down) if x is not None) + sum(t.numel() * t.element_size() for t in l.extra.values())
        return tot


def pack_linear(rows: torch.Tensor, dtype: torch.dtype) -> Linear:
    """rows [N_pad, K] (N_pad a multiple of 256, K of 64)."""
    n, k = rows.shape
    assert n % 256 == 0 and k % 64 == 0, (n, k)
    if dtype == torch.float32:
        return Linear(rows.float().contiguous(), n, k)
    return Linear(L.tile_weight_int8(rows.to(torch.bfloat16).contiguous().view(torch.int8).reshape(n, k * 2)), n, k)


def project_layout(mixer, mlp: Optional[ClampedGlu]) -> tuple:
    """(segment offsets, stored columns, first gate | up tile, rows in all)."""
    off, n = {}, 0
    for name, rows in mixer.segments():
        off[name] = n
        n = (n + rows + 7) // 8 * 8
    tile0 = (n + 255) // 256
    return off, n, tile0, (tile0 + ((mlp.ff + 127) // 128 if mlp is not None else 0)) * 256


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
    layers = []
    for i, l in enumerate(cfg.layers):
        p, m = f"l{i}.", l.mixer
        beside = l.mlp if cfg.parallel else None
        off, n_plain, tile0, rows = project_layout(m, beside)
        r, seg_rows, bias = zeros(rows, KW), dict(m.segments()), None
        for name, tensor, first in m.sources():
            r[off[name]: off[name] + seg_rows[name], :W] = t(f"{p}mix.{tensor}")[first: first + seg_rows[name]]
        if m.biases():
            bias = torch.zeros(L.round_up(n_plain, 8), dtype=torch.float32, device=dev)
            for name, tensor, first in m.sources():
                if name in m.biases():
                    bias[off[name]: off[name] + seg_rows[name]] = f32(f"{p}mix.{tensor}.b")
        mix_k = L.round_up(m.out_features, 64)
        ff_k = L.round_up(l.mlp.ff, 128) if beside is not None else 0
        o = zeros(NW, mix_k + ff_k)
        o[:W, : m.out_features] = t(p + "mix.o")
        if beside is not None:
            gu = r[tile0 * 256:].view(-1, 2, 128, KW)                  # [tile][gate | up][feature][K]
            for half, name in enumerate(("gate", "up")):
                full = zeros(ff_k, KW)
                full[: l.mlp.ff, :W] = t(f"{p}mlp.{name}")
                gu[:, half] = full.view(-1, 128, KW)
            o[:W, mix_k: mix_k + l.mlp.ff] = t(p + "mlp.down")
        extra = {}
        if isinstance(m, DeltaMixer):
            extra["conv"] = torch.cat([f32(f"{p}mix.{n}.conv") for n in ("q", "k", "v")]).contiguous()
            for n in ("A_log", "dt_bias", "norm"):
                extra[n] = f32(f"{p}mix.{n}")
        elif isinstance(m, OuterMixer):
            for n in ("norm", *(("A_log", "dt_bias", "D") if m.decay is None else ())):
                extra[n] = f32(f"{p}mix.{n}")
            if m.decay is not None:
                extra["decay"] = torch.tensor(m.decay, dtype=torch.float32, device=dev)
            if m.taps:                                                 # stored v | k | q, read q | k | v
                kd, vd = m.kv_heads * m.dim, m.heads * m.vdim
                for n, key in (("conv", "conv"), ("conv.b", "conv_b")):
                    c = f32(f"{p}mix.{n}")
                    extra[key] = torch.cat([c[vd + kd:], c[vd: vd + kd], c[:vd]]).contiguous()
        elif isinstance(m, LatentMixer):
            extra["dkv_norm"] = f32(p + "mix.dkv.norm")
            for n in ("uk", "uv"):                                     # row stride: the padded latent
                full = t(f"{p}mix.{n}")
                extra[n] = torch.zeros(full.shape[0], m.rank_pad, dtype=dtype, device=dev)
                extra[n][:, : m.kv_rank] = full
            half = m.rot_dim // 2
            extra["freq"] = torch.tensor([m.rot_base ** (-2.0 * j / m.rot_dim) for j in range(half)] or [1.0], dtype=torch.float32, device=dev)
        lw = StackLayer(norm(p + "norm1"), pack_linear(r, dtype), pack_linear(o, dtype), off, n_plain, tile0, mix_k, extra, bias)
        del r, o
        if l.mlp is not None and not cfg.parallel:
            ff = l.mlp.ff
            u, d = zeros(L.round_up(ff, 256), KW), zeros(NW, L.round_up(ff, 64))
            u[:ff, :W], d[:W, :ff] = t(p + "mlp.up"), t(p + "mlp.down")
            lw.norm2, lw.up, lw.down = norm(p + "norm2"), pack_linear(u, dtype), pack_linear(d, dtype)
            del u, d
        layers.append(lw)
    head = zeros(L.round_up(cfg.vocab, 256), KW)
    head[: cfg.vocab, :W] = t("head")
    out = StackWeights(t("embed").to(dtype).contiguous(), layers, norm("final.norm"), pack_linear(head, dtype))
    if cfg.loop is not None:
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
