"""Decoders described layer by layer: an ordered list of layers, each with its mixer and feed-forward (side by
side behind one norm or a norm each, or one after the other), an optional block of layers that runs several times, and the
constants of all of them.  `models.stack.StackModel` runs
any such description; an architecture is a reader of its `config.json` (ARCHITECTURES) and the order and
names of its tensors (`models.stack_weights`).
"""
from __future__ import annotations

import dataclasses
import json
import math
import os
import struct
from dataclasses import dataclass
from pathlib import Path
from typing import Optional


@dataclass(frozen=True)
class Rotation:
    """Rotary positions on the first `dims` values of a head: pair i turns by position * f_i, f_i = base^(-2 i / dims) / factor.
    yarn = (original, fast, slow): only the slow pairs are divided by the factor.  Pair i makes original f_i / 2 pi turns over
    `original` positions; those with more than `fast` keep f_i, those with fewer than `slow` are divided, a ramp over whole pair
    numbers lies between, and the rotated vector grows by 0.1 ln(factor) + 1."""
    base: float
    dims: int
    interleaved: bool = False         # pair i is (x[2 i], x[2 i + 1]) instead of (x[i], x[i + dims / 2])
    factor: float = 1.0
    yarn: Optional[tuple] = None

    def frequencies(self) -> list:
        f = [self.base ** (-2.0 * i / self.dims) for i in range(self.dims // 2)]
        if self.yarn is None:
            return [x / self.factor for x in f]
        original, fast, slow = self.yarn
        pair = lambda turns: self.dims * math.log(original / (2 * math.pi * turns)) / (2 * math.log(self.base))    # noqa: E731
        lo, hi = max(math.floor(pair(fast)), 0), min(math.ceil(pair(slow)), self.dims - 1)
        ramp = [min(max((i - lo) / max(hi - lo, 0.001), 0.0), 1.0) for i in range(len(f))]
        return [x / self.factor * r + x * (1.0 - r) for x, r in zip(f, ramp)]

    @property
    def amplitude(self) -> float:
        return 1.0 if self.yarn is None else 0.1 * math.log(self.factor) + 1.0

    @staticmethod
    def from_json(d: dict, interleaved: bool = False) -> "Rotation":
        s = d.get("scaling") or {}
        yarn = (float(s["original"]), float(s["fast"]), float(s["slow"])) if "original" in s else None
        return Rotation(float(d["base"]), d["dims"], interleaved, float(s.get("factor", 1.0)), yarn)


class Mixer:
    """What a layer asks of its mixer.  `segments` are the rows of the input projection, in order."""
    kind = ""
    kv_from: Optional[int] = None     # layer whose pages this mixer reads (it has none of its own)
    out_bias = False
    q_rank = 0                        # > 0: the first segment is a latent of this size, normed and carried on by a linear of its own

    def segments(self) -> list:
        """(name, rows)"""
        raise NotImplementedError

    def sources(self) -> list:
        """(segment, tensor, first row of the tensor): where the projection's rows come from."""
        return [(name, name, 0) for name, _ in self.segments()]

    def biases(self) -> list:
        """Segments whose tensor has a bias beside it (its name with '.b')."""
        return []

    def parts(self) -> list:
        """(prefix of names, mixer, factor of its result): several where mixers stand side by side."""
        return [("", self, 1.0)]

    def out_tensors(self) -> list:
        """(output tensor, its input features, whether it has a bias) of every part."""
        return [("o", self.out_features, self.out_bias)]

    def extra_shapes(self) -> dict:
        """Tensors beside the projections, name -> shape."""
        return {}

    def slot_bytes(self) -> int:
        return 0

    def page_token_bytes(self, elem: int) -> int:
        return 0


def _scan_width(n: int, what: str) -> int:
    """Key sizes the recurrence kernels are instantiated for."""
    for w in (64, 128, 192, 256, 384, 512):
        if w >= n:
            return w
    raise ValueError(f"{what}: key size {n} is above 512")


@dataclass(frozen=True)
class DeltaMixer(Mixer):
    """Gated delta rule: `kv_heads` query / key heads of size dim, `heads` value heads of size vdim, a causal
    convolution of `taps` over q, k and v."""
    heads: int
    kv_heads: int
    dim: int
    vdim: int
    taps: int
    unit_eps: float = 1e-6            # inside the root of the unit norm of q and k
    kind = "delta"

    @property
    def out_features(self) -> int:
        return self.heads * self.vdim

    @property
    def channels(self) -> int:        # convolution channels q | k | v
        return 2 * self.kv_heads * self.dim + self.heads * self.vdim

    @property
    def dim_pad(self) -> int:
        return _scan_width(self.dim, "delta mixer")

    @property
    def vdim_pad(self) -> int:
        return (self.vdim + 7) // 8 * 8

    def segments(self) -> list:
        """(name, rows) of the input projection."""
        return [("q", self.kv_heads * self.dim), ("k", self.kv_heads * self.dim), ("v", self.heads * self.vdim),
                ("b", self.heads), ("a", self.heads), ("g", self.heads * self.vdim)]

    def extra_shapes(self) -> dict:
        t = {f"{name}.conv": (rows, self.taps) for name, rows in self.segments()[:3]}
        return {**t, "A_log": (self.heads,), "dt_bias": (self.heads,), "norm": (self.vdim,)}

    def slot_bytes(self) -> int:
        return 4 * (self.heads * self.vdim_pad * self.dim_pad + self.taps * self.channels)


@dataclass(frozen=True)
class LatentMixer(Mixer):
    """Latent attention: a cached latent of kv_rank values and one rotated key part of rot_dim per token.  q_rank: queries come from
    a normed latent of their own.  kv_from: that layer's latents and key parts, with this layer's own carriers."""
    heads: int
    dim: int
    rot_dim: int
    vdim: int
    kv_rank: int
    scale: float
    rot: Rotation
    q_rank: int = 0
    gate_heads: bool = False          # output gate: one per head, else one per value
    kv_from: Optional[int] = None
    kind = "latent_attention"

    @property
    def out_features(self) -> int:
        return self.heads * self.vdim

    @staticmethod
    def _pad16(n: int) -> int:
        return (n + 15) // 16 * 16

    @property
    def rank_pad(self) -> int:
        return self._pad16(self.kv_rank)

    @property
    def rot_pad(self) -> int:
        return self._pad16(self.rot_dim)

    @property
    def dim_pad(self) -> int:
        return self._pad16(self.dim)

    @property
    def vdim_pad(self) -> int:        # value sizes the expanded form is instantiated for (above: the absorbed form only)
        return next((n for n in (32, 64, 128, 256) if n >= self.vdim), self._pad16(self.vdim))

    def segments(self) -> list:
        q = ("dq", self.q_rank) if self.q_rank else ("q", self.query_rows)
        kv = [] if self.kv_from is not None else [("dkv", self.kv_rank + self.rot_dim)]
        return [q, *kv, ("g", self.heads if self.gate_heads else self.heads * self.vdim)]

    @property
    def query_rows(self) -> int:
        return self.heads * (self.dim + self.rot_dim)

    def extra_shapes(self) -> dict:
        t = {"dq.norm": (self.q_rank,), "uq": (self.query_rows, self.q_rank)} if self.q_rank else {}
        if self.kv_from is None:
            t["dkv.norm"] = (self.kv_rank,)
        return {**t, "uk": (self.heads * self.dim, self.kv_rank), "uv": (self.heads * self.vdim, self.kv_rank)}

    def page_token_bytes(self, elem: int) -> int:
        return 0 if self.kv_from is not None else elem * (self.rank_pad + self.rot_pad)

    @property
    def key_tile(self) -> int:        # an expanded key in whole 64-wide tiles
        return (self.dim_pad + self.rot_pad + 63) // 64 * 64

    def expanded_token_bytes(self, elem: int) -> int:
        return elem * self.heads * (self.key_tile + self.vdim_pad)


@dataclass(frozen=True)
class OuterMixer(Mixer):
    """Decayed outer products: S <- a S + k (w v)^T, o = S^T q, fp32 state of `heads` heads (dim x vdim).

    decay given     constant per head, w = 1; q, k, v are silu of the projection (linear attention)
    decay None      a and w follow from a step size per token and head, a skip connection, q | k | v pass a causal
                    convolution of `taps` with a bias (state-space duality)
    The read-out is normed in `norm_groups` parts; gate_first: silu(gate) ahead of the norm, else sigmoid(gate) after it."""
    heads: int
    kv_heads: int                     # key / query heads; value heads share them in equal groups
    dim: int
    vdim: int
    taps: int = 0                     # 0: no convolution
    decay: Optional[tuple] = None
    norm_groups: int = 1
    gate_first: bool = False
    packed: Optional[str] = None      # one tensor holds gate | v | k | q | dt
    kind = "outer"

    @property
    def out_features(self) -> int:
        return self.heads * self.vdim

    @property
    def channels(self) -> int:        # convolution channels q | k | v
        return 2 * self.kv_heads * self.dim + self.heads * self.vdim

    @property
    def dim_pad(self) -> int:
        return _scan_width(self.dim, "decayed outer products")

    @property
    def vdim_pad(self) -> int:
        return (self.vdim + 7) // 8 * 8

    def segments(self) -> list:
        kd, vd = self.kv_heads * self.dim, self.heads * self.vdim
        return [("q", kd), ("k", kd), ("v", vd), ("g", vd)] + ([("dt", self.heads)] if self.decay is None else [])

    def sources(self) -> list:
        if self.packed is None:
            return super().sources()
        n, at, out = dict(self.segments()), 0, []
        for name in ("g", "v", "k", "q", "dt"):
            out.append((name, self.packed, at))
            at += n[name]
        return out

    def extra_shapes(self) -> dict:
        t = {"norm": (self.heads * self.vdim,)}
        if self.taps:
            t["conv"], t["conv.b"] = (self.channels, self.taps), (self.channels,)
        if self.decay is None:
            t["dt_bias"] = t["A_log"] = t["D"] = (self.heads,)
        return t

    def slot_bytes(self) -> int:
        return 4 * (self.heads * self.vdim_pad * self.dim_pad + self.taps * self.channels)


@dataclass(frozen=True)
class GroupedMixer(Mixer):
    """Grouped-query attention: q and k over their root mean square per head, rotated, capped scores, keys of the query's own
    chunk of positions or of a sliding window, a learned number per head in the denominator, an output gate; each where asked for.
    taps: q, k and v pass a causal convolution of their own; q and k are then normed over all their heads at once, with weights,
    and values per head.  kv_from: the pages of that layer are read, with this layer's queries and mask."""
    heads: int
    kv_heads: int
    dim: int
    vdim: int
    scale: float
    softcap: float = 0.0              # 0: scores are not capped
    chunk: int = 0                    # 0: every earlier key
    qk_norm: bool = True
    bias: bool = True
    kv_from: Optional[int] = None
    rot: Optional[Rotation] = None
    sink: bool = False
    gate: bool = False                # sigmoid of a projection, value by value
    window: int = 0                   # > 0: the last `window` keys, the query's own among them
    taps: int = 0
    out_bias: bool = False
    kind = "attention"

    @property
    def channels(self) -> int:        # convolution channels q | k | v
        return (self.heads + self.kv_heads) * self.dim + self.kv_heads * self.vdim

    @property
    def out_features(self) -> int:
        return self.heads * self.vdim

    @property
    def score_dim(self) -> int:       # in whole steps of the tensor cores
        return (self.dim + 15) // 16 * 16

    @property
    def key_pad(self) -> int:         # a cached key in whole 64-wide tiles
        return (self.dim + 63) // 64 * 64

    @property
    def vdim_pad(self) -> int:
        return (self.vdim + 31) // 32 * 32

    def segments(self) -> list:
        q, g = [("q", self.heads * self.dim)], [("g", self.heads * self.vdim)] if self.gate else []
        return q + g if self.kv_from is not None else q + [("k", self.kv_heads * self.dim), ("v", self.kv_heads * self.vdim)] + g

    def biases(self) -> list:
        return [name for name, _ in self.segments() if name != "g"] if self.bias else []

    def extra_shapes(self) -> dict:
        t = {"sink": (self.heads,)} if self.sink else {}
        if self.taps:
            rows = dict(self.segments())
            t.update({f"{n}.conv": (rows[n], self.taps) for n in ("q", "k", "v")})
            t.update({f"{n}.norm": (rows[n],) for n in ("q", "k")})
        return t

    def slot_bytes(self) -> int:
        return 4 * self.taps * self.channels

    def page_token_bytes(self, elem: int) -> int:
        return 0 if self.kv_from is not None else elem * self.kv_heads * (self.key_pad + self.vdim_pad)


@dataclass(frozen=True)
class ChannelDeltaMixer(Mixer):
    """Delta rule with a decay and a removal rate per head and key channel, keys and values of one size: S <- diag(w) S - (a u) (u^T S)
    + k v^T with the unit key u, both terms of the old state; o = S^T r.  Decays come through `rank` values shared by the heads."""
    heads: int
    dim: int
    rank: int
    unit_eps: float = 1e-6            # inside the root of the unit norm of k
    kind = "channel_delta"
    taps = 0

    @property
    def out_features(self) -> int:
        return self.heads * self.dim

    @property
    def dim_pad(self) -> int:
        return _scan_width(self.dim, "delta mixer")

    @property
    def vdim_pad(self) -> int:
        return (self.dim + 7) // 8 * 8

    def segments(self) -> list:
        n = self.out_features
        return [("r", n), ("k", n), ("v", n), ("a", n), ("w1", self.rank), ("g", n)]

    def biases(self) -> list:
        return ["a"]

    def extra_shapes(self) -> dict:
        n = self.out_features
        return {"w2": (n, self.rank), "w0": (n,), "norm": (n,)}

    def slot_bytes(self) -> int:
        return 4 * self.heads * self.vdim_pad * self.dim_pad


@dataclass(frozen=True)
class SideBySideMixer(Mixer):
    """Two mixers over the same rows: left_scale * left + right_scale * right."""
    left: Mixer
    right: Mixer
    left_scale: float = 1.0
    right_scale: float = 1.0
    kind = "side_by_side"

    def parts(self) -> list:
        return [("left.", self.left, self.left_scale), ("right.", self.right, self.right_scale)]

    def _all(self, what) -> list:
        return [(pre + name, *rest) for pre, m, _ in self.parts() for name, *rest in what(m)]

    def segments(self) -> list:
        return self._all(lambda m: m.segments())

    def sources(self) -> list:
        return [(pre + seg, pre + tensor, first) for pre, m, _ in self.parts() for seg, tensor, first in m.sources()]

    def biases(self) -> list:
        return [pre + name for pre, m, _ in self.parts() for name in m.biases()]

    def extra_shapes(self) -> dict:
        return dict(self._all(lambda m: m.extra_shapes().items()))

    def out_tensors(self) -> list:
        return self._all(lambda m: m.out_tensors())

    def slot_bytes(self) -> int:
        return self.left.slot_bytes() + self.right.slot_bytes()

    def page_token_bytes(self, elem: int) -> int:
        return self.left.page_token_bytes(elem) + self.right.page_token_bytes(elem)


class FeedForward:
    """What a layer asks of its feed-forward.  Its rows are tiles of 256 behind the mixer's: `per_tile` features each."""
    act_kind = 0                      # the linear epilogue's activation
    per_tile = 256
    k_step = 64                       # the activation's width goes up to a multiple of this
    limit = alpha = 0.0

    @property
    def inner(self) -> int:
        """Width of the activation that one linear produces and the next consumes (0: none)."""
        return self.ff

    @property
    def tiles(self) -> int:
        return (self.inner + self.per_tile - 1) // self.per_tile

    def shapes(self, width: int) -> dict:
        return {"up": (self.ff, width), "down": (width, self.ff)}


@dataclass(frozen=True)
class ClampedGlu(FeedForward):
    """g = min(gate, limit), u = clamp(up, -limit, limit), y = g sigmoid(alpha g) (u + 1)."""
    ff: int
    limit: float
    alpha: float = 1.702
    per_tile = k_step = 128

    def shapes(self, width: int) -> dict:
        return {"gate": (self.ff, width), **super().shapes(width)}


@dataclass(frozen=True)
class SquaredRelu(FeedForward):
    """y = max(up, 0)^2, no gate."""
    ff: int
    act_kind = 1


@dataclass(frozen=True)
class Gelu(FeedForward):
    """y = gelu(up + b) by the error function; a bias behind either matrix."""
    ff: int
    act_kind = 3

    def shapes(self, width: int) -> dict:
        return {"up": (self.ff, width), "up.b": (self.ff,), "down": (width, self.ff), "down.b": (width,)}


GATED_ACTS = {"gelu_tanh": 4, "silu": 5}


@dataclass(frozen=True)
class GatedUnit(FeedForward):
    """y = act(gate) up; act: gelu (by tanh) or silu."""
    ff: int
    act: str = "silu"
    per_tile = k_step = 128

    @property
    def act_kind(self) -> int:
        return GATED_ACTS[self.act]

    def shapes(self, width: int) -> dict:
        return {"gate": (self.ff, width), **super().shapes(width)}


@dataclass(frozen=True)
class ExpertMix(FeedForward):
    """Mixture of experts: softmax over `experts` scores, the `top` best of the `keep` groups of neighbours whose best
    score is best, weighted by their scores as they are; experts are squared ReLUs.  shared: the size of one more expert for every
    token, times the sigmoid of a number of its own.
    gated: experts are gated silu units, the shared one is added as it is.
    sigmoid: scores are sigmoids; a correction per expert joins them for the choice, where a group counts by the sum of its two best;
    the weights are the chosen scores over their sum, times `scale`."""
    experts: int
    top: int
    ff: int
    groups: int = 1
    keep: int = 1
    shared: int = 0
    gated: bool = False
    sigmoid: bool = False
    scale: float = 1.0

    @property
    def act_kind(self) -> int:        # of the shared expert
        return GATED_ACTS["silu"] if self.gated else 2

    @property
    def expert_act_kind(self) -> int:
        return GATED_ACTS["silu"] if self.gated else 1

    @property
    def per_tile(self) -> int:        # not gated: and the shared expert's gate row behind them
        return 128 if self.gated else 248

    @property
    def k_step(self) -> int:
        return 128 if self.gated else 64

    @property
    def inner(self) -> int:
        return self.shared

    @property
    def matrices(self) -> tuple:      # of an expert, ahead of `down`
        return ("gate", "up") if self.gated else ("up",)

    def shapes(self, width: int) -> dict:
        t = {}
        for e in range(self.experts):
            t.update({f"e{e}.{n}": (self.ff, width) for n in self.matrices})
            t[f"e{e}.down"] = (width, self.ff)
        t["router"] = (self.experts, width)
        if self.sigmoid:
            t["correction"] = (self.experts,)
        if self.shared:
            t.update({f"shared.{n}": (self.shared, width) for n in self.matrices})
            t["shared.down"] = (width, self.shared)
            if not self.gated:
                t["shared.sg"] = (1, width)
        return t


@dataclass(frozen=True)
class LayerSpec:
    mixer: Mixer
    mlp: Optional[FeedForward] = None


@dataclass(frozen=True)
class LoopSpec:
    """Layers start .. stop - 1 run `times` times in a row."""
    start: int
    stop: int
    times: int


@dataclass(frozen=True)
class LayerRun:
    """One pass through one layer: cache and state belong to the run, weights to the layer."""
    index: int
    layer: int
    enter: Optional[int] = None       # number of the pass that starts here (the loop's input step comes first)


@dataclass(frozen=True)
class StackConfig:
    name: str
    arch: str
    vocab: int
    width: int
    layers: tuple
    eps: float = 1e-6
    embed_scale: float = 1.0
    parallel: bool = True             # mixer and feed-forward side by side; else one after the other, a norm each
    two_norms: bool = False           # side by side: the feed-forward reads a norm of its own
    logit_cap: float = 0.0            # logits become cap tanh(logits / cap)
    norm_offset: float = 0.0          # norms multiply by offset + weight
    post_norms: bool = False          # one after the other: a sublayer's result is normed, too, before it joins the stream
    residual_mult: float = 1.0        # and multiplied by this
    token_shift: bool = False         # what a mixer reads is blended with the token before
    loop: Optional[LoopSpec] = None
    loop_linear: bool = True          # a pass starts with a linear over [stream; embedding], else with its vector only
    page_tokens: int = 64
    max_ctx: int = 32768
    source: Optional[str] = None      # folder the description was read from
    # what the serving plane asks of every model description
    moe = None
    drafter = None

    @property
    def hidden(self) -> int:
        return self.width

    @property
    def runs(self) -> tuple:
        n, out = len(self.layers), []
        spans = [(0, n, 1)] if self.loop is None else [(0, self.loop.start, 1), (self.loop.start, self.loop.stop, self.loop.times),
                                                       (self.loop.stop, n, 1)]
        for which, (a, b, times) in enumerate(spans):
            for t in range(times):
                for i in range(a, b):
                    enter = t if (self.loop is not None and which == 1 and i == a) else None
                    out.append(LayerRun(len(out), i, enter))
        return tuple(out)

    def mixers(self) -> list:
        """Every mixer of every layer."""
        return [m for l in self.layers for _, m, _ in l.mixer.parts()]

    def __post_init__(self):
        if not self.layers:
            raise ValueError(f"{self.name}: no layers")
        if self.loop is not None and not (0 <= self.loop.start < self.loop.stop <= len(self.layers) and self.loop.times >= 1):
            raise ValueError(f"{self.name}: loop {self.loop} does not fit {len(self.layers)} layers")
        for i, l in enumerate(self.layers):
            m = l.mixer
            if isinstance(m, DeltaMixer) and (m.heads % m.kv_heads or m.taps < 1):
                raise ValueError(f"{self.name}: layer {i}: heads {m.heads} / kv_heads {m.kv_heads} / taps {m.taps}")
            if isinstance(m, OuterMixer) and (m.heads % m.kv_heads or m.out_features % m.norm_groups or m.taps < 0
                                              or (m.decay is not None and len(m.decay) != m.heads)):
                raise ValueError(f"{self.name}: layer {i}: heads {m.heads} / kv_heads {m.kv_heads} / norm_groups {m.norm_groups} / decay {m.decay}")
            if isinstance(m, GroupedMixer):
                self._check_grouped(i, m)
            if isinstance(m, SideBySideMixer):
                if not self.post_norms or any(x.kv_from is not None for _, x, _ in m.parts()):
                    raise ValueError(f"{self.name}: layer {i}: mixers side by side stand ahead of normed results and have pages of their own")
                for _, x, _ in m.parts():
                    if isinstance(x, GroupedMixer):
                        self._check_grouped(i, x)
            if isinstance(m, ChannelDeltaMixer) and not self.post_norms:
                raise ValueError(f"{self.name}: layer {i}: a channel delta rule stands ahead of a normed result")
            for _, x, _ in m.parts():
                if isinstance(x, ChannelDeltaMixer) and not (x.heads >= 1 and 1 <= x.dim <= 512 and 1 <= x.rank <= 2048):
                    raise ValueError(f"{self.name}: layer {i}: heads {x.heads} / dim {x.dim} / rank {x.rank}")
            if self.post_norms:
                if l.mlp is not None and not (isinstance(l.mlp, GatedUnit) or (isinstance(l.mlp, ExpertMix) and l.mlp.gated)):
                    raise ValueError(f"{self.name}: layer {i}: ahead of normed results feed-forwards are gated units or mixtures of them")
            elif isinstance(l.mlp, GatedUnit) or (isinstance(l.mlp, ExpertMix) and l.mlp.gated):
                raise ValueError(f"{self.name}: layer {i}: {type(l.mlp).__name__} stands ahead of a normed result only")
            elif not self.parallel and isinstance(l.mlp, (Gelu, ExpertMix)):
                raise ValueError(f"{self.name}: layer {i}: {type(l.mlp).__name__} stands beside its mixer only")
            if isinstance(l.mlp, ExpertMix):
                self._check_experts(i, l.mlp)
            if isinstance(m, LatentMixer):
                if m.rot_dim % 2 or m.kv_rank > 1024 or m.dim > 1024 or m.rot.dims != m.rot_dim:
                    raise ValueError(f"{self.name}: layer {i}: rot_dim {m.rot_dim} (rotated {m.rot.dims}), kv_rank {m.kv_rank}, dim {m.dim}")
                self._check_source(i, m, lambda s: (s.kv_rank, s.rot_dim, s.rot))
        if self.two_norms and (not self.parallel or self.loop is not None):
            raise ValueError(f"{self.name}: a second norm needs layers side by side and no loop")
        if self.post_norms and (self.parallel or self.width > 16384 or any(not isinstance(m, (GroupedMixer, ChannelDeltaMixer)) for m in self.mixers())):
            raise ValueError(f"{self.name}: normed results join a stream of up to 16384 values, one sublayer after the other; mixers are attention and channel delta rules")
        if not self.post_norms and (self.token_shift or self.residual_mult != 1.0 or not self.loop_linear):
            raise ValueError(f"{self.name}: blended tokens, factors and passes without a linear come with normed results")

    def _check_experts(self, i: int, f: ExpertMix) -> None:
        if not (1 <= f.experts <= 1024 and 1 <= f.top <= 32 and f.groups >= 1 and f.experts % f.groups == 0 and 1 <= f.keep <= f.groups
                and f.top <= f.experts // f.groups * f.keep):
            raise ValueError(f"{self.name}: layer {i}: top {f.top} of {f.experts} experts in {f.keep} of {f.groups} groups")
        if not self.two_norms and not self.post_norms:
            raise ValueError(f"{self.name}: layer {i}: a mixture of experts reads a norm of its own")

    def _check_source(self, i: int, m: Mixer, sizes) -> None:
        """A layer that reads another's pages finds a layer of its kind and sizes there."""
        if m.kv_from is None:
            return
        s = self.layers[m.kv_from].mixer if 0 <= m.kv_from < i else None
        if self.loop is not None or type(s) is not type(m) or s.kv_from is not None or sizes(s) != sizes(m):
            raise ValueError(f"{self.name}: layer {i} cannot read the keys and values of layer {m.kv_from}")

    def _check_grouped(self, i: int, m: GroupedMixer) -> None:
        if m.heads % m.kv_heads or m.chunk < 0 or m.window < 0 or (m.chunk and m.window) or m.dim > 2048 or m.vdim > 2048:
            raise ValueError(f"{self.name}: layer {i}: heads {m.heads} / kv_heads {m.kv_heads} / chunk {m.chunk} / window {m.window} / dim {m.dim} / vdim {m.vdim}")
        if m.taps and (m.kv_from is not None or m.qk_norm or m.gate or not self.post_norms):
            raise ValueError(f"{self.name}: layer {i}: a convolution of q, k and v comes with keys of its own, without a norm per head or a gate")
        if m.out_bias and not self.post_norms:
            raise ValueError(f"{self.name}: layer {i}: a bias behind the output stands ahead of a normed result")
        if m.rot is not None and (m.rot.dims % 2 or m.rot.dims > min(m.dim, 1024) or m.rot.interleaved):
            raise ValueError(f"{self.name}: layer {i}: rotation of {m.rot.dims} of {m.dim} values")
        self._check_source(i, m, lambda s: (s.kv_heads, s.dim, s.vdim, s.rot))

    def pages_of(self, run: LayerRun) -> int:
        """The run whose pages a run reads."""
        src = self.layers[run.layer].mixer.kv_from
        return run.index if src is None else src      # (no loop: runs and layers are the same)

    # ---- byte accounting (launch plan)
    def page_token_bytes(self, elem: int = 2) -> int:
        return sum(self.layers[r.layer].mixer.page_token_bytes(elem) for r in self.runs)

    def slot_bytes(self) -> int:
        return sum(self.layers[r.layer].mixer.slot_bytes() + (4 * self.width if self.token_shift else 0) for r in self.runs)

    def expanded_token_bytes(self, elem: int = 2) -> int:
        return max([l.mixer.expanded_token_bytes(elem) for l in self.layers if isinstance(l.mixer, LatentMixer)], default=0)

    def widest_project(self) -> int:
        return max(sum(n for _, n in l.mixer.segments()) + (l.mixer.query_rows if l.mixer.q_rank else 0) for l in self.layers)

    def expert_row_bytes(self, rows: int, elem: int = 2) -> int:
        """Scratch of the routed rows of a step (one layer at a time)."""
        return max([rows * l.mlp.top * elem * (l.mlp.ff + self.width) for l in self.layers if isinstance(l.mlp, ExpertMix)], default=0)

    def scan_row_bytes(self, rows: int) -> int:
        """Scratch of the prompt scans of channel delta rules and of convolved queries, keys and values (one layer at a time)."""
        n = [0]
        for m in self.mixers():
            if isinstance(m, ChannelDeltaMixer):
                n.append(m.heads * (17 * m.dim_pad + 64 + 4 * m.vdim_pad + 128) // 4 + m.heads * m.vdim_pad)
            elif isinstance(m, GroupedMixer) and m.taps:
                n.append(m.channels + 32)
        return 4 * rows * max(n)

    def param_count(self) -> int:
        from .stack_weights import tensor_shapes
        tot = 0
        for shape in tensor_shapes(self).values():
            n = 1
            for d in shape:
                n *= d
            tot += n
        return tot


# ------------------------------------------------------------------------------------ Renosun
def renosun_from_json(doc: dict, name: str = "renosun", source: Optional[str] = None, max_ctx: int = 32768, shapes: Optional[dict] = None) -> StackConfig:
    layers = []
    for i, l in enumerate(doc["layers"]):
        m = l["mixer"]
        if l["type"] == "delta":
            mixer = DeltaMixer(m["heads"], m["kv_heads"], m["dim"], m["vdim"], m["conv"])
        elif l["type"] == "latent_attention":
            if m["rot"]["dims"] != m["rot_dim"]:
                raise ValueError(f"layer {i}: rot.dims {m['rot']['dims']} is not rot_dim {m['rot_dim']}")
            mixer = LatentMixer(m["heads"], m["dim"], m["rot_dim"], m["vdim"], m["kv_rank"], float(m["scale"]), Rotation.from_json(m["rot"]))
        else:
            raise ValueError(f"layer {i}: unknown mixer type {l['type']!r}")
        mlp = None
        if l.get("mlp") is not None:
            if l["mlp"]["kind"] != "dense":
                raise ValueError(f"layer {i}: unknown feed-forward kind {l['mlp']['kind']!r}")
            mlp = ClampedGlu(l["mlp"]["ff"], float(l["mlp"]["limit"]))
        layers.append(LayerSpec(mixer, mlp))
    lp = doc.get("loop")
    return StackConfig(name=name, arch="Renosun", vocab=doc["vocab"], width=doc["width"], layers=tuple(layers), eps=float(doc["norm"]["eps"]),
                       embed_scale=float(doc["embedding"]["scale"]), loop=None if lp is None else LoopSpec(lp["start"], lp["stop"], lp["times"]),
                       source=source, max_ctx=max_ctx)


# ------------------------------------------------------------------------------------ Tepavik
def tepavik_from_json(doc: dict, name: str = "tepavik", source: Optional[str] = None, max_ctx: int = 32768, shapes: Optional[dict] = None) -> StackConfig:
    layers = []
    for i, l in enumerate(doc["layers"]):
        m = l["mixer"]
        if l["type"] == "lightning":
            mixer = OuterMixer(m["heads"], m["heads"], m["dim"], m["vdim"], decay=tuple(float(x) for x in m["decay"]))
        elif l["type"] == "mamba2":
            mixer = OuterMixer(m["heads"], m["groups"], m["state"], m["vdim"], taps=m["conv"], norm_groups=m["norm_groups"], gate_first=True, packed="in")
        elif l["type"] == "attention":
            mixer = GroupedMixer(m["heads"], m["kv_heads"], m["dim"], m["vdim"], float(m["scale"]), float(m.get("softcap") or 0.0), (m.get("mask") or {}).get("size", 0),
                                 kv_from=m.get("kv_from"))
        else:
            raise ValueError(f"layer {i}: unknown mixer type {l['type']!r}")
        mlp = None
        if l.get("mlp") is not None:
            if l["mlp"]["kind"] != "dense":
                raise ValueError(f"layer {i}: unknown feed-forward kind {l['mlp']['kind']!r}")
            mlp = SquaredRelu(l["mlp"]["ff"])
        layers.append(LayerSpec(mixer, mlp))
    return StackConfig(name=name, arch="Tepavik", vocab=doc["vocab"], width=doc["width"], layers=tuple(layers), eps=float(doc["norm"]["eps"]),
                       parallel=False, norm_offset=1.0, source=source, max_ctx=max_ctx)


# ------------------------------------------------------------------------------------ Fitatar
def fitatar_from_json(doc: dict, name: str = "fitatar", source: Optional[str] = None, max_ctx: int = 32768, shapes: Optional[dict] = None) -> StackConfig:
    layers = []
    for i, l in enumerate(doc["layers"]):
        m, f = l["mixer"], l.get("mlp")
        if l["type"] == "latent_attention":
            mixer = LatentMixer(m["heads"], m["dim"], m["rot_dim"], m["vdim"], m["kv_rank"], float(m["scale"]), Rotation.from_json(m["rot"], interleaved=True),
                                q_rank=m["q_rank"], gate_heads=True, kv_from=m.get("kv_from"))
        elif l["type"] == "attention":
            mixer = GroupedMixer(m["heads"], m["kv_heads"], m["dim"], m["vdim"], float(m["scale"]), qk_norm=False, bias=False,
                                 rot=Rotation.from_json(m["rot"]), sink=True, gate=True)
        else:
            raise ValueError(f"layer {i}: unknown mixer type {l['type']!r}")
        if f is None:
            mlp = None
        elif f["kind"] == "dense":
            mlp = Gelu(f["ff"])
        elif f["kind"] == "moe":
            r, g = f["router"], f["router"].get("groups") or {}
            mlp = ExpertMix(r["experts"], r["top"], f["expert"]["ff"], g.get("count", 1), g.get("keep", 1), (f.get("shared") or {}).get("ff", 0))
        else:
            raise ValueError(f"layer {i}: unknown feed-forward kind {f['kind']!r}")
        layers.append(LayerSpec(mixer, mlp))
    return StackConfig(name=name, arch="Fitatar", vocab=doc["vocab"], width=doc["width"], layers=tuple(layers), eps=float(doc["norm"]["eps"]),
                       embed_scale=float(doc["embedding"]["scale"]), two_norms=True, logit_cap=float(doc.get("logit_softcap") or 0.0),
                       source=source, max_ctx=max_ctx)


# ------------------------------------------------------------------------------------ Sofunex
def sofunex_from_json(doc: dict, name: str = "sofunex", source: Optional[str] = None, max_ctx: int = 32768, shapes: Optional[dict] = None) -> StackConfig:
    layers = []
    for i, l in enumerate(doc["layers"]):
        m, f = l["mixer"], l.get("mlp")
        if l["type"] != "parallel":
            raise ValueError(f"layer {i}: unknown mixer type {l['type']!r}")
        a, d, w1 = m["left"], m["right"], f"l{i}.mix.right.w1"
        if shapes is None or w1 not in shapes:
            raise ValueError(f"layer {i}: the size of tensor {w1!r} is missing (decays pass through that many values)")
        left = GroupedMixer(a["heads"], a["kv_heads"], a["dim"], a["vdim"], float(a["scale"]), qk_norm=False, rot=Rotation.from_json(a["rot"]),
                            window=(a.get("mask") or {}).get("size", 0), taps=a["conv"], out_bias=True)
        mixer = SideBySideMixer(left, ChannelDeltaMixer(d["heads"], d["dim"], shapes[w1][0]), float(m["left_scale"]), float(m["right_scale"]))
        if f is None:
            mlp = None
        elif f["kind"] == "dense":
            mlp = GatedUnit(f["ff"], "gelu_tanh")
        elif f["kind"] == "moe":
            r, g = f["router"], f["router"].get("groups") or {}
            mlp = ExpertMix(r["experts"], r["top"], f["expert"]["ff"], g.get("count", 1), g.get("keep", 1), (f.get("shared") or {}).get("ff", 0),
                            gated=True, sigmoid=True, scale=float(r.get("scale", 1.0)))
        else:
            raise ValueError(f"layer {i}: unknown feed-forward kind {f['kind']!r}")
        layers.append(LayerSpec(mixer, mlp))
    lp = doc.get("loop")
    return StackConfig(name=name, arch="Sofunex", vocab=doc["vocab"], width=doc["width"], layers=tuple(layers), eps=float(doc["norm"]["eps"]),
                       embed_scale=float(doc["embedding"]["scale"]), parallel=False, post_norms=True, residual_mult=float(doc.get("residual_mult", 1.0)),
                       token_shift=True, loop=None if lp is None else LoopSpec(lp["start"], lp["stop"], lp["times"]), loop_linear=False,
                       source=source, max_ctx=max_ctx)


ARCHITECTURES = {"Renosun": renosun_from_json, "Tepavik": tepavik_from_json, "Fitatar": fitatar_from_json, "Sofunex": sofunex_from_json}


def from_json(doc: dict, **kw) -> StackConfig:
    """shapes: sizes of the model's tensors by name, where its description alone does not settle all of them."""
    arch = doc.get("architecture")
    if arch not in ARCHITECTURES:
        raise KeyError(f"unknown architecture {arch!r}; known: {sorted(ARCHITECTURES)}")
    return ARCHITECTURES[arch](doc, **kw)


def is_model_dir(path: str) -> bool:
    return os.path.isfile(os.path.join(path, "config.json"))


def load_dir(path: str) -> StackConfig:
    """The description in a model folder (config.json beside model.safetensors)."""
    p = Path(path)
    return from_json(json.loads((p / "config.json").read_text()), name=p.resolve().name, source=str(p), shapes=file_shapes(p / "model.safetensors"))


def file_shapes(path) -> Optional[dict]:
    """Tensor sizes of a safetensors file, from its header (None: there is no such file)."""
    if not os.path.isfile(path):
        return None
    with open(path, "rb") as f:
        (n,) = struct.unpack("<Q", f.read(8))
        return {name: tuple(d["shape"]) for name, d in json.loads(f.read(n)).items() if name != "__metadata__"}


# ---- built-in descriptions (random weights)
def renosun_mini() -> StackConfig:
    """Small sizes for smoke tests and demos."""
    d = LayerSpec(DeltaMixer(6, 2, 64, 48, 3), ClampedGlu(384, 4.0))
    a = LayerSpec(LatentMixer(3, 64, 32, 40, 96, 96 ** -0.5, Rotation(1e4, 32)), ClampedGlu(384, 4.0))
    return StackConfig("renosun-mini", "Renosun", vocab=1024, width=320, layers=(a, d, d, a, d), embed_scale=8.0, loop=LoopSpec(1, 4, 2),
                       max_ctx=4096)


def renosun_bench(name: str, width: int, ff: int, kv_heads: int, heads: int, attn_heads: int, n_layers: int = 8, vocab: int = 65536) -> StackConfig:
    """Layers of a real model's size: three delta layers to one attention layer."""
    d = LayerSpec(DeltaMixer(heads, kv_heads, 128, 128, 4), ClampedGlu(ff, 7.0))
    a = LayerSpec(LatentMixer(attn_heads, 128, 64, 128, 512, 192 ** -0.5, Rotation(1e6, 64)), ClampedGlu(ff, 7.0))
    layers = tuple(a if i % 4 == 3 else d for i in range(n_layers))
    return StackConfig(name, "Renosun", vocab=vocab, width=width, layers=layers, embed_scale=width ** 0.5, loop=LoopSpec(n_layers // 4, n_layers // 2, 2))


def _decays(heads: int) -> tuple:
    return tuple(math.exp(-2.0 ** (-8.0 * (h + 1) / heads)) for h in range(heads))


def tepavik_mini() -> StackConfig:
    """Small sizes for smoke tests and demos."""
    ff = SquaredRelu(448)
    s = LayerSpec(OuterMixer(6, 2, 40, 32, taps=4, norm_groups=3, gate_first=True, packed="in"), ff)
    r = LayerSpec(OuterMixer(5, 5, 48, 40, decay=_decays(5)), ff)
    a = GroupedMixer(6, 2, 48, 56, 0.14, 25.0, 192)
    return StackConfig("tepavik-mini", "Tepavik", vocab=1024, width=288, parallel=False, norm_offset=1.0, max_ctx=4096,
                       layers=(s, LayerSpec(a, ff), r, LayerSpec(dataclasses.replace(a, kv_from=1, chunk=320), ff)))


def tepavik_bench(name: str, width: int, ff: int, heads: int, kv_heads: int, chunk: int = 8192, n_layers: int = 10, vocab: int = 65536) -> StackConfig:
    """Layers of a real model's size, two rounds of: two state-space layers (inner size 2 x width), attention, linear
    attention, attention over the keys of the first."""
    mlp = SquaredRelu(ff)
    s = LayerSpec(OuterMixer(2 * width // 64, 8, 128, 64, taps=4, norm_groups=8, gate_first=True, packed="in"), mlp)
    r = LayerSpec(OuterMixer(heads, heads, 128, 128, decay=_decays(heads)), mlp)
    layers = []
    for i in range(n_layers):
        a = GroupedMixer(heads, kv_heads, 128, 128, 128 ** -0.5, 30.0, chunk, kv_from=i - 2 if i % 5 == 4 else None)
        layers.append({2: LayerSpec(a, mlp), 3: r, 4: LayerSpec(a, mlp)}.get(i % 5, s))
    return StackConfig(name, "Tepavik", vocab=vocab, width=width, layers=tuple(layers), parallel=False, norm_offset=1.0)


def fitatar_mini() -> StackConfig:
    """Small sizes for smoke tests and demos."""
    a = GroupedMixer(6, 2, 48, 40, 0.15, qk_norm=False, bias=False, rot=Rotation(1e4, 24, factor=2.0), sink=True, gate=True)
    la = LatentMixer(4, 48, 32, 56, 80, 0.12, Rotation(1e5, 32, True, 4.0, (1024.0, 32.0, 1.0)), q_rank=112, gate_heads=True)
    moe = ExpertMix(24, 3, 96, 6, 2, 160)
    layers = (LayerSpec(a, Gelu(448)), LayerSpec(la, moe), LayerSpec(a, moe), LayerSpec(dataclasses.replace(la, kv_from=1), moe))
    return StackConfig("fitatar-mini", "Fitatar", vocab=1024, width=288, layers=layers, embed_scale=10.0, two_norms=True, logit_cap=20.0, max_ctx=4096)


def fitatar_bench(name: str, width: int, ff: int, heads: int, kv_heads: int, expert_ff: int, experts: int = 64, top: int = 6, shared: int = 2,
                  n_layers: int = 8, vocab: int = 65536) -> StackConfig:
    """Layers of a real model's size: a dense layer, then mixtures of experts; every fourth mixer is latent attention, the later
    ones on the latents of the first."""
    a = GroupedMixer(heads, kv_heads, 128, 128, 128 ** -0.5, qk_norm=False, bias=False, rot=Rotation(1e6, 64, factor=4.0), sink=True, gate=True)
    la = LatentMixer(heads, 128, 64, 128, 512, 192 ** -0.5, Rotation(1e6, 64, True, 8.0, (4096.0, 32.0, 1.0)), q_rank=1536, gate_heads=True)
    moe = ExpertMix(experts, top, expert_ff, 8, 4, shared * expert_ff)
    layers = []
    for i in range(n_layers):
        m = dataclasses.replace(la, kv_from=None if i < 4 else 1) if i % 4 == 1 else a
        layers.append(LayerSpec(m, moe if i else Gelu(ff)))
    return StackConfig(name, "Fitatar", vocab=vocab, width=width, layers=tuple(layers), embed_scale=width ** 0.5, two_norms=True, logit_cap=30.0)


def sofunex_mini() -> StackConfig:
    """Small sizes for smoke tests and demos."""
    def mix(heads, kv_heads, window):
        a = GroupedMixer(heads, kv_heads, 48, 40, 0.14, qk_norm=False, rot=Rotation(1e4, 32, factor=2.0), window=window, taps=4, out_bias=True)
        return SideBySideMixer(a, ChannelDeltaMixer(5, 56, 24), 0.7, 0.4)
    dense, moe = GatedUnit(448, "gelu_tanh"), ExpertMix(12, 3, 96, 3, 2, 160, gated=True, sigmoid=True, scale=1.5)
    layers = (LayerSpec(mix(6, 2, 192), dense), LayerSpec(mix(4, 4, 100), moe), LayerSpec(mix(6, 2, 192), moe), LayerSpec(mix(4, 1, 192), dense))
    return StackConfig("sofunex-mini", "Sofunex", vocab=1024, width=288, layers=layers, embed_scale=10.0, parallel=False, post_norms=True,
                       residual_mult=0.5, token_shift=True, loop=LoopSpec(1, 3, 2), loop_linear=False, max_ctx=4096)


def sofunex_bench(name: str, width: int, ff: int, heads: int, kv_heads: int, expert_ff: int, experts: int = 64, top: int = 6, shared: int = 2,
                  window: int = 8192, n_layers: int = 8, vocab: int = 65536) -> StackConfig:
    """Layers of a real model's size: attention and a delta rule of the stream's width side by side; a dense layer in four, else
    mixtures of experts; the third and fourth layer run twice."""
    a = GroupedMixer(heads, kv_heads, 128, 128, 128 ** -0.5, qk_norm=False, rot=Rotation(1e6, 128, factor=4.0), window=window, taps=4, out_bias=True)
    mixer = SideBySideMixer(a, ChannelDeltaMixer(heads, 128, 96), 0.6, 0.6)
    moe = ExpertMix(experts, top, expert_ff, 8, 4, shared * expert_ff, gated=True, sigmoid=True, scale=2.0)
    layers = tuple(LayerSpec(mixer, moe if i % 4 else GatedUnit(ff, "gelu_tanh")) for i in range(n_layers))
    return StackConfig(name, "Sofunex", vocab=vocab, width=width, layers=layers, embed_scale=width ** 0.5, parallel=False, post_norms=True,
                       residual_mult=0.3, token_shift=True, loop=LoopSpec(2, 4, 2), loop_linear=False)


NAMED = {"sofunex-mini": sofunex_mini,
         "sofunex-2k": lambda: sofunex_bench("sofunex-2k", 2048, 6144, 16, 4, 768),
         "sofunex-4k": lambda: sofunex_bench("sofunex-4k", 4096, 12288, 32, 8, 1024),
         "sofunex-5k": lambda: sofunex_bench("sofunex-5k", 5120, 13824, 40, 8, 1536),
         "fitatar-mini": fitatar_mini,
         "fitatar-2k": lambda: fitatar_bench("fitatar-2k", 2048, 8192, 16, 4, 1024),
         "fitatar-4k": lambda: fitatar_bench("fitatar-4k", 4096, 16384, 32, 8, 1536),
         "fitatar-5k": lambda: fitatar_bench("fitatar-5k", 5120, 20480, 40, 8, 2048),
         "tepavik-mini": tepavik_mini,
         "tepavik-2k": lambda: tepavik_bench("tepavik-2k", 2048, 8192, 16, 4),
         "tepavik-4k": lambda: tepavik_bench("tepavik-4k", 4096, 16384, 32, 8),
         "tepavik-5k": lambda: tepavik_bench("tepavik-5k", 5120, 20480, 40, 8),
         "renosun-mini": renosun_mini,
         "renosun-2k": lambda: renosun_bench("renosun-2k", 2048, 6144, 8, 16, 16),
         "renosun-4k": lambda: renosun_bench("renosun-4k", 4096, 12288, 16, 32, 32),
         "renosun-5k": lambda: renosun_bench("renosun-5k", 5120, 17408, 16, 48, 40)}
