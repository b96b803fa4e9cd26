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
    chunk of positions, a learned number per head in the denominator, an output gate; each where asked for.  kv_from: the pages
    of that layer are read, with this layer's queries and mask."""
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
    kind = "attention"

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
        return {"sink": (self.heads,)} if self.sink else {}

    def page_token_bytes(self, elem: int) -> int:
        return 0 if self.kv_from is not None else elem * self.kv_heads * (self.key_pad + self.vdim_pad)


class FeedForward:
    """What a layer asks of its feed-forward.  Its rows are tiles of 256 behind the mixer's: `per_tile` features each."""
    act_kind = 0                      # the linear epilogue's activation
    per_tile = 256
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
    per_tile = 128

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


@dataclass(frozen=True)
class ExpertMix(FeedForward):
    """Mixture of squared-ReLU experts: softmax over `experts` scores, the `top` best of the `keep` groups of neighbours whose best
    score is best, weighted by their scores as they are.  shared: the size of one more expert for every token, times the
    sigmoid of a number of its own."""
    experts: int
    top: int
    ff: int
    groups: int = 1
    keep: int = 1
    shared: int = 0
    act_kind = 2
    per_tile = 248                    # and the shared expert's gate row behind them

    @property
    def inner(self) -> int:
        return self.shared

    def shapes(self, width: int) -> dict:
        t = {}
        for e in range(self.experts):
            t[f"e{e}.up"], t[f"e{e}.down"] = (self.ff, width), (width, self.ff)
        t["router"] = (self.experts, width)
        if self.shared:
            t.update({"shared.up": (self.shared, width), "shared.down": (width, self.shared), "shared.sg": (1, width)})
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
    loop: Optional[LoopSpec] = None
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
            if not self.parallel and isinstance(l.mlp, (Gelu, ExpertMix)):
                raise ValueError(f"{self.name}: layer {i}: {type(l.mlp).__name__} stands beside its mixer only")
            if isinstance(l.mlp, ExpertMix):
                self._check_experts(i, l.mlp)
            if isinstance(m, LatentMixer):
                if m.rot_dim % 2 or m.kv_rank > 1024 or m.dim > 1024 or m.rot.dims != m.rot_dim:
                    raise ValueError(f"{self.name}: layer {i}: rot_dim {m.rot_dim} (rotated {m.rot.dims}), kv_rank {m.kv_rank}, dim {m.dim}")
                self._check_source(i, m, lambda s: (s.kv_rank, s.rot_dim, s.rot))
        if self.two_norms and (not self.parallel or self.loop is not None):
            raise ValueError(f"{self.name}: a second norm needs layers side by side and no loop")

    def _check_experts(self, i: int, f: ExpertMix) -> None:
        if not (1 <= f.experts <= 1024 and 1 <= f.top <= 32 and f.groups >= 1 and f.experts % f.groups == 0 and 1 <= f.keep <= f.groups
                and f.top <= f.experts // f.groups * f.keep):
            raise ValueError(f"{self.name}: layer {i}: top {f.top} of {f.experts} experts in {f.keep} of {f.groups} groups")
        if not self.two_norms:
            raise ValueError(f"{self.name}: layer {i}: a mixture of experts reads a norm of its own")

    def _check_source(self, i: int, m: Mixer, sizes) -> None:
        """A layer that reads another's pages finds a layer of its kind and sizes there."""
        if m.kv_from is None:
            return
        s = self.layers[m.kv_from].mixer if 0 <= m.kv_from < i else None
        if self.loop is not None or type(s) is not type(m) or s.kv_from is not None or sizes(s) != sizes(m):
            raise ValueError(f"{self.name}: layer {i} cannot read the keys and values of layer {m.kv_from}")

    def _check_grouped(self, i: int, m: GroupedMixer) -> None:
        if m.heads % m.kv_heads or m.chunk < 0 or m.dim > 2048 or m.vdim > 2048:
            raise ValueError(f"{self.name}: layer {i}: heads {m.heads} / kv_heads {m.kv_heads} / chunk {m.chunk} / dim {m.dim} / vdim {m.vdim}")
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
        return sum(self.layers[r.layer].mixer.slot_bytes() for r in self.runs)

    def expanded_token_bytes(self, elem: int = 2) -> int:
        return max([l.mixer.expanded_token_bytes(elem) for l in self.layers if isinstance(l.mixer, LatentMixer)], default=0)

    def widest_project(self) -> int:
        return max(sum(n for _, n in l.mixer.segments()) + (l.mixer.query_rows if l.mixer.q_rank else 0) for l in self.layers)

    def expert_row_bytes(self, rows: int, elem: int = 2) -> int:
        """Scratch of the routed rows of a step (one layer at a time)."""
        return max([rows * l.mlp.top * elem * (l.mlp.ff + self.width) for l in self.layers if isinstance(l.mlp, ExpertMix)], default=0)

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
def renosun_from_json(doc: dict, name: str = "renosun", source: Optional[str] = None, max_ctx: int = 32768) -> StackConfig:
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
def tepavik_from_json(doc: dict, name: str = "tepavik", source: Optional[str] = None, max_ctx: int = 32768) -> StackConfig:
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
def fitatar_from_json(doc: dict, name: str = "fitatar", source: Optional[str] = None, max_ctx: int = 32768) -> StackConfig:
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


ARCHITECTURES = {"Renosun": renosun_from_json, "Tepavik": tepavik_from_json, "Fitatar": fitatar_from_json}


def from_json(doc: dict, **kw) -> StackConfig:
    arch = doc.get("architecture")
    if arch not in ARCHITECTURES:
        raise KeyError(f"unknown architecture {arch!r}; known: {sorted(ARCHITECTURES)}")
    return ARCHITECTURES[arch](doc, **kw)


def is_model_dir(path: str) -> bool:
    return os.path.isfile(os.path.join(path, "config.json"))


def load_dir(path: str) -> StackConfig:
    """The description in a model folder (config.json beside model.safetensors)."""
    p = Path(path)
    return from_json(json.loads((p / "config.json").read_text()), name=p.resolve().name, source=str(p))


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


NAMED = {"fitatar-mini": fitatar_mini,
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
