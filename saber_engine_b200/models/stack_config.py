"""Decoders described layer by layer: an ordered list of layers, each with its mixer and feed-forward, an
optional block of layers that runs several times, and the constants of both.  `models.stack.StackModel` runs
any such description; an architecture is a reader of its `config.json` (ARCHITECTURES) and the order and
names of its tensors (`models.stack_weights`).
"""
from __future__ import annotations

import json
import os
from dataclasses import dataclass
from pathlib import Path
from typing import Optional


@dataclass(frozen=True)
class DeltaMixer:
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
    def dim_pad(self) -> int:         # key sizes the kernels are instantiated for
        for n in (64, 128, 192, 256, 384, 512):
            if n >= self.dim:
                return n
        raise ValueError(f"delta mixer: key size {self.dim} is above 512")

    @property
    def vdim_pad(self) -> int:
        return (self.vdim + 7) // 8 * 8

    def segments(self) -> list:
        """(name, rows) of the input projection."""
        return [("q", self.kv_heads * self.dim), ("k", self.kv_heads * self.dim), ("v", self.heads * self.vdim),
                ("b", self.heads), ("a", self.heads), ("g", self.heads * self.vdim)]

    def slot_bytes(self) -> int:
        return 4 * (self.heads * self.vdim_pad * self.dim_pad + self.taps * self.channels)

    def page_token_bytes(self, elem: int) -> int:
        return 0


@dataclass(frozen=True)
class LatentMixer:
    """Latent attention: a cached latent of kv_rank values and one rotated key part of rot_dim per token."""
    heads: int
    dim: int
    rot_dim: int
    vdim: int
    kv_rank: int
    scale: float
    rot_base: float
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
        return [("q", self.heads * (self.dim + self.rot_dim)), ("dkv", self.kv_rank + self.rot_dim), ("g", self.heads * self.vdim)]

    def slot_bytes(self) -> int:
        return 0

    def page_token_bytes(self, elem: int) -> int:
        return elem * (self.rank_pad + self.rot_pad)

    @property
    def key_tile(self) -> int:        # an expanded key in whole 64-wide tiles
        return (self.dim_pad + self.rot_pad + 63) // 64 * 64

    def expanded_token_bytes(self, elem: int) -> int:
        return elem * self.heads * (self.key_tile + self.vdim_pad)


@dataclass(frozen=True)
class ClampedGlu:
    """g = min(gate, limit), u = clamp(up, -limit, limit), y = g sigmoid(alpha g) (u + 1)."""
    ff: int
    limit: float
    alpha: float = 1.702


@dataclass(frozen=True)
class LayerSpec:
    mixer: object
    mlp: Optional[ClampedGlu] = None


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
            if isinstance(m, LatentMixer) and (m.rot_dim % 2 or m.kv_rank > 1024 or m.dim > 1024):
                raise ValueError(f"{self.name}: layer {i}: rot_dim {m.rot_dim}, kv_rank {m.kv_rank}, dim {m.dim}")

    # ---- byte accounting (launch plan)
    def page_token_bytes(self, elem: int = 2) -> int:
        return sum(self.layers[r.layer].mixer.page_token_bytes(elem) for r in self.runs)

    def slot_bytes(self) -> int:
        return sum(self.layers[r.layer].mixer.slot_bytes() for r in self.runs)

    def expanded_token_bytes(self, elem: int = 2) -> int:
        return max([l.mixer.expanded_token_bytes(elem) for l in self.layers if isinstance(l.mixer, LatentMixer)], default=0)

    def widest_project(self) -> int:
        return max(sum(n for _, n in l.mixer.segments()) for l in self.layers)

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
            mixer = LatentMixer(m["heads"], m["dim"], m["rot_dim"], m["vdim"], m["kv_rank"], float(m["scale"]), float(m["rot"]["base"]))
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


ARCHITECTURES = {"Renosun": renosun_from_json}


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
    a = LayerSpec(LatentMixer(3, 64, 32, 40, 96, 96 ** -0.5, 1e4), ClampedGlu(384, 4.0))
    return StackConfig("renosun-mini", "Renosun", vocab=1024, width=320, layers=(a, d, d, a, d), embed_scale=8.0, loop=LoopSpec(1, 4, 2),
                       max_ctx=4096)


def renosun_bench(name: str, width: int, ff: int, kv_heads: int, heads: int, attn_heads: int, n_layers: int = 8, vocab: int = 65536) -> StackConfig:
    """Layers of a real model's size: three delta layers to one attention layer."""
    d = LayerSpec(DeltaMixer(heads, kv_heads, 128, 128, 4), ClampedGlu(ff, 7.0))
    a = LayerSpec(LatentMixer(attn_heads, 128, 64, 128, 512, 192 ** -0.5, 1e6), ClampedGlu(ff, 7.0))
    layers = tuple(a if i % 4 == 3 else d for i in range(n_layers))
    return StackConfig(name, "Renosun", vocab=vocab, width=width, layers=layers, embed_scale=width ** 0.5, loop=LoopSpec(n_layers // 4, n_layers // 2, 2))


NAMED = {"renosun-mini": renosun_mini,
         "renosun-2k": lambda: renosun_bench("renosun-2k", 2048, 6144, 8, 16, 16),
         "renosun-4k": lambda: renosun_bench("renosun-4k", 4096, 12288, 16, 32, 32),
         "renosun-5k": lambda: renosun_bench("renosun-5k", 5120, 17408, 16, 48, 40)}
