"""Plain, slow restatement of the Fitatar decoder for tests: one function per mechanism, whole sequences at once,
float64 unless told otherwise.  Shares no code with the package under test.

Notation: a row vector x_t per token t; weights are [out, in] and applied as W x."""
from __future__ import annotations

import math

import torch


def rms(x, eps, w):
    return x / torch.sqrt((x * x).mean(-1, keepdim=True) + eps) * w


def frequencies(base, dims, scaling):
    """(f_i for each of the dims / 2 pairs, factor on cosine and sine)."""
    f = [base ** (-2 * i / dims) for i in range(dims // 2)]
    if not scaling:
        return torch.tensor(f, dtype=torch.float64), 1.0
    s = scaling["factor"]
    if "fast" not in scaling:                                    # every position divided by s
        return torch.tensor([x / s for x in f], dtype=torch.float64), 1.0

    def turns(t):                                                # the (fractional) index whose pair makes t turns over `original` positions
        return dims * math.log(scaling["original"] / (2 * math.pi * t)) / (2 * math.log(base))
    lo, hi = max(math.floor(turns(scaling["fast"])), 0), min(math.ceil(turns(scaling["slow"])), dims - 1)
    out = []
    for i, x in enumerate(f):
        ramp = min(max((i - lo) / max(hi - lo, 0.001), 0.0), 1.0)
        out.append(x / s * ramp + x * (1 - ramp))
    return torch.tensor(out, dtype=torch.float64), 0.1 * math.log(s) + 1


def rotate(x, rot, interleaved):
    """x [T, heads, size]: the first rot.dims columns turn with the position, the rest stay."""
    n = rot["dims"]
    f, amp = frequencies(rot["base"], n, rot.get("scaling"))
    a = torch.arange(x.shape[0], dtype=torch.float64)[:, None, None] * f
    c, s = (amp * torch.cos(a)).to(x.dtype), (amp * torch.sin(a)).to(x.dtype)
    first, second = (slice(0, n, 2), slice(1, n, 2)) if interleaved else (slice(0, n // 2), slice(n // 2, n))
    u, v, out = x[..., first], x[..., second], x.clone()
    out[..., first], out[..., second] = u * c - v * s, v * c + u * s
    return out


def causal_weights(scores, sink=None):
    """scores [H, T, T] -> softmax over keys not later than the query; sink [H]: one more logit without key and value."""
    T = scores.shape[-1]
    s = scores.masked_fill(torch.ones(T, T).triu(1).bool(), float("-inf"))
    if sink is not None:
        s = torch.cat([s, sink[:, None, None].expand(-1, T, 1)], -1)
    return torch.softmax(s, -1)[..., :T]


def latent_mixer(h, m, w, eps, kv=None):
    """kv: another layer's (latents, rotated key parts), used instead of this layer's own."""
    T, H, D, R, C = h.shape[0], m["heads"], m["dim"], m["rot_dim"], m["kv_rank"]
    q = (rms(h @ w["dq"].T, eps, w["dq.norm"]) @ w["uq"].T).view(T, H, D + R)
    qn, qr = q[..., :D], rotate(q[..., D:], m["rot"], True)
    if kv is None:
        d = h @ w["dkv"].T
        kv = rms(d[:, :C], eps, w["dkv.norm"]), rotate(d[:, None, C:], m["rot"], True)[:, 0]
    c, kr = kv
    k, v = (c @ w["uk"].T).view(T, H, D), (c @ w["uv"].T).view(T, H, m["vdim"])
    s = (torch.einsum("thd,shd->hts", qn, k) + torch.einsum("thr,sr->hts", qr, kr)) * m["scale"]
    o = torch.einsum("hts,shv->thv", causal_weights(s), v) * torch.sigmoid(h @ w["g"].T)[..., None]
    return o.reshape(T, -1) @ w["o"].T, kv


def attention_mixer(h, m, w, eps, kv=None):
    T, H, G = h.shape[0], m["heads"], m["kv_heads"]
    q, k = (rotate((h @ w[n].T).view(T, heads, m["dim"]), m["rot"], False) for n, heads in (("q", H), ("k", G)))
    v = (h @ w["v"].T).view(T, G, m["vdim"])
    k, v = (x[:, torch.arange(H) // (H // G)] for x in (k, v))
    p = causal_weights(torch.einsum("thd,shd->hts", q, k) * m["scale"], w["sink"])
    o = torch.einsum("hts,shv->thv", p, v).reshape(T, -1) * torch.sigmoid(h @ w["g"].T)
    return o @ w["o"].T, None


def gelu(z):
    return z * (1 + torch.erf(z / math.sqrt(2))) / 2


def dense_ff(h, m, w):
    return gelu(h @ w["up"].T + w["up.b"]) @ w["down"].T + w["down.b"]


def squared_relu_ff(h, up, down):
    return torch.relu(h @ up.T) ** 2 @ down.T


def route(scores, top, groups):
    """scores [E] -> chosen experts: the `top` best of the `keep` groups whose best member is best."""
    n = len(scores) // groups["count"]
    best = sorted(range(groups["count"]), key=lambda g: -max(scores[g * n:(g + 1) * n]))[: groups["keep"]]
    return sorted((e for g in best for e in range(g * n, (g + 1) * n)), key=lambda e: -scores[e])[:top]


def moe_ff(h, m, w):
    r = m["router"]
    s = torch.softmax(h @ w["router"].T, -1)
    out = torch.zeros_like(h)
    for t in range(h.shape[0]):
        for e in route(s[t].tolist(), r["top"], r["groups"]):
            out[t] += s[t, e] * squared_relu_ff(h[t], w[f"e{e}.up"], w[f"e{e}.down"])
    if m.get("shared"):
        out = out + squared_relu_ff(h, w["shared.up"], w["shared.down"]) * torch.sigmoid(h @ w["shared.sg"].T)
    return out


MIXERS = {"latent_attention": latent_mixer, "attention": attention_mixer}
FEED_FORWARDS = {"dense": dense_ff, "moe": moe_ff}


class Oracle:
    def __init__(self, cfg: dict, tensors: dict, dtype=torch.float64):
        self.cfg = cfg
        self.t = {k: v.to(dtype) for k, v in tensors.items()}
        self.eps = cfg["norm"]["eps"]

    def _sub(self, prefix):
        return {k[len(prefix):]: v for k, v in self.t.items() if k.startswith(prefix)}

    def forward(self, tokens, trace=None):
        """Logits [T, vocab]; `trace` (a list) receives the residual stream after every layer."""
        x = self.t["embed"][torch.tensor(tokens)] * self.cfg["embedding"]["scale"]
        kvs = []
        for i, spec in enumerate(self.cfg["layers"]):
            m, src = spec["mixer"], spec["mixer"].get("kv_from")
            y, kv = MIXERS[spec["type"]](rms(x, self.eps, self.t[f"l{i}.norm1"]), m, self._sub(f"l{i}.mix."), self.eps, None if src is None else kvs[src])
            kvs.append(kv)
            if spec.get("mlp"):
                y = y + FEED_FORWARDS[spec["mlp"]["kind"]](rms(x, self.eps, self.t[f"l{i}.norm2"]), spec["mlp"], self._sub(f"l{i}.mlp."))
            x = x + y
            if trace is not None:
                trace.append(x)
        z = rms(x, self.eps, self.t["final.norm"]) @ self.t["head"].T
        cap = self.cfg["logit_softcap"]
        return cap * torch.tanh(z / cap)

    def greedy(self, prompt, n):
        """(tokens, smallest gap between the best and the second logit on the way)."""
        ids, out, gap = list(prompt), [], float("inf")
        for _ in range(n):
            top = torch.topk(self.forward(ids)[-1], 2)
            gap = min(gap, float(top.values[0] - top.values[1]))
            out.append(int(top.indices[0]))
            ids.append(out[-1])
        return out, gap
