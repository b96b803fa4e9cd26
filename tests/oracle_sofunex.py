"""Plain, slow restatement of the Sofunex decoder for tests: one function per mechanism, whole sequences at once,
float64 unless told otherwise.  Shares no code with the package under test.

Notation: a row vector x_t per token t; weights are [out, in] and applied as W x."""
from __future__ import annotations

import math

import torch


def rms(x, eps, w=None):
    y = x / torch.sqrt((x * x).mean(-1, keepdim=True) + eps)
    return y if w is None else y * w


def shifted(h, mu):
    """Every token reads a blend with the token before it (nothing is before the first)."""
    before = torch.cat([torch.zeros_like(h[:1]), h[:-1]])
    return h + (before - h) * mu


def causal_conv(u, w):
    """u [T, channels], w [channels, taps]: tap n - 1 meets the current token."""
    T, n = u.shape[0], w.shape[1]
    pad = torch.cat([torch.zeros(n - 1, u.shape[1], dtype=u.dtype), u])
    return sum(pad[j:j + T] * w[:, j] for j in range(n))


def rotate(x, rot):
    """x [T, heads, size]: column i of the first half of rot.dims turns with column i of the second."""
    n = rot["dims"]
    f = torch.tensor([rot["base"] ** (-2 * i / n) for i in range(n // 2)], dtype=torch.float64) / (rot.get("scaling") or {}).get("factor", 1.0)
    a = torch.arange(x.shape[0], dtype=torch.float64)[:, None, None] * f
    c, s = torch.cos(a).to(x.dtype), torch.sin(a).to(x.dtype)
    u, v = x[..., : n // 2], x[..., n // 2: n]
    return torch.cat([u * c - v * s, v * c + u * s, x[..., n:]], -1)


def window_weights(scores, size):
    """scores [H, T, T] -> softmax over the last `size` tokens, the query's own included (0: every earlier one)."""
    T = scores.shape[-1]
    d = torch.arange(T)[:, None] - torch.arange(T)[None, :]
    seen = (d >= 0) & (d < size) if size else d >= 0
    return torch.softmax(scores.masked_fill(~seen, float("-inf")), -1)


def window_attention(h, m, w, eps):
    T, H, G = h.shape[0], m["heads"], m["kv_heads"]
    q, k, v = (causal_conv(h @ w[n].T + w[n + ".b"], w[n + ".conv"]) for n in ("q", "k", "v"))
    q, k = (rotate(rms(x, eps, w[n + ".norm"]).view(T, -1, m["dim"]), m["rot"]) for n, x in (("q", q), ("k", k)))
    v = rms(v.view(T, G, m["vdim"]), eps)
    k, v = (x[:, torch.arange(H) // (H // G)] for x in (k, v))
    p = window_weights(torch.einsum("thd,shd->hts", q, k) * m["scale"], (m.get("mask") or {}).get("size", 0))
    return torch.einsum("hts,shv->thv", p, v).reshape(T, -1) @ w["o"].T + w["o.b"]


def channel_rates(h, w, heads):
    """(decay, removal rate) of every head's key channels."""
    T = h.shape[0]
    decay = torch.exp(-math.exp(-0.5) * torch.sigmoid(torch.tanh(h @ w["w1"].T) @ w["w2"].T + w["w0"]))
    return decay.view(T, heads, -1), torch.sigmoid(h @ w["a"].T + w["a.b"]).view(T, heads, -1)


def delta_states(r, k, v, decay, rate, state=None):
    """r, k, v, decay, rate [T, H, D] -> (read-outs [T, H, D], last state [H, key, value])."""
    T, H, D = r.shape
    S = torch.zeros(H, D, v.shape[-1], dtype=r.dtype) if state is None else state
    u = k / torch.sqrt((k * k).sum(-1, keepdim=True) + 1e-6)
    out = []
    for t in range(T):
        held = torch.einsum("hd,hdv->hv", u[t], S)
        S = decay[t][..., None] * S - (rate[t] * u[t])[..., None] * held[:, None] + k[t][..., None] * v[t][:, None]
        out.append(torch.einsum("hdv,hd->hv", S, r[t]))
    return torch.stack(out), S


def channel_delta(h, m, w, eps):
    T, H = h.shape[0], m["heads"]
    r, k, v = ((h @ w[n].T).view(T, H, m["dim"]) for n in ("r", "k", "v"))
    o, _ = delta_states(r, k, v, *channel_rates(h, w, H))
    return (rms(o, eps).reshape(T, -1) * w["norm"] * torch.sigmoid(h @ w["g"].T)) @ w["o"].T


def side_by_side(h, m, w, eps):
    sub = lambda side: {k[len(side) + 1:]: v for k, v in w.items() if k.startswith(side + ".")}      # noqa: E731
    return m["left_scale"] * window_attention(h, m["left"], sub("left"), eps) + m["right_scale"] * channel_delta(h, m["right"], sub("right"), eps)


def gelu_tanh(z):
    return z / 2 * (1 + torch.tanh(math.sqrt(2 / math.pi) * (z + 0.044715 * z ** 3)))


def silu(z):
    return z * torch.sigmoid(z)


def gated_ff(h, w, act, at=""):
    return (act(h @ w[at + "gate"].T) * (h @ w[at + "up"].T)) @ w[at + "down"].T


def route(scores, correction, top, groups):
    """[(expert, share)]: the best by corrected score among the `keep` groups whose two best members sum highest; shares of the plain scores."""
    c = [s + b for s, b in zip(scores, correction)]
    n = len(c) // groups["count"]
    strength = [sum(sorted(c[g * n:(g + 1) * n])[-2:]) for g in range(groups["count"])]
    kept = sorted(range(groups["count"]), key=lambda g: -strength[g])[: groups["keep"]]
    chosen = sorted((e for g in sorted(kept) for e in range(g * n, (g + 1) * n)), key=lambda e: -c[e])[:top]
    total = sum(scores[e] for e in chosen) + 1e-20
    return [(e, scores[e] / total) for e in chosen]


def moe_ff(h, m, w):
    r = m["router"]
    s, out = torch.sigmoid(h @ w["router"].T), torch.zeros_like(h)
    groups = r.get("groups") or {"count": 1, "keep": 1}
    for t in range(h.shape[0]):
        for e, share in route(s[t].tolist(), w["correction"].tolist(), r["top"], groups):
            out[t] += share * r["scale"] * gated_ff(h[t], w, silu, f"e{e}.")
    return out + gated_ff(h, w, silu, "shared.") if m.get("shared") else out


class Oracle:
    def __init__(self, cfg: dict, tensors: dict, dtype=torch.float64):
        self.cfg = cfg
        self.t = {k: v.to(dtype) for k, v in tensors.items()}
        self.eps = cfg["norm"]["eps"]

    def _sub(self, prefix):
        return {k[len(prefix):]: v for k, v in self.t.items() if k.startswith(prefix)}

    def _layer(self, i, x):
        spec, m, p = self.cfg["layers"][i], self.cfg["residual_mult"], f"l{i}."
        h = shifted(rms(x, self.eps, self.t[p + "norm1"]), self.t[p + "shift"])
        x = x + m * rms(side_by_side(h, spec["mixer"], self._sub(p + "mix."), self.eps), self.eps, self.t[p + "norm1b"])
        f = spec.get("mlp")
        if not f:
            return x
        h, w = rms(x, self.eps, self.t[p + "norm2"]), self._sub(p + "mlp.")
        return x + m * rms(gated_ff(h, w, gelu_tanh) if f["kind"] == "dense" else moe_ff(h, f, w), self.eps, self.t[p + "norm2b"])

    def order(self):
        """(layer, number of the pass that starts with it or None)"""
        n, lp = len(self.cfg["layers"]), self.cfg.get("loop")
        if not lp:
            return [(i, None) for i in range(n)]
        a, b = lp["start"], lp["stop"]
        return [(i, None) for i in range(a)] + [(i, t if i == a else None) for t in range(lp["times"]) for i in range(a, b)] + [(i, None) for i in range(b, n)]

    def forward(self, tokens, trace=None):
        """Logits [T, vocab]; `trace` (a list) receives the residual stream after every layer run."""
        x = self.t["embed"][torch.tensor(tokens)] * self.cfg["embedding"]["scale"]
        for i, enter in self.order():
            if enter is not None:
                x = x + self.t["loop.step"][enter]
            x = self._layer(i, x)
            if trace is not None:
                trace.append(x)
        return rms(x, self.eps, self.t["final.norm"]) @ self.t["head"].T

    def greedy(self, prompt, n):
        """(tokens, smallest gap between the best and the second logit on the way)."""
        ids, out, gap = list(prompt), [], float("inf")
        for _ in range(n):
            top = torch.topk(self.forward(ids)[-1], 2)
            gap = min(gap, float(top.values[0] - top.values[1]))
            out.append(int(top.indices[0]))
            ids.append(out[-1])
        return out, gap
