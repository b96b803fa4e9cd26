"""Plain, slow restatement of the Renosun decoder for tests: one function per mechanism, whole
sequences at once or a token at a time, float64 unless told otherwise.  Shares no code with the
package under test.

Notation: a row vector x_t per token t; weights are [out, in] and applied as W x."""
from __future__ import annotations

import torch


def rms(x, eps, w=None):
    y = x / torch.sqrt((x * x).mean(-1, keepdim=True) + eps)
    return y if w is None else y * w


def unit(x):
    return x / torch.sqrt((x * x).sum(-1, keepdim=True) + 1e-6)


def silu(x):
    return x * torch.sigmoid(x)


def softplus(x):
    return torch.where(x > 30, x, torch.log1p(torch.exp(torch.clamp(x, max=30.0))))


def causal_conv_silu(x, w):
    """x [T, C], w [C, taps]: y_t = silu(sum_j w[:, j] x_{t - (taps - 1) + j}), zeros before the start."""
    T, taps = x.shape[0], w.shape[1]
    y = torch.zeros_like(x)
    for j in range(taps):
        back = taps - 1 - j
        if back < T:
            y[back:] += x[: T - back] * w[:, j]
    return silu(y)


def delta_rule(q, k, v, beta, g):
    """q, k [T, H, D], v [T, H, V], beta, g [T, H] -> o [T, H, V].  Decay, correct, write, then read."""
    T, H, D = q.shape
    S = torch.zeros(H, D, v.shape[-1], dtype=q.dtype)
    out = torch.zeros_like(v)
    for t in range(T):
        S = S * g[t][:, None, None]
        u = beta[t][:, None] * (v[t] - torch.einsum("hdv,hd->hv", S, k[t]))
        S = S + k[t][:, :, None] * u[:, None, :]
        out[t] = torch.einsum("hdv,hd->hv", S, q[t])
    return out


def delta_mixer(h, m, w, eps):
    """w: tensors by short name ('q', 'q.conv', ...)."""
    T = h.shape[0]
    H, HK, D, V = m["heads"], m["kv_heads"], m["dim"], m["vdim"]
    q = causal_conv_silu(h @ w["q"].T, w["q.conv"]).view(T, HK, D)
    k = causal_conv_silu(h @ w["k"].T, w["k.conv"]).view(T, HK, D)
    v = causal_conv_silu(h @ w["v"].T, w["v.conv"]).view(T, H, V)
    group = torch.arange(H) // (H // HK)
    q, k = unit(q)[:, group] * D ** -0.5, unit(k)[:, group]
    beta = torch.sigmoid(h @ w["b"].T)
    g = torch.exp(-torch.exp(w["A_log"]) * softplus(h @ w["a"].T + w["dt_bias"]))
    o = delta_rule(q, k, v, beta, g)
    o = rms(o, eps, w["norm"]) * silu(h @ w["g"].T).view(T, H, V)
    return o.reshape(T, H * V) @ w["o"].T


def rotate_half(x, pos, dims, base):
    """x [T, ..., D]: the first `dims` entries rotate, entry i with entry i + dims / 2."""
    half = dims // 2
    f = torch.tensor([base ** (-2.0 * i / dims) for i in range(half)], dtype=x.dtype)
    a = pos.to(x.dtype)[:, None] * f
    a = a.view(a.shape[0], *([1] * (x.dim() - 2)), half)
    u, v = x[..., :half], x[..., half:dims]
    return torch.cat([u * torch.cos(a) - v * torch.sin(a), v * torch.cos(a) + u * torch.sin(a), x[..., dims:]], -1)


def latent_attention(h, m, w, eps):
    T = h.shape[0]
    H, D, R, V, C = m["heads"], m["dim"], m["rot_dim"], m["vdim"], m["kv_rank"]
    pos = torch.arange(T)
    q = (h @ w["q"].T).view(T, H, D + R)
    down = h @ w["dkv"].T
    c = rms(down[:, :C], eps, w["dkv.norm"])
    kr = rotate_half(down[:, C:], pos, m["rot"]["dims"], m["rot"]["base"])
    qn, qr = q[..., :D], rotate_half(q[..., D:], pos, m["rot"]["dims"], m["rot"]["base"])
    kn = (c @ w["uk"].T).view(T, H, D)
    val = (c @ w["uv"].T).view(T, H, V)
    s = (torch.einsum("thd,shd->hts", qn, kn) + torch.einsum("thr,sr->hts", qr, kr)) * m["scale"]
    s = s.masked_fill(torch.arange(T)[None, :] > torch.arange(T)[:, None], float("-inf"))
    o = torch.einsum("hts,shv->thv", torch.softmax(s, -1), val).reshape(T, H * V)
    return (o * torch.sigmoid(h @ w["g"].T)) @ w["o"].T


def clamped_glu(h, limit, gate, up, down):
    g = torch.clamp(h @ gate.T, max=limit)
    u = torch.clamp(h @ up.T, -limit, limit)
    return (g * torch.sigmoid(1.702 * g) * (u + 1)) @ down.T


MIXERS = {"delta": delta_mixer, "latent_attention": latent_attention}


class Oracle:
    def __init__(self, cfg: dict, tensors: dict, dtype=torch.float64):
        self.cfg = cfg
        self.t = {k: v.to(dtype) for k, v in tensors.items()}
        self.eps = cfg["norm"]["eps"]

    def _sub(self, prefix):
        return {k[len(prefix):]: v for k, v in self.t.items() if k.startswith(prefix)}

    def order(self):
        """(layer, pass or None, first of its pass) in running order."""
        n, lp = len(self.cfg["layers"]), self.cfg.get("loop")
        if not lp:
            return [(i, None, False) for i in range(n)]
        out = [(i, None, False) for i in range(lp["start"])]
        for t in range(lp["times"]):
            out += [(i, t, i == lp["start"]) for i in range(lp["start"], lp["stop"])]
        return out + [(i, None, False) for i in range(lp["stop"], n)]

    def layer(self, i, x):
        spec = self.cfg["layers"][i]
        h = rms(x, self.eps, self.t[f"l{i}.norm1"])
        y = MIXERS[spec["type"]](h, spec["mixer"], self._sub(f"l{i}.mix."), self.eps)
        if spec.get("mlp"):
            f = self._sub(f"l{i}.mlp.")
            y = y + clamped_glu(h, spec["mlp"]["limit"], f["gate"], f["up"], f["down"])
        return x + y

    def forward(self, tokens, trace=None):
        """Logits [T, vocab]; `trace` (a list) receives the residual stream after every layer run."""
        x0 = self.t["embed"][torch.tensor(tokens)] * self.cfg["embedding"]["scale"]
        x = x0
        for i, t, first in self.order():
            if first:
                x = torch.cat([x, x0], -1) @ self.t["loop.in"].T + self.t["loop.step"][t]
            x = self.layer(i, x)
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
