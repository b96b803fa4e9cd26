"""Plain, slow restatement of the Tepavik decoder for tests: one function per mechanism, whole sequences at
once, float64 unless told otherwise.  Shares no code with the package under test.

Notation: a row vector x_t per token t; weights are [out, in] and applied as W x."""
from __future__ import annotations

import torch


def rms(x, eps):
    return x / torch.sqrt((x * x).mean(-1, keepdim=True) + eps)


def norm_around_zero(x, eps, w):
    return rms(x, eps) * (1 + w)


def silu(x):
    return x * torch.sigmoid(x)


def softplus(x):
    return torch.where(x > 30, x, torch.log1p(torch.exp(torch.clamp(x, max=30.0))))


def causal_conv(x, w, b):
    """x [T, C], w [C, taps], b [C]: y_t = b + sum_j w[:, j] x_{t - (taps - 1) + j}, zeros before the start."""
    T, taps = x.shape[0], w.shape[1]
    y = b.expand(T, -1).clone()
    for j in range(taps):
        back = taps - 1 - j
        if back < T:
            y[back:] += x[: T - back] * w[:, j]
    return y


def decayed_outer_products(q, k, v, a):
    """q, k [T, H, N], v [T, H, V], a [T, H]: S_t = a_t S_{t-1} + k_t v_t^T, o_t = S_t^T q_t, from S = 0."""
    T, H, N = q.shape
    S = torch.zeros(H, N, v.shape[-1], dtype=q.dtype)
    out = torch.zeros_like(v)
    for t in range(T):
        S = a[t][:, None, None] * S + k[t][:, :, None] * v[t][:, None, :]
        out[t] = (S * q[t][:, :, None]).sum(1)
    return out


def lightning_mixer(h, m, w, eps, kv=None):
    T, H, V = h.shape[0], m["heads"], m["vdim"]
    q, k, v = (silu(h @ w[n].T).view(T, H, -1) for n in ("q", "k", "v"))
    a = torch.tensor(m["decay"], dtype=h.dtype).expand(T, H)
    o = decayed_outer_products(q, k, v, a).reshape(T, H * V)
    return (rms(o, eps) * w["norm"] * torch.sigmoid(h @ w["g"].T)) @ w["o"].T, None


def mamba2_mixer(h, m, w, eps, kv=None):
    T, H, V, N, G = h.shape[0], m["heads"], m["vdim"], m["state"], m["groups"]
    inner = H * V
    z, xbc, dt = torch.split(h @ w["in"].T, [inner, inner + 2 * G * N, H], -1)
    x, B, C = torch.split(silu(causal_conv(xbc, w["conv"], w["conv.b"])), [inner, G * N, G * N], -1)
    x = x.reshape(T, H, V)
    group = torch.arange(H) // (H // G)
    B, C = B.reshape(T, G, N)[:, group], C.reshape(T, G, N)[:, group]
    dt = softplus(dt + w["dt_bias"])
    a = torch.exp(-torch.exp(w["A_log"]) * dt)
    y = decayed_outer_products(C, B, dt[:, :, None] * x, a) + w["D"][:, None] * x
    y = (y.reshape(T, inner) * silu(z)).view(T, m["norm_groups"], inner // m["norm_groups"])
    return (rms(y, eps).reshape(T, inner) * w["norm"]) @ w["o"].T, None


def visible(T, size):
    """[query, key]: not later than the query and in the same chunk of `size` positions."""
    i, j = torch.arange(T)[:, None], torch.arange(T)[None, :]
    return (j <= i) & (i // size == j // size)


def attention_mixer(h, m, w, eps, kv=None):
    """kv: another layer's (keys, values), used instead of this layer's own."""
    T, H, G, D, V = h.shape[0], m["heads"], m["kv_heads"], m["dim"], m["vdim"]
    proj = lambda n, heads, size: (h @ w[n].T + w[n + ".b"]).view(T, heads, size)    # noqa: E731
    q = rms(proj("q", H, D), eps)
    if kv is None:
        kv = rms(proj("k", G, D), eps), proj("v", G, V)
    k, v = (x[:, torch.arange(H) // (H // G)] for x in kv)
    s = torch.einsum("thd,shd->hts", q, k) * m["scale"]
    s = m["softcap"] * torch.tanh(s / m["softcap"])
    s = s.masked_fill(~visible(T, m["mask"]["size"]), float("-inf"))
    o = torch.einsum("hts,shv->thv", torch.softmax(s, -1), v).reshape(T, H * V)
    return o @ w["o"].T, kv


def squared_relu_ff(h, up, down):
    return torch.relu(h @ up.T) ** 2 @ down.T


MIXERS = {"lightning": lightning_mixer, "mamba2": mamba2_mixer, "attention": attention_mixer}


class Oracle:
    def __init__(self, cfg: dict, tensors: dict, dtype=torch.float64):
        self.cfg = cfg
        self.t = {k: v.to(dtype) for k, v in tensors.items()}
        self.eps = cfg["norm"]["eps"]

    def _sub(self, prefix):
        return {k[len(prefix):]: v for k, v in self.t.items() if k.startswith(prefix)}

    def forward(self, tokens, trace=None):
        """Logits [T, vocab]; `trace` (a list) receives the residual stream after every layer."""
        x = self.t["embed"][torch.tensor(tokens)]
        kvs = []
        for i, spec in enumerate(self.cfg["layers"]):
            m = spec["mixer"]
            h = norm_around_zero(x, self.eps, self.t[f"l{i}.norm1"])
            src = m.get("kv_from")
            y, kv = MIXERS[spec["type"]](h, m, self._sub(f"l{i}.mix."), self.eps, None if src is None else kvs[src])
            kvs.append(kv)
            x = x + y
            if spec.get("mlp"):
                h = norm_around_zero(x, self.eps, self.t[f"l{i}.norm2"])
                x = x + squared_relu_ff(h, self.t[f"l{i}.mlp.up"], self.t[f"l{i}.mlp.down"])
            if trace is not None:
                trace.append(x)
        return norm_around_zero(x, self.eps, self.t["final.norm"]) @ self.t["head"].T

    def greedy(self, prompt, n):
        """(tokens, smallest gap between the best and the second logit on the way)."""
        ids, out, gap = list(prompt), [], float("inf")
        for _ in range(n):
            top = torch.topk(self.forward(ids)[-1], 2)
            gap = min(gap, float(top.values[0] - top.values[1]))
            out.append(int(top.indices[0]))
            ids.append(out[-1])
        return out, gap
