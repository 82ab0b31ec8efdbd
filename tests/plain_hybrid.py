"""Plain, slow restatement of the hybrid decoder's mechanisms: float64 on the CPU, one function per mechanism, one
sequence at a time, no caches.  It shares no code with the package (only reads its configuration objects)."""

from __future__ import annotations

import math

import torch


def rms(x, eps):
    return torch.sqrt((x * x).mean(-1, keepdim=True) + eps)


def norm(x, weight, eps, offset=1.0):
    return x / rms(x, eps) * (offset + weight)


def gelu(x):
    return 0.5 * x * (1 + torch.erf(x / math.sqrt(2)))


def gelu_tanh(x):
    return 0.5 * x * (1 + torch.tanh(math.sqrt(2 / math.pi) * (x + 0.044715 * x ** 3)))


def silu(x):
    return x / (1 + torch.exp(-x))


def softplus(x):
    return torch.where(x > 0, x + torch.log1p(torch.exp(-x.abs())), torch.log1p(torch.exp(-x.abs())))


def query_temperature(position: int, coef: float, every: int) -> float:
    return 1 + coef * math.log((position + 1) // every + 1)


def slope(head: int, heads: int) -> float:
    return 2.0 ** (-8.0 * (head + 1) / heads)


def attention(q, k, v, scale, coef=0.0, every=1, bias=True, first=0):
    """q [n, H, d] at positions first .. first + n - 1 over k [T, G, d], v [T, G, e]; returns [n, H, e]."""
    n, heads, _ = q.shape
    per_group = heads // k.shape[1]
    out = torch.zeros(n, heads, v.shape[2], dtype=torch.float64)
    for i in range(n):
        p = first + i
        for h in range(heads):
            g = h // per_group
            scores = (k[:p + 1, g] @ q[i, h]) * (scale * query_temperature(p, coef, every))
            if bias:
                scores = scores - slope(h, heads) * (p - torch.arange(p + 1, dtype=torch.float64))
            w = torch.exp(scores - scores.max())
            out[i, h] = (w / w.sum()) @ v[:p + 1, g]
    return out


def convolution(x, weight, bias):
    """Causal, per channel, silu; x [n, channels], weight [channels, taps] with the current token's tap last."""
    taps = weight.shape[1]
    out = torch.zeros_like(x)
    for i in range(x.shape[0]):
        for j in range(taps):
            source = i - (taps - 1) + j
            if source >= 0:
                out[i] += weight[:, j] * x[source]
    return silu(out + bias)


def recurrence(x, b, c, dt_raw, dt_bias, a_log, d, state=None):
    """x [n, H, P], b and c [n, G, N]; returns y [n, H, P] and the final state [H, N, P]."""
    n, heads, p = x.shape
    groups, size = b.shape[1:]
    s = torch.zeros(heads, size, p, dtype=torch.float64) if state is None else state.clone()
    y = torch.zeros_like(x)
    for t in range(n):
        dt = softplus(dt_raw[t] + dt_bias)
        for h in range(heads):
            g = h // (heads // groups)
            s[h] = torch.exp(-torch.exp(a_log[h]) * dt[h]) * s[h] + dt[h] * torch.outer(b[t, g], x[t, h])
            y[t, h] = s[h].T @ c[t, g] + d[h] * x[t, h]
    return y, s


def gated_norm(y, z, weight, parts, eps):
    y = y * silu(z)
    split = y.reshape(y.shape[0], parts, -1)
    return (split / rms(split, eps)).reshape(y.shape) * weight


class PlainHybrid:
    """The whole model over one token sequence.  `rounded`: what a 16-bit model may store in bf16 — inputs and outputs
    of matrix products, of the convolution and of the recurrence — is rounded to bf16, to see what that alone does."""

    def __init__(self, config, state_dict, rounded=False):
        self.config = config
        self.w = {name: t.double() for name, t in state_dict.items()}
        self.r = (lambda x: x.bfloat16().double()) if rounded else (lambda x: x)

    def _attention(self, i, m, h, kv):
        w, p, n, r = self.w, f"l{i}.mix.", h.shape[0], self.r
        q = r(h @ w[p + "q"].T).reshape(n, m.heads, m.dim)
        if m.kv_from is None:
            kv[i] = (r(h @ w[p + "k"].T).reshape(n, m.kv_heads, m.dim), r(h @ w[p + "v"].T).reshape(n, m.kv_heads, m.vdim))
        k, v = kv[i if m.kv_from is None else m.kv_from]
        return r(attention(q, k, v, m.scale, m.temp_coef, m.temp_every).reshape(n, -1)) @ w[p + "o"].T

    def _mamba2(self, i, m, h):
        w, p, n, r = self.w, f"l{i}.mix.", h.shape[0], self.r
        inner, gn = m.heads * m.vdim, m.groups * m.state
        z, xbc, dt = r(h @ w[p + "in"].T).split((inner, inner + 2 * gn, m.heads), 1)
        x, b, c = r(convolution(xbc, w[p + "conv"], w[p + "conv.b"])).split((inner, gn, gn), 1)
        y, _ = recurrence(x.reshape(n, m.heads, m.vdim), b.reshape(n, m.groups, m.state), c.reshape(n, m.groups, m.state), dt,
                          w[p + "dt_bias"], w[p + "A_log"], w[p + "D"])
        return r(gated_norm(r(y.reshape(n, inner)), z, w[p + "norm"], m.norm_groups, self.config.eps)) @ w[p + "o"].T

    def __call__(self, tokens, layers=None):
        """Logits [tokens, vocab]; `layers`, a list, receives the residual after every layer."""
        w, eps, kv, r = self.w, self.config.eps, {}, self.r
        x = w["embed"][torch.tensor(tokens)]
        for i, layer in enumerate(self.config.layers):
            h = r(norm(x, w[f"l{i}.norm1"], eps))
            mixed = self._attention(i, layer.mixer, h, kv) if hasattr(layer.mixer, "kv_heads") else self._mamba2(i, layer.mixer, h)
            if layer.ff:
                mixed = mixed + r(gelu(r(h @ w[f"l{i}.mlp.up"].T))) @ w[f"l{i}.mlp.down"].T
            x = x + r(mixed)
            if layers is not None:
                layers.append(x)
        return r(norm(x, w["final.norm"], eps)) @ w["head"].T
