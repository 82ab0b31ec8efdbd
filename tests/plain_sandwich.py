"""Plain, slow restatement of the mechanisms of a decoder with a norm on both sides of every sublayer: float64 on the CPU, one
function per mechanism, one sequence at a time, no caches.  It shares no code with the package and reads the JSON configuration
itself."""

from __future__ import annotations

import math

import torch


def layer_norm(x, weight, eps):
    centred = x - x.mean(-1, keepdim=True)
    return centred / torch.sqrt((centred * centred).mean(-1, keepdim=True) + eps) * weight


def rms_norm(x, weight, eps):
    return x / torch.sqrt((x * x).mean(-1, keepdim=True) + eps) * weight


def sigmoid(x):
    return 1 / (1 + torch.exp(-x))


def gelu_tanh(z):
    return 0.5 * z * (1 + torch.tanh(math.sqrt(2 / math.pi) * (z + 0.044715 * z ** 3)))


def soft_cap(x, cap):
    return cap * torch.tanh(x / cap)


def frequencies(base, dims, scaling=None):
    """Turns per position of every pair, and the amplitude of the turned pairs."""
    turns = [base ** (-2.0 * i / dims) for i in range(dims // 2)]
    if not scaling:
        return turns, 1.0
    def pair_that_makes(t):                      # the (real) index of the pair that makes t turns over the original length
        return dims * math.log(scaling["original"] / (2 * math.pi * t)) / (2 * math.log(base))
    low = max(math.floor(pair_that_makes(scaling["fast"])), 0)
    high = min(math.ceil(pair_that_makes(scaling["slow"])), dims - 1)
    out = []
    for i, f in enumerate(turns):
        slow_share = min(max((i - low) / max(high - low, 0.001), 0.0), 1.0)
        out.append(f / scaling["factor"] * slow_share + f * (1 - slow_share))
    return out, 0.1 * math.log(scaling["factor"]) + 1


def rotate(x, positions, turns, amplitude=1.0):
    """x [n, ..., d]: pairs (i, i + dims / 2) of the first dims = 2 * len(turns) dimensions turned by position * turns[i] and
    stretched by the amplitude."""
    y, half = x.clone(), len(turns)
    for i, f in enumerate(turns):
        angle = positions.double() * f
        c, s = ((amplitude * g(angle)).reshape(-1, *[1] * (x.dim() - 2)) for g in (torch.cos, torch.sin))
        u, v = x[..., i], x[..., i + half]
        y[..., i], y[..., i + half] = u * c - v * s, v * c + u * s
    return y


def attention(q, k, v, scale, window=0, sink=None, first=0):
    """q [n, H, d] at positions first .. over k [T, G, d], v [T, G, e]: query head h reads key/value head h // (H / G); a row sees
    itself and the window - 1 keys before it (window 0: all of them); sink [H]: one more term of a head's denominator."""
    n, heads, share = q.shape[0], q.shape[1], q.shape[1] // k.shape[1]
    group = torch.arange(heads) // share
    out = torch.zeros(n, heads, v.shape[2], dtype=torch.float64)
    for i in range(n):
        p = first + i
        lo = max(p - window + 1, 0) if window else 0
        scores = torch.einsum("hd,thd->ht", q[i], k[lo:p + 1, group]) * scale
        top = scores.amax(1)
        if sink is not None:
            top = torch.maximum(top, sink)
        weights = torch.exp(scores - top[:, None])
        total = weights.sum(1)
        if sink is not None:
            total = total + torch.exp(sink - top)
        out[i] = torch.einsum("ht,the->he", weights, v[lo:p + 1, group]) / total[:, None]
    return out


def short_conv(u, weight):
    """u [n, C], weight [C, taps]: y_t = sum_j weight[:, j] u_(t - taps + 1 + j), nothing before the start."""
    n, taps = u.shape[0], weight.shape[1]
    y = torch.zeros_like(u)
    for t in range(n):
        for j in range(taps):
            if t - taps + 1 + j >= 0:
                y[t] = y[t] + weight[:, j] * u[t - taps + 1 + j]
    return y


def gated_unit(h, gate, up, down, r=lambda x: x):
    return r(gelu_tanh(r(h @ gate.T)) * r(h @ up.T)) @ down.T


class PlainSandwich:
    """The whole model over one token sequence.  `rounded` (1, 2, ..): what a 16-bit model may store in bf16 is rounded to bf16, to
    see what that alone does; from 2 on after a random shift of up to half a unit in the last place (other roundings, as
    another order of summation gives)."""

    def __init__(self, config: dict, state_dict, rounded=0):
        self.config = config
        self.w = {name: t.double() for name, t in state_dict.items()}
        g = torch.Generator().manual_seed(rounded)
        shift = lambda x: x * (1 + (torch.rand(x.shape, generator=g).double() - 0.5) * 2.0 ** -8) if rounded > 1 else x
        self.r = (lambda x: shift(x).bfloat16().double()) if rounded else (lambda x: x)
        self.eps = config["norm"]["eps"]

    def latent(self, p, m, h, second):
        """`second`: the kind with a sink, scaled frequencies and one gate per head; else one gate per element."""
        w, r, n, heads, d = self.w, self.r, h.shape[0], m["heads"], m["dim"]
        turns, amplitude = frequencies(m["rot"]["base"], m["rot"]["dims"], m["rot"].get("scaling") if second else None)
        turn = lambda x: r(rotate(x, torch.arange(n), turns, amplitude))
        c_q = r(rms_norm(r(h @ w[p + "dq"].T), w[p + "dq.norm"], self.eps))
        q = r(c_q @ w[p + "uq"].T).reshape(n, heads, -1)
        q = torch.cat([q[..., :d], turn(q[..., d:])], -1)
        down = r(h @ w[p + "dkv"].T)
        c = r(rms_norm(down[:, :m["kv_rank"]], w[p + "dkv.norm"], self.eps))
        shared = turn(down[:, m["kv_rank"]:])
        k = torch.cat([r(c @ w[p + "uk"].T).reshape(n, heads, d), shared[:, None].expand(n, heads, -1)], -1)
        v = r(c @ w[p + "uv"].T).reshape(n, heads, m["vdim"])
        out = r(attention(q, k, v, m["scale"], sink=w[p + "sink"] if second else None))
        gate = sigmoid(r(h @ w[p + "g"].T)).reshape(n, heads, -1)
        return r((out * gate).reshape(n, -1)) @ w[p + "o"].T

    def windowed(self, p, m, h):
        w, r, n = self.w, self.r, h.shape[0]
        q, k, v = (short_conv(r(h @ w[p + x].T + w[p + x + ".b"]), w[p + x + ".conv"]) for x in "qkv")
        q, k = (r(rms_norm(r(x).reshape(n, -1, m["dim"]), 1.0, self.eps)) for x in (q, k))
        out = r(attention(q, k, r(v).reshape(n, -1, m["vdim"]), m["scale"], m["mask"]["size"]))
        return r(out.reshape(n, -1) * sigmoid(r(h @ w[p + "g"].T))) @ w[p + "o"].T

    def __call__(self, tokens, layers=None):
        """Logits [tokens, vocab]; `layers`, a list, receives the residual after every layer."""
        w, c, r = self.w, self.config, self.r
        x = w["embed"][torch.tensor(tokens)]
        for i, entry in enumerate(c["layers"]):
            p, m = f"l{i}.", entry["mixer"]
            h = r(layer_norm(x, w[p + "norm1"], self.eps))
            y = self.windowed(p + "mix.", m, h) if entry["type"] == "attention" else \
                self.latent(p + "mix.", m, h, entry["type"] == "latent_attention_2")
            x = x + c["residual_mult"] * layer_norm(r(y), w[p + "norm1b"], self.eps)
            if entry["mlp"]:
                h = r(layer_norm(x, w[p + "norm2"], self.eps))
                y = gated_unit(h, *(w[f"{p}mlp.{name}"] for name in ("gate", "up", "down")), r)
                x = x + c["residual_mult"] * layer_norm(r(y), w[p + "norm2b"], self.eps)
            if layers is not None:
                layers.append(x)
        return soft_cap(r(layer_norm(x, w["final.norm"], self.eps)) @ w["embed"].T, c["logit_softcap"])
