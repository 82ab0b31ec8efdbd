"""Plain, slow restatement of the mechanisms of a decoder over hyper-connected streams: float64 on the CPU, one function per
mechanism, one sequence at a time, no caches.  It shares no code with the package and reads the JSON configuration itself."""

from __future__ import annotations

import math

import torch


def rms_norm(x, weight, eps):
    return x / torch.sqrt((x * x).mean(-1, keepdim=True) + eps) * weight


def sigmoid(x):
    return 1 / (1 + torch.exp(-x))


def silu(x):
    return x * sigmoid(x)


def bigram_rows(tokens, buckets, mul_prev, mul_cur):
    """Table row of every token of a sequence: a hash of the token and the one before it, the last row for the first token."""
    rows = [buckets]
    for before, token in zip(tokens, tokens[1:]):
        rows.append((before * mul_prev + token * mul_cur) % buckets)
    return rows


def rotate(x, positions, base, dims):
    """x [n, ..., d]: pairs (2i, 2i + 1) of the first `dims` dimensions turned by position * base^(-2i / dims)."""
    y = x.clone()
    for i in range(dims // 2):
        angle = positions.double() * base ** (-2.0 * i / dims)
        c, s = (f(angle).reshape(-1, *[1] * (x.dim() - 2)) for f in (torch.cos, torch.sin))
        u, v = x[..., 2 * i], x[..., 2 * i + 1]
        y[..., 2 * i], y[..., 2 * i + 1] = u * c - v * s, v * c + u * s
    return y


def windowed_attention(q, k, v, scale, window, first=0):
    """q [n, H, d] at positions first .. over k [T, H, d], v [T, H, e]; a row sees itself and the window - 1 keys before it
    (window 0: all of them).  Returns [n, H, e]."""
    out = torch.zeros(q.shape[0], q.shape[1], v.shape[2], dtype=torch.float64)
    for i in range(q.shape[0]):
        p = first + i
        lo = max(p - window + 1, 0) if window else 0
        scores = torch.einsum("hd,thd->ht", q[i], k[lo:p + 1]) * scale
        w = torch.exp(scores - scores.max(1, keepdim=True).values)
        out[i] = torch.einsum("ht,the->he", w / w.sum(1, keepdim=True), v[lo:p + 1])
    return out


def decayed_attention(q, k, v, decay, state=None):
    """q, k [n, H, d], v [n, H, e]: S_t = decay S_(t-1) + k_t v_t^T, o_t = S_t^T q_t.  Returns o [n, H, e] and the last S [H, d, e]."""
    n, heads, d = q.shape
    s = torch.zeros(heads, d, v.shape[2], dtype=torch.float64) if state is None else state.clone()
    out = torch.zeros_like(v)
    for t in range(n):
        s = decay[:, None, None] * s + k[t, :, :, None] * v[t, :, None, :]
        out[t] = torch.einsum("hde,hd->he", s, q[t])
    return out, s


def gated_output(y, gate, weight, eps):
    return rms_norm(y, weight, eps) * sigmoid(gate)


def clamped_unit(gate, up, limit):
    g, u = torch.clamp(gate, max=limit), torch.clamp(up, -limit, limit)
    return g * sigmoid(1.702 * g) * (u + 1)


def route(logits, correction, top):
    """Chosen experts [n, top] (by score + correction) and their weights (by score alone)."""
    scores = torch.softmax(logits, -1)
    chosen = torch.sort(scores + correction, dim=-1, descending=True, stable=True).indices[:, :top]
    picked = scores.gather(1, chosen)
    return chosen, picked / (picked.sum(1, keepdim=True) + 1e-20)


def expert(h, up, down, r=lambda x: x):
    return r(r(torch.relu(r(h @ up.T)) ** 2) @ down.T)


def read_streams(streams, coefficients):
    return sum(c * x for c, x in zip(coefficients, streams))


def write_streams(streams, y, out, mix):
    return [sum(mix[s, t] * streams[s] for s in range(len(streams))) + out[t] * y for t in range(len(streams))]


class PlainStream:
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

    def embed(self, tokens):
        x, b = self.w["embed"][torch.tensor(tokens)], (self.config.get("embedding") or {}).get("bigram")
        if b:
            x = x + self.w["bigram"][torch.tensor(bigram_rows(tokens, b["buckets"], b["mul_prev"], b["mul_cur"]))]
        return rms_norm(x, self.w["embed.norm"], self.eps)

    def latent(self, p, m, h):
        w, r, n, heads = self.w, self.r, h.shape[0], m["heads"]
        positions, d, rot = torch.arange(n), m["dim"], m["rot"]
        turn = lambda x: torch.cat([x[..., :d], r(rotate(x[..., d:], positions, rot["base"], rot["dims"]))], -1)
        c_q = r(rms_norm(r(h @ w[p + "dq"].T), w[p + "dq.norm"], self.eps))
        q = turn(r(c_q @ w[p + "uq"].T).reshape(n, heads, -1))
        down = r(h @ w[p + "dkv"].T)
        c = r(rms_norm(down[:, :m["kv_rank"]], w[p + "dkv.norm"], self.eps))
        shared = r(rotate(down[:, m["kv_rank"]:], positions, rot["base"], rot["dims"]))
        k = torch.cat([r(c @ w[p + "uk"].T).reshape(n, heads, d), shared[:, None].expand(n, heads, -1)], -1)
        v = r(c @ w[p + "uv"].T).reshape(n, heads, m["vdim"])
        out = windowed_attention(q, k, v, m["scale"], m["mask"]["size"] if m.get("mask") else 0)
        return r(out.reshape(n, -1)) @ w[p + "o"].T

    def lightning(self, p, m, h):
        w, r, n, heads = self.w, self.r, h.shape[0], m["heads"]
        q, k, v = (r(silu(r(h @ w[p + name].T))).reshape(n, heads, -1) for name in "qkv")
        y, _ = decayed_attention(q, k, v, torch.tensor(m["decay"], dtype=torch.float64))
        return r(gated_output(r(y.reshape(n, -1)), r(h @ w[p + "g"].T), w[p + "norm"], self.eps)) @ w[p + "o"].T

    def feed_forward(self, p, f, h):
        w, r = self.w, self.r
        if f["kind"] == "dense":
            return r(clamped_unit(r(h @ w[p + "gate"].T), r(h @ w[p + "up"].T), f["limit"])) @ w[p + "down"].T
        chosen, weights = route(h @ w[p + "router"].T, w[p + "correction"], f["router"]["top"])
        y = torch.zeros_like(h)
        for e in range(f["router"]["experts"]):
            share = (weights * (chosen == e)).sum(1, keepdim=True)
            y = y + share * expert(h, w[f"{p}e{e}.up"], w[f"{p}e{e}.down"], r)
        return y

    def __call__(self, tokens, layers=None):
        """Logits [tokens, vocab]; `layers`, a list, receives the sum of the streams after every layer run."""
        w, c, r = self.w, self.config, self.r
        streams = [self.embed(tokens)] * c["streams"]
        order = list(range(len(c["layers"])))
        if c.get("loop"):
            start, stop, times = (c["loop"][k] for k in ("start", "stop", "times"))
            order = order[:start] + order[start:stop] * times + order[stop:]
        for i in order:
            entry = c["layers"][i]
            for q in (1, 2):
                if q == 2 and not entry["mlp"]:
                    continue
                hc = f"l{i}.hc{q}."
                h = r(rms_norm(read_streams(streams, w[hc + "in"]), w[f"l{i}.norm{q}"], self.eps))
                if q == 2:
                    y = self.feed_forward(f"l{i}.mlp.", entry["mlp"], h)
                else:
                    y = (self.latent if entry["type"] == "latent_attention" else self.lightning)(f"l{i}.mix.", entry["mixer"], h)
                streams = write_streams(streams, r(y), w[hc + "out"], w[hc + "mix"])
            if layers is not None:
                layers.append(sum(streams))
        return r(rms_norm(sum(streams), w["final.norm"], self.eps)) @ w["head"].T
