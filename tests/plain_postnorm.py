"""Plain, slow restatement of the mechanisms of a decoder that norms its sublayers' outputs only: float64 on the CPU, one function per
mechanism, one sequence at a time, no caches.  It shares no code with the package and reads the JSON configuration itself."""

from __future__ import annotations

import torch


def rms_norm(x, eps, weight=1.0):
    return x / torch.sqrt((x * x).mean(-1, keepdim=True) + eps) * weight


def sigmoid(x):
    return 1 / (1 + torch.exp(-x))


def silu(x):
    return x * sigmoid(x)


def softplus(x):
    return torch.clamp(x, min=0) + torch.log1p(torch.exp(-x.abs()))


def unit_vector(x):
    return x / torch.sqrt((x * x).sum(-1, keepdim=True) + 1e-6)


def rotate(x, positions, base, dims, halves):
    """x [n, H, d]: the first `dims` dimensions turned in pairs, (i, i + dims / 2) with `halves`, else (2i, 2i + 1)."""
    y = x.clone()
    for i in range(dims // 2):
        a, b = (i, i + dims // 2) if halves else (2 * i, 2 * i + 1)
        angle = positions.double()[:, None] * base ** (-2.0 * i / dims)
        c, s = torch.cos(angle), torch.sin(angle)
        y[..., a], y[..., b] = x[..., a] * c - x[..., b] * s, x[..., b] * c + x[..., a] * s
    return y


def short_conv(u, weight):
    """u [n, C], weight [C, taps]: y_t = sum_j weight[:, j] u_(t - taps + 1 + j), nothing before the start."""
    n, taps = u.shape[0], weight.shape[1]
    y = torch.zeros_like(u)
    for t in range(n):
        for j in range(taps):
            if t - taps + 1 + j >= 0:
                y[t] = y[t] + weight[:, j] * u[t - taps + 1 + j]
    return y


def channel_decay(x, a_log, dt_bias):
    """x, dt_bias [.., H, d], a_log [H]: the logarithm of every key channel's decay."""
    return -torch.exp(a_log)[:, None] * softplus(x + dt_bias)


def delta_rule(q, k, v, log_decay, beta, state=None):
    """q, k, log_decay [n, H, d], v [n, H, e], beta [n, H], state [H, d, e] (None: zeros): reads [n, H, e], and the state afterwards.
    A token decays the state's rows, writes the part of its value the key does not yet give, and then reads."""
    n, heads, d = q.shape
    s = torch.zeros(heads, d, v.shape[2], dtype=torch.float64) if state is None else state.clone()
    out = torch.zeros(n, heads, v.shape[2], dtype=torch.float64)
    for t in range(n):
        s = torch.exp(log_decay[t])[:, :, None] * s
        u = beta[t][:, None] * (v[t] - torch.einsum("hde,hd->he", s, k[t]))
        s = s + k[t][:, :, None] * u[:, None, :]
        out[t] = torch.einsum("hde,hd->he", s, q[t])
    return out, s


def retention(q, k, v, decay):
    """q, k [n, H, d], v [n, H, e], decay [H]."""
    s = torch.zeros(q.shape[1], q.shape[2], v.shape[2], dtype=torch.float64)
    out = torch.zeros(v.shape, dtype=torch.float64)
    for t in range(q.shape[0]):
        s = decay[:, None, None] * s + k[t][:, :, None] * v[t][:, None, :]
        out[t] = torch.einsum("hde,hd->he", s, q[t])
    return out


def talking_attention(q, k, v, scale, temp, cap, window, keep, talk, first=0):
    """q [n, H, d] at positions first .. over k [T, G, d], v [T, G, e].  Scores are scaled, multiplied by the head's temperature and
    bounded softly; a row sees the last `window` keys and the first `keep`; head h of the result applies sum_g talk[h, g] weights_g to
    the values of its own key/value head."""
    n, heads, share = q.shape[0], q.shape[1], q.shape[1] // k.shape[1]
    group = torch.arange(heads) // share
    out = torch.zeros(n, heads, v.shape[2], dtype=torch.float64)
    for i in range(n):
        p = first + i
        j = torch.arange(p + 1)
        j = j[(p - j < window) | (j < keep)]
        scores = torch.einsum("hd,thd->ht", q[i], k[j][:, group]) * scale * temp[:, None]
        scores = cap * torch.tanh(scores / cap)
        weights = torch.exp(scores - scores.amax(1, keepdim=True))
        weights = talk @ (weights / weights.sum(1, keepdim=True))
        out[i] = torch.einsum("ht,the->he", weights, v[j][:, group])
    return out


def gated_unit(h, gate, up, down, r=lambda x: x):
    return r(silu(r(h @ gate.T)) * r(h @ up.T)) @ down.T


def experts(h, router, bias, top, expert):
    """expert(e, rows): the output of expert e.  The `top` largest logits are chosen, weighted by the softmax over them alone."""
    z = h @ router.T + bias
    out = torch.zeros_like(h)
    for i in range(h.shape[0]):
        chosen = sorted(range(z.shape[1]), key=lambda e: -z[i, e].item())[:top]
        weights = torch.exp(z[i, chosen] - z[i, chosen].max())
        for e, w in zip(chosen, weights / weights.sum()):
            out[i] += w * expert(e, h[i:i + 1])[0]
    return out


class PlainPostNorm:
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

    def channel_delta(self, p, m, h):
        w, r, n, heads, d = self.w, self.r, h.shape[0], m["heads"], m["dim"]
        q, k, v = (r(silu(short_conv(r(h @ w[p + x].T), w[p + x + ".conv"]))) for x in "qkv")
        own = torch.arange(heads) // (heads // m["kv_heads"])
        q, k = (r(unit_vector(x.reshape(n, -1, d)))[:, own] for x in (q, k))
        beta = sigmoid(h @ w[p + "b"].T)
        low = r(h @ w[p + "a1"].T)
        log_decay = channel_decay((low @ w[p + "a2"].T).reshape(n, heads, d), w[p + "A_log"], w[p + "dt_bias"].reshape(heads, d))
        o, _ = delta_rule(q * d ** -0.5, k, v.reshape(n, heads, -1), log_decay, beta)
        gate = r(r(h @ w[p + "g1"].T) @ w[p + "g2"].T)
        o = rms_norm(r(o), self.eps, w[p + "norm"]).reshape(n, -1) * sigmoid(gate)
        return r(o) @ w[p + "o"].T

    def attention(self, p, m, h):
        w, r, n = self.w, self.r, h.shape[0]
        q, k, v = (r(h @ w[p + x].T).reshape(n, -1, m[size]) for x, size in (("q", "dim"), ("k", "dim"), ("v", "vdim")))
        at = torch.arange(n)
        q, k = (r(rotate(rms_norm(x, self.eps, w[f"{p}{name}.norm"]), at, m["rot"]["base"], m["rot"]["dims"], False))
                for name, x in (("q", q), ("k", k)))
        out = talking_attention(q, k, v, m["scale"], w[p + "temp"], m["softcap"], m["mask"]["size"], m["mask"]["keep_first"], w[p + "talk"])
        return r(out.reshape(n, -1)) @ w[p + "o"].T

    def retention(self, p, m, h):
        w, r, n, d = self.w, self.r, h.shape[0], m["dim"]
        q, k, v = (r(h @ w[p + x].T).reshape(n, m["heads"], -1) for x in "qkv")
        q, k = (rotate(x, torch.arange(n), m["rot"]["base"], m["rot"]["dims"], True) for x in (q, k))
        o = retention(r(q), r(k * d ** -0.5), v, torch.tensor(m["decay"], dtype=torch.float64))
        o = rms_norm(r(o), self.eps).reshape(n, -1) * silu(r(h @ w[p + "g"].T))
        return r(o) @ w[p + "o"].T

    def feed_forward(self, p, m, h):
        w, r = self.w, self.r
        unit = lambda name, rows: gated_unit(rows, w[name + ".gate"], w[name + ".up"], w[name + ".down"], r)
        if m["kind"] == "dense":
            return unit(p[:-1], h)
        y = experts(h, w[p + "router"], w[p + "router.b"], m["router"]["top"], lambda e, rows: r(unit(f"{p}e{e}", rows)))
        return y + r(unit(p + "shared", h)) if m.get("shared") else y

    def __call__(self, tokens, layers=None):
        """Logits [tokens, vocab]; `layers`, a list, receives the residual after every layer."""
        w, c, r = self.w, self.config, self.r
        x = w["embed"][torch.tensor(tokens)]
        for i, entry in enumerate(c["layers"]):
            own = i
            while c["layers"][own].get("weights_of") is not None:
                own = c["layers"][own]["weights_of"]
            p = f"l{own}."
            y = getattr(self, entry["type"])(p + "mix.", entry["mixer"], r(x))
            x = x + rms_norm(r(y), self.eps, w[p + "norm1"])
            if entry["mlp"]:
                x = x + rms_norm(r(self.feed_forward(p + "mlp.", entry["mlp"], r(x))), self.eps, w[p + "norm2"])
            if layers is not None:
                layers.append(x)
        return r(rms_norm(x, self.eps, w["final.norm"])) @ w["head"].T
