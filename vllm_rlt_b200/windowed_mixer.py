"""Windowed attention behind a short convolution as a mixer of the model classes: no rotation, queries and keys of unit root mean square,
an output gate.

    GEMM (q, k, v with biases, gate), conv_heads (convolution, unit norm, keys and values to their pages), then
    long portions:  gathered keys and values of the window, attention with the gate, and
    short ones:     attention over the pages, head_gate;   GEMM (output)

The last taps - 1 projected values of q, k and v are a sequence's state; every key and value stays in its page.
"""

from __future__ import annotations

from dataclasses import dataclass

import torch
import torch.nn.functional as F

from .attention import ScoreTerms
from .latent import latent_gather, latent_prompt_supported, packed_attention
from .latent_mixer import SHORT_PORTION
from .layers import head_gate
from .model_parts import check_positive, stack_blocks, take_keys
from .recurrent import conv_heads
from .sequence_cache import KVSpec, StateSpec


@dataclass(frozen=True)
class WindowedAttentionConfig:
    heads: int
    kv_heads: int
    dim: int
    vdim: int
    taps: int
    window: int
    scale: float

    @classmethod
    def from_json(cls, entry: dict, what: str) -> "WindowedAttentionConfig":
        m = take_keys(entry, what, ("heads", "kv_heads", "dim", "vdim", "conv", "mask", "scale"))
        window = take_keys(m["mask"], what + " mask", ("size",))["size"]
        check_positive(what, **{k: m[k] for k in ("heads", "kv_heads", "dim", "vdim", "conv")})
        check_positive(what + " mask", size=window)
        if m["heads"] % m["kv_heads"]:
            raise ValueError(f"{what}: heads must be a multiple of kv_heads")
        return cls(m["heads"], m["kv_heads"], m["dim"], m["vdim"], m["conv"], window, float(m["scale"]))

    @property
    def projections(self) -> dict[str, int]:
        """The convolved projections and their channels, in the order of the state."""
        return {"q": self.heads * self.dim, "k": self.kv_heads * self.dim, "v": self.kv_heads * self.vdim}

    @property
    def cache(self) -> KVSpec:
        return KVSpec(self.kv_heads, self.dim, self.vdim)

    @property
    def state(self) -> StateSpec:
        return StateSpec((self.taps - 1, sum(self.projections.values())))

    def parameter_shapes(self, prefix: str, width: int) -> dict[str, tuple]:
        shapes = {}
        for name, channels in self.projections.items():
            shapes.update({name: (channels, width), name + ".b": (channels,), name + ".conv": (channels, self.taps)})
        shapes["g"], shapes["o"] = (self.heads * self.vdim, width), (width, self.heads * self.vdim)
        return {prefix + name: shape for name, shape in shapes.items()}


class WindowedAttention:
    """One layer's stacked weights, and its step.  `take(name, dtype=None)` gives a parameter on the device."""

    def __init__(self, config: WindowedAttentionConfig, prefix: str, take, kernels, eps: float):
        m = self.config = config
        self.kernels, self.eps = kernels, eps
        names = list(m.projections)
        blocks = [take(prefix + name) for name in (*names, "g")]
        self.w_in, offsets, total = stack_blocks(blocks, 0)
        self.columns, self.g_col = tuple(offsets[:3]), offsets[3]
        self.bias = torch.zeros(total, dtype=self.w_in.dtype, device=self.w_in.device)
        for name, at in zip(names, self.columns):
            self.bias[at:at + m.projections[name]] = take(f"{prefix}{name}.b")
        self.conv = torch.cat([take(f"{prefix}{name}.conv", torch.float32) for name in names]).t().contiguous()
        self.w_o = take(prefix + "o")
        self.terms = ScoreTerms(m.scale, window=m.window)

    def __call__(self, h, key, value, state, batch):
        """The mixer's output for the rows of a step; keys, values and the sequences' last inputs are stored."""
        m, rows = self.config, h.shape[0]
        proj = F.linear(h, self.w_in, self.bias)
        gate = proj[:, self.g_col:self.g_col + m.heads * m.vdim]
        q = torch.empty(rows, m.heads, m.dim, dtype=h.dtype, device=h.device)
        out = torch.empty(rows, m.heads, m.vdim, dtype=h.dtype, device=h.device)
        for group in batch.groups:
            conv_heads(proj, self.columns, self.conv, self.eps, state, q, key, value, group)
            part = group.rows
            if group.max_new > SHORT_PORTION and group.portions is not None and latent_prompt_supported(m.dim, 0, m.vdim, h.dtype):
                ranges = group.key_ranges(m.window)
                keys, values = (latent_gather(cache.flatten(2).unsqueeze(2), group.tables, ranges).unflatten(1, cache.shape[2:])
                                for cache in (key, value))
                packed_attention(q[part], keys, values, out[part], ranges, m.scale, m.window, gate=gate[part])
            else:
                self.kernels.scored(q[part], out[part], key, value, group.tables, group.lengths, group.local_cu, group.max_new, self.terms)
                head_gate(out[part], gate[part])
        return F.linear(out.view(rows, -1), self.w_o)
