"""The gated delta rule with a decay per key channel as a mixer of the model classes.

    GEMM (q, k, v, write strength, both low-rank gates' first halves), causal_conv (q, k, v, silu), GEMM (decays), GEMM (output gate),
    delta_scan (unit norms, decays, strengths and the recurrence), gated_norm (a norm per head, the gate behind it), GEMM (output)

A sequence keeps the last taps - 1 projected values of q, k and v, and one fp32 matrix [dim, vdim] per head.
"""

from __future__ import annotations

from dataclasses import dataclass

import torch
import torch.nn.functional as F

from .model_parts import check_positive, stack_blocks, take_keys
from .recurrent import causal_conv, delta_scan, gated_norm
from .sequence_cache import StateSpec


@dataclass(frozen=True)
class ChannelDeltaConfig:
    heads: int
    kv_heads: int         # heads of q and k
    dim: int
    vdim: int
    taps: int

    @classmethod
    def from_json(cls, entry: dict, what: str) -> "ChannelDeltaConfig":
        m = take_keys(entry, what, ("heads", "kv_heads", "dim", "vdim", "conv"))
        check_positive(what, **m)
        if m["heads"] % m["kv_heads"]:
            raise ValueError(f"{what}: heads must be a multiple of kv_heads")
        return cls(m["heads"], m["kv_heads"], m["dim"], m["vdim"], m["conv"])

    @property
    def projections(self) -> dict[str, int]:
        """The convolved projections and their channels."""
        return {"q": self.kv_heads * self.dim, "k": self.kv_heads * self.dim, "v": self.heads * self.vdim}

    @property
    def channels(self) -> int:        # of the convolution's state: every projection starts at a multiple of 8
        return sum(-(-n // 8) * 8 for n in self.projections.values())

    @property
    def states(self) -> dict[str, StateSpec]:
        return {"conv": StateSpec((self.taps - 1, self.channels)), "state": StateSpec((self.heads, self.dim, self.vdim), torch.float32)}

    def parameter_shapes(self, prefix: str, width: int, rank_of) -> dict[str, tuple]:
        """rank_of(name): the rank of a low-rank projection, which only its first tensor tells."""
        shapes = {}
        for name, channels in self.projections.items():
            shapes.update({name: (channels, width), name + ".conv": (channels, self.taps)})
        keys, values = self.heads * self.dim, self.heads * self.vdim
        shapes.update({"b": (self.heads, width), "A_log": (self.heads,), "dt_bias": (keys,), "norm": (self.vdim,), "o": (width, values)})
        for first, second, n in (("a1", "a2", keys), ("g1", "g2", values)):
            rank = rank_of(prefix + first)
            shapes.update({first: (rank, width), second: (n, rank)})
        return {prefix + name: shape for name, shape in shapes.items()}


class ChannelDelta:
    """One layer's stacked weights, and its step.  `take(name, dtype=None)` gives a parameter on the device."""

    def __init__(self, config: ChannelDeltaConfig, prefix: str, take, eps: float):
        m = self.config = config
        self.eps = eps
        names = list(m.projections)
        blocks = [take(prefix + name) for name in (*names, "b", "a1", "g1")]
        self.ranks = blocks[4].shape[0], blocks[5].shape[0]
        self.w_in, offsets, _ = stack_blocks(blocks, 0)
        self.columns, (self.b_col, self.a_col, self.g_col) = offsets[:3], offsets[3:]
        weight = torch.zeros(m.channels, m.taps, dtype=torch.float32, device=self.w_in.device)
        for name, at in zip(names, self.columns):
            weight[at:at + m.projections[name]] = take(f"{prefix}{name}.conv", torch.float32)
        self.conv, self.no_bias = weight, torch.zeros(m.channels, dtype=torch.float32, device=weight.device)
        self.w_decay, self.w_gate, self.w_o = take(prefix + "a2"), take(prefix + "g2"), take(prefix + "o")
        self.dt_bias, self.a_log = take(prefix + "dt_bias", torch.float32), take(prefix + "A_log", torch.float32)
        self.norm = take(prefix + "norm", torch.float32).repeat(m.heads)

    def __call__(self, h, state, batch):
        """The mixer's output for the rows of a step; `state(name)` gives the sequences' slots, which are updated."""
        m, rows = self.config, h.shape[0]
        proj = F.linear(h, self.w_in)
        qkv = torch.empty(rows, m.channels, dtype=h.dtype, device=h.device)
        decay = F.linear(proj[:, self.a_col:self.a_col + self.ranks[0]], self.w_decay)
        gate = F.linear(proj[:, self.g_col:self.g_col + self.ranks[1]], self.w_gate)
        beta = proj[:, self.b_col:self.b_col + m.heads]
        q, k, v = (qkv[:, at:at + n] for at, n in zip(self.columns, m.projections.values()))
        y = torch.empty(rows, m.heads * m.vdim, dtype=h.dtype, device=h.device)
        for group in batch.groups:
            causal_conv(proj[:, :m.channels], self.conv, self.no_bias, state("conv"), qkv, group)
            delta_scan(q, k, v, decay, beta, self.dt_bias, self.a_log, state("state"), y, group)
        return F.linear(gated_norm(y, gate, self.norm, torch.empty_like(y), m.heads, self.eps, gate_behind=True), self.w_o)
