"""Retention as a mixer of the model classes: linear attention with a constant decay per head over rotated queries and keys.

    GEMM (q, k, v, gate), rotate_heads (q and k, in place), decay_scan, gated_norm (a norm per head, the gate behind it), GEMM (output)

A sequence keeps one fp32 matrix [dim, vdim] per head.
"""

from __future__ import annotations

from dataclasses import dataclass

import torch
import torch.nn.functional as F

from .latent import rotate_heads, rotation_frequencies
from .latent_mixer import RotationConfig
from .model_parts import check_positive, stack_blocks, take_keys
from .recurrent import decay_scan, decay_table, gated_norm
from .sequence_cache import StateSpec


@dataclass(frozen=True)
class RetentionConfig:
    heads: int
    dim: int
    vdim: int
    decay: tuple
    rotation: RotationConfig

    @classmethod
    def from_json(cls, entry: dict, what: str) -> "RetentionConfig":
        m = take_keys(entry, what, ("heads", "dim", "vdim", "decay", "rot"))
        check_positive(what, heads=m["heads"], dim=m["dim"], vdim=m["vdim"])
        decay = tuple(float(d) for d in m["decay"])
        if len(decay) != m["heads"] or not all(0.0 <= d <= 1.0 for d in decay):
            raise ValueError(f"{what}: decay needs one number between 0 and 1 per head")
        return cls(m["heads"], m["dim"], m["vdim"], decay, RotationConfig.from_json(m["rot"], what + " rot", m["dim"], halves=True))

    @property
    def states(self) -> dict[str, StateSpec]:
        return {"state": StateSpec((self.heads, self.dim, self.vdim), torch.float32)}

    def parameter_shapes(self, prefix: str, width: int, rank_of=None) -> dict[str, tuple]:
        keys, inner = self.heads * self.dim, self.heads * self.vdim
        return {prefix + "q": (keys, width), prefix + "k": (keys, width), prefix + "v": (inner, width), prefix + "g": (inner, width),
                prefix + "o": (width, inner)}


class Retention:
    """One layer's stacked weights, and its step.  `take(name, dtype=None)` gives a parameter on the device."""

    def __init__(self, config: RetentionConfig, prefix: str, take, eps: float):
        m = self.config = config
        self.eps = eps
        # q and k heads side by side, so that one launch turns both
        blocks = [torch.cat([take(prefix + "q"), take(prefix + "k")]), take(prefix + "v"), take(prefix + "g")]
        self.w_in, (_, self.v_col, self.g_col), _ = stack_blocks(blocks, 0)
        self.w_o = take(prefix + "o")
        self.decay = decay_table(m.decay, self.w_in.device)
        self.frequencies = rotation_frequencies(m.rotation.base, m.rotation.dims, self.w_in.device)

    def __call__(self, h, state, batch):
        """The mixer's output for the rows of a step; `state(name)` gives the sequences' slots, which are updated."""
        m, rows = self.config, h.shape[0]
        keys, inner = m.heads * m.dim, m.heads * m.vdim
        proj = F.linear(h, self.w_in)
        qk = proj[:, :2 * keys].unflatten(1, (2 * m.heads, m.dim))
        rotate_heads(qk, qk, self.frequencies, batch.positions, halves=m.rotation.halves, scale=m.dim ** -0.5, scaled_from=m.heads)
        y = torch.empty(rows, inner, dtype=h.dtype, device=h.device)
        for group in batch.groups:
            decay_scan(proj[:, :keys], proj[:, keys:2 * keys], proj[:, self.v_col:self.v_col + inner], self.decay, state("state"), y, group)
        gate = proj[:, self.g_col:self.g_col + inner]
        return F.linear(gated_norm(y, gate, None, torch.empty_like(y), m.heads, self.eps, gate_behind="silu"), self.w_o)
