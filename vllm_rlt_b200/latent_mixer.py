"""Latent attention as a mixer of the model classes: queries, keys and values through latents, a key part shared by all heads.

    GEMM (both down projections, and the gate's), latent_write (query latent normed, cache row written), GEMM (queries), then
    long portions:  rotate_heads, latent_gather, GEMM (keys and values), attention with the gate, and
    short ones:     per-head GEMM (queries into the latent's space), rotate_heads, attention over the cache rows themselves,
                    per-head GEMM (values out of it), head_gate;   GEMM (output)

The cache row of a token is [latent | rotated key part], shared by all heads.  Parts that a model may have or not: a sliding window, a sink
per head, an output gate (one value per element or per head, from the mixer's input), and how the rotated part is turned.
"""

from __future__ import annotations

from dataclasses import dataclass

import torch
import torch.nn.functional as F

from .attention import ScoreTerms
from .latent import (YarnScaling, latent_gather, latent_prompt_attention, latent_prompt_supported, latent_write, rotate_heads,
                     rotation_frequencies)
from .layers import head_gate
from .model_parts import check_positive, stack_blocks, take_keys
from .sequence_cache import KVSpec

SHORT_PORTION = 16      # groups of portions up to this long attend over the cache rows, longer ones over expanded keys and values


@dataclass(frozen=True)
class RotationConfig:
    base: float
    dims: int                         # how many of the rotated part's dimensions are turned
    halves: bool = False              # pairs (i, i + dims / 2) and not (2i, 2i + 1)
    scaling: YarnScaling | None = None

    @classmethod
    def from_json(cls, entry: dict, what: str, rot_dim: int, *, halves: bool = False, scaled: bool = False) -> "RotationConfig":
        """`scaled`: the entry may have a `scaling`."""
        rot = take_keys(entry, what, ("base", "dims"), ("scaling",) if scaled else ())
        check_positive(what, dims=rot["dims"])
        if rot["dims"] % 2 or rot["dims"] > rot_dim:
            raise ValueError(f"{what}: rot.dims must be even and at most rot_dim")
        scaling = None
        if rot.get("scaling"):
            s = take_keys(rot["scaling"], what + " scaling", ("factor", "original", "fast", "slow"))
            if not all(s[k] > 0 for k in s) or rot["base"] <= 1:
                raise ValueError(f"{what}: scaling needs positive numbers and a base above 1")
            scaling = YarnScaling(*(float(s[k]) for k in ("factor", "original", "fast", "slow")))
        return cls(float(rot["base"]), rot["dims"], halves, scaling)


@dataclass(frozen=True)
class LatentAttentionConfig:
    heads: int
    dim: int              # unrotated query / key dimensions of a head
    rot_dim: int          # rotated ones
    vdim: int
    q_rank: int
    kv_rank: int
    scale: float
    rotation: RotationConfig
    window: int = 0       # 0: every earlier key
    sink: bool = False    # a learned term of every head's denominator
    gate: str | None = None   # "element" or "head": what one value of the output gate multiplies

    @classmethod
    def from_json(cls, entry: dict, what: str, *, windowed: bool = False, halves: bool = False, scaled: bool = False, sink: bool = False,
                  gate: str | None = None) -> "LatentAttentionConfig":
        """`windowed`, `scaled`: the entry may have a `mask` with a window's size, a `scaling` of its rotation."""
        m = take_keys(entry, what, ("heads", "dim", "rot_dim", "vdim", "q_rank", "kv_rank", "scale", "rot"), ("mask",) if windowed else ())
        check_positive(what, **{k: m[k] for k in ("heads", "dim", "rot_dim", "vdim", "q_rank", "kv_rank")})
        rotation = RotationConfig.from_json(m["rot"], what + " rot", m["rot_dim"], halves=halves, scaled=scaled)
        window = 0
        if m.get("mask"):
            window = take_keys(m["mask"], what + " mask", ("size",))["size"]
            check_positive(what + " mask", size=window)
        return cls(m["heads"], m["dim"], m["rot_dim"], m["vdim"], m["q_rank"], m["kv_rank"], float(m["scale"]), rotation, window, sink, gate)

    @property
    def row(self) -> int:             # elements of a cache row
        return self.kv_rank + self.rot_dim

    @property
    def gate_width(self) -> int:
        return {None: 0, "head": self.heads, "element": self.heads * self.vdim}[self.gate]

    @property
    def cache(self) -> KVSpec:
        return KVSpec(1, self.row, 0)

    def parameter_shapes(self, prefix: str, width: int) -> dict[str, tuple]:
        shapes = {"dq": (self.q_rank, width), "dq.norm": (self.q_rank,), "uq": (self.heads * (self.dim + self.rot_dim), self.q_rank),
                  "dkv": (self.row, width), "dkv.norm": (self.kv_rank,), "uk": (self.heads * self.dim, self.kv_rank),
                  "uv": (self.heads * self.vdim, self.kv_rank), "o": (width, self.heads * self.vdim)}
        if self.sink:
            shapes["sink"] = (self.heads,)
        if self.gate:
            shapes["g"] = (self.gate_width, width)
        return {prefix + name: shape for name, shape in shapes.items()}


class LatentAttention:
    """One layer's stacked weights, and its step.  `take(name, dtype=None)` gives a parameter on the device."""

    def __init__(self, config: LatentAttentionConfig, prefix: str, take, kernels, eps: float, device):
        m = self.config = config
        self.kernels, self.eps = kernels, eps
        blocks = [take(prefix + name) for name in ("dq", "dkv") + (("g",) if m.gate else ())]
        self.w_down, offsets, _ = stack_blocks(blocks, 0)
        self.q_col, self.kv_col = offsets[:2]
        self.g_col = offsets[2] if m.gate else 0
        self.q_norm, self.kv_norm = take(prefix + "dq.norm", torch.float32), take(prefix + "dkv.norm", torch.float32)
        self.w_q = take(prefix + "uq")
        keys = m.heads * m.dim
        self.w_kv = torch.cat([take(prefix + "uk"), take(prefix + "uv")])       # all heads' keys, then all values
        self.w_uk, self.w_uv = self.w_kv[:keys].view(m.heads, m.dim, m.kv_rank), self.w_kv[keys:].view(m.heads, m.vdim, m.kv_rank)
        self.w_o = take(prefix + "o")
        self.sink = take(prefix + "sink", torch.float32) if m.sink else None
        self.terms = ScoreTerms(m.scale, window=m.window, sink=self.sink)
        r = m.rotation
        self.frequencies = rotation_frequencies(r.base, r.dims, device, r.scaling)
        self.turn = dict(halves=r.halves, amplitude=r.scaling.amplitude if r.scaling else 1.0)

    def __call__(self, h, pages, batch):
        """The mixer's output for the rows of a step; their cache rows are written to `pages`."""
        m, rows = self.config, h.shape[0]
        down = F.linear(h, self.w_down)
        latent = latent_write(down, self.q_col, self.kv_col, self.q_norm, self.kv_norm, self.eps, self.frequencies, pages, batch, **self.turn)
        q = F.linear(latent, self.w_q).view(rows, m.heads, m.dim + m.rot_dim)
        gate = down[:, self.g_col:self.g_col + m.gate_width] if m.gate else None
        out = torch.empty(rows, m.heads, m.vdim, dtype=h.dtype, device=h.device)
        for group in batch.groups:
            expand = group.max_new > SHORT_PORTION and group.portions is not None and m.kv_rank % 8 == 0 and \
                latent_prompt_supported(m.dim, m.rot_dim, m.vdim, h.dtype)
            attend = self._attend_expanded if expand else self._attend_latents
            part = group.rows
            attend(q[part], out[part], None if gate is None else gate[part], pages, batch.positions[part], group)
        return F.linear(out.view(rows, -1), self.w_o)

    def _attend_expanded(self, q, out, gate, pages, positions, group):
        """Over keys and values expanded from the latents of every position the portions see."""
        m = self.config
        ranges = group.key_ranges(m.window)
        rows = latent_gather(pages, group.tables, ranges)
        rotate_heads(q[:, :, m.dim:], q[:, :, m.dim:], self.frequencies, positions, **self.turn)
        latent_prompt_attention(q, F.linear(rows[:, :m.kv_rank], self.w_kv), rows[:, m.kv_rank:], out, m.dim, ranges, m.scale, m.window,
                                sink=self.sink, gate=gate)

    def _attend_latents(self, q, out, gate, pages, positions, group):
        """Over the cache rows themselves: a head's query is taken into the latent's space (q . W_uk c = W_uk^T q . c), so all
        heads score the one row of a key, and the weighted sum of latents is taken out of it by W_uv."""
        m, rows = self.config, q.shape[0]
        operand = torch.empty(rows, m.heads, m.row, dtype=q.dtype, device=q.device)
        torch.bmm(q[:, :, :m.dim].transpose(0, 1), self.w_uk, out=operand[:, :, :m.kv_rank].transpose(0, 1))
        rotate_heads(q[:, :, m.dim:], operand[:, :, m.kv_rank:], self.frequencies, positions, **self.turn)
        latents = torch.empty(rows, m.heads, m.kv_rank, dtype=q.dtype, device=q.device)
        self.kernels.scored(operand, latents, pages, pages[..., :m.kv_rank], group.tables, group.lengths, group.local_cu, group.max_new,
                            self.terms)
        torch.bmm(latents.transpose(0, 1), self.w_uv.transpose(1, 2), out=out.transpose(0, 1))
        if gate is not None:
            head_gate(out, gate)
