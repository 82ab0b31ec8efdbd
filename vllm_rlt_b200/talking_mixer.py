"""Windowed attention with kept first tokens, bounded scores and heads that talk behind the softmax, as a mixer of the model classes.

    GEMM (q, k, v), norm_rotate (norms of q and k, rotation, keys and values to their pages), then
    attention of every head over the values of every key/value head, head_mix;   GEMM (output)

Every key and value stays in its page.
"""

from __future__ import annotations

from dataclasses import dataclass

import torch
import torch.nn.functional as F

from .attention import ScoreTerms
from .latent import rotation_frequencies
from .latent_mixer import RotationConfig
from .layers import head_mix, norm_rotate
from .model_parts import check_positive, stack_blocks, take_keys
from .sequence_cache import KVSpec


@dataclass(frozen=True)
class TalkingAttentionConfig:
    heads: int
    kv_heads: int
    dim: int
    vdim: int
    scale: float
    softcap: float
    window: int
    keep_first: int
    rotation: RotationConfig

    @classmethod
    def from_json(cls, entry: dict, what: str) -> "TalkingAttentionConfig":
        m = take_keys(entry, what, ("heads", "kv_heads", "dim", "vdim", "scale", "softcap", "mask", "rot"))
        mask = take_keys(m["mask"], what + " mask", ("size",), ("keep_first",))
        keep = mask["keep_first"] or 0
        check_positive(what, **{k: m[k] for k in ("heads", "kv_heads", "dim", "vdim")})
        check_positive(what + " mask", size=mask["size"])
        if m["heads"] % m["kv_heads"]:
            raise ValueError(f"{what}: heads must be a multiple of kv_heads")
        if not m["softcap"] > 0 or not isinstance(keep, int) or keep < 0:
            raise ValueError(f"{what}: softcap must be positive, mask.keep_first a whole number of tokens")
        return cls(m["heads"], m["kv_heads"], m["dim"], m["vdim"], float(m["scale"]), float(m["softcap"]), mask["size"], keep,
                   RotationConfig.from_json(m["rot"], what + " rot", m["dim"]))

    @property
    def cache(self) -> KVSpec:
        return KVSpec(self.kv_heads, self.dim, self.vdim)

    def parameter_shapes(self, prefix: str, width: int, rank_of=None) -> dict[str, tuple]:
        h = self.heads
        shapes = {"q": (h * self.dim, width), "k": (self.kv_heads * self.dim, width), "v": (self.kv_heads * self.vdim, width), "q.norm": (self.dim,),
                  "k.norm": (self.dim,), "temp": (h,), "talk": (h, h), "o": (width, h * self.vdim)}
        return {prefix + name: shape for name, shape in shapes.items()}


def talking_attention(kernels, q, key, value, out, group, terms: ScoreTerms, talk):
    """Attention of a group's portions over the pages with score terms, heads mixed by `talk` (float32 `[heads, heads]`) behind the softmax;
    q `[rows, heads, dim]`, out `[rows, heads, vdim]` of the group's rows."""
    rows, heads, vdim = out.shape
    spread = torch.empty(rows, heads, value.shape[2] * vdim, dtype=q.dtype, device=q.device)
    kernels.scored(q, spread, key, value, group.tables, group.lengths, group.local_cu, group.max_new, terms, all_values=True)
    return head_mix(spread, talk, out, value.shape[2])


class TalkingAttention:
    """One layer's stacked weights, and its step.  `take(name, dtype=None)` gives a parameter on the device."""

    def __init__(self, config: TalkingAttentionConfig, prefix: str, take, kernels, eps: float):
        m = self.config = config
        self.kernels, self.eps = kernels, eps
        self.w_in, self.columns, _ = stack_blocks([take(prefix + name) for name in "qkv"], 0)
        self.q_norm, self.k_norm, self.talk = (take(prefix + name, torch.float32) for name in ("q.norm", "k.norm", "talk"))
        self.w_o = take(prefix + "o")
        self.frequencies = rotation_frequencies(m.rotation.base, m.rotation.dims, self.w_in.device)
        self.terms = ScoreTerms(m.scale, window=m.window, keep_first=m.keep_first, softcap=m.softcap, head_scale=take(prefix + "temp", torch.float32))

    def __call__(self, h, key, value, batch):
        """The mixer's output for the rows of a step; their keys and values are stored."""
        m, rows = self.config, h.shape[0]
        proj = F.linear(h, self.w_in)
        q = torch.empty(rows, m.heads, m.dim, dtype=h.dtype, device=h.device)
        norm_rotate(proj, self.columns, self.q_norm, self.k_norm, self.eps, self.frequencies, q, key, value, batch, halves=m.rotation.halves)
        out = torch.empty(rows, m.heads, m.vdim, dtype=h.dtype, device=h.device)
        for group in batch.groups:
            talking_attention(self.kernels, q[group.rows], key, value, out[group.rows], group, self.terms, self.talk)
        return F.linear(out.view(rows, -1), self.w_o)
