"""Windowed attention with kept first tokens, bounded scores and heads that talk behind the softmax, as a mixer of the model classes.

    GEMM (q, k, v), norm_rotate (norms of q and k, rotation, keys and values to their pages), then
    long portions:  gathered keys and values of the window and the kept tokens, attention of every head over the values of every
                    key/value head, head_mix, and
    short ones:     the same over the pages, heads mixed where the splits of a context are merged;   GEMM (output)

Every key and value stays in its page.  32-bit models and sizes outside the kernels' alignment take the general attention and head_mix.
"""

from __future__ import annotations

from dataclasses import dataclass

import torch
import torch.nn.functional as F

from . import _capi
from .attention import ScoreTerms, check_sink
from .latent import latent_gather, rotation_frequencies
from .latent_mixer import SHORT_PORTION, RotationConfig
from .layers import head_mix, norm_rotate
from .model_parts import check_positive, stack_blocks, take_keys
from .sequence_cache import KVSpec


PROMPT_ROWS = 128        # query rows of a tile of the prompt kernel


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
    kv_heads, dim = key.shape[2], q.shape[2]
    sizes, rest = (heads, kv_heads, dim, vdim), (float(terms.softcap), _capi.DTYPE_CODES[q.dtype])
    short = group.max_new <= SHORT_PORTION or group.portions is None
    if short and _capi.load().rlt_talking_attention_supported(*sizes, key.shape[1], *rest):
        return talking_decode(q, key, value, out, group, terms, talk)
    spread = torch.empty(rows, heads, kv_heads * vdim, dtype=q.dtype, device=q.device)
    if not short and _capi.load().rlt_talking_prompt_supported(*sizes, *rest):
        ranges = group.key_ranges(terms.window, terms.keep_first, PROMPT_ROWS)
        keys, values = (latent_gather(cache.flatten(2).unsqueeze(2), group.tables, ranges) for cache in (key, value))
        talking_prompt(q, keys, values, spread, ranges, terms, kv_heads)
    else:
        kernels.scored(q, spread, key, value, group.tables, group.lengths, group.local_cu, group.max_new, terms, all_values=True)
    return head_mix(spread, talk, out, kv_heads)


def _check(q, out, terms: ScoreTerms, talk=None) -> None:
    heads = q.shape[1]
    check_sink(terms.head_scale, heads, "head_scale")
    if terms.sink is not None or terms.distance_bias or terms.temp_coef:
        raise ValueError("talking attention takes a window, kept first tokens, a soft cap and a scale per head")
    if talk is not None and (talk.dtype != torch.float32 or talk.shape != (heads, heads) or not talk.is_contiguous()):
        raise ValueError("talk must be contiguous float32 [heads, heads]")
    if any(t.stride(2) != 1 or t.stride(1) != t.shape[2] for t in (q, out)) or out.dtype != q.dtype:
        raise ValueError("q and out must have heads side by side and one dtype")


def talking_decode(q, key, value, out, group, terms: ScoreTerms, talk):
    """`rlt_talking_attention`: short portions over the pages."""
    _capi.require_cuda(q, key, value, out, talk, terms.head_scale, group.tables, group.lengths, group.local_cu)
    _check(q, out, terms, talk)
    rows, heads, dim = q.shape
    pages, block, kv_heads, vdim = value.shape
    if key.shape != (pages, block, kv_heads, dim) or any(c.stride(3) != 1 or c.stride(2) != c.shape[3] or c.dtype != q.dtype for c in (key, value)):
        raise ValueError("caches must be [pages, block, kv_heads, dim] of q's dtype with a contiguous tail")
    if rows == 0:
        return out
    lib, width = _capi.load(), group.tables.shape[1]
    seen = min(width * block, terms.window + terms.keep_first + group.max_new) if terms.window else width * block
    sizes = rows, group.sequences, group.max_new, heads, kv_heads, dim, vdim, block, seen
    with torch.cuda.device(q.device):
        nbytes = lib.rlt_talking_attention_workspace_bytes(*sizes)
        workspace = torch.empty(nbytes, dtype=torch.uint8, device=q.device)
        code = lib.rlt_talking_attention(
            _capi.ptr(q), q.stride(0), _capi.ptr(out), out.stride(0), _capi.ptr(key), key.stride(0), key.stride(1), _capi.ptr(value), value.stride(0),
            value.stride(1), pages, block, heads, kv_heads, dim, vdim, _capi.DTYPE_CODES[q.dtype], _capi.ptr(group.tables), group.sequences, width,
            _capi.ptr(group.lengths), _capi.ptr(group.local_cu), rows, group.max_new, float(terms.scale), int(terms.window), int(terms.keep_first),
            float(terms.softcap), _capi.ptr(terms.head_scale), _capi.ptr(talk), seen, _capi.ptr(workspace), nbytes, _capi.stream_of(q))
    _capi.check(code, "talking_attention")
    return out


def talking_prompt(q, keys, values, spread, ranges, terms: ScoreTerms, kv_heads: int):
    """`rlt_talking_prompt`: long portions over packed keys `[ranges.rows, kv_heads * dim]` and values `[ranges.rows, kv_heads * vdim]`."""
    _capi.require_cuda(q, keys, values, spread, terms.head_scale, ranges.tiles)
    _check(q, spread, terms)
    rows, heads, dim = q.shape
    if keys.shape != (ranges.rows, kv_heads * dim) or values.shape[0] != ranges.rows or spread.shape != (rows, heads, values.shape[1]) \
            or values.shape[1] % kv_heads or any(t.stride(1) != 1 or t.dtype != q.dtype for t in (keys, values)):
        raise ValueError("keys [packed, kv_heads * dim], values [packed, kv_heads * vdim], spread [rows, heads, kv_heads * vdim] of one dtype")
    if rows == 0:
        return spread
    workspace = torch.empty(256, dtype=torch.uint8, device=q.device)
    with torch.cuda.device(q.device):
        code = _capi.load().rlt_talking_prompt(
            _capi.ptr(q), q.stride(0), _capi.ptr(keys), keys.stride(0), _capi.ptr(values), values.stride(0), _capi.ptr(spread), spread.stride(0), rows,
            ranges.rows, heads, kv_heads, dim, values.shape[1] // kv_heads, _capi.ptr(ranges.tiles), ranges.tiles.shape[0], float(terms.scale),
            int(terms.window), int(terms.keep_first), float(terms.softcap), _capi.ptr(terms.head_scale), _capi.DTYPE_CODES[q.dtype],
            _capi.ptr(workspace), _capi.stream_of(q))
    _capi.check(code, "talking_prompt")
    return spread


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
