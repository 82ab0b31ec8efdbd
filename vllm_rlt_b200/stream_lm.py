"""Sugosun: a decoder over hyper-connected residual streams whose mixers are latent attention or lightning attention, with
dense or mixture-of-experts feed-forwards, and a range of layers that may run several times.

The residual is S 32-bit streams.  Every sublayer (mixer, feed-forward) reads a weighted sum of them through its norm and
writes to all of them through a small mixing matrix; `stream_mix` does the writing of one sublayer and the reading of the
next in one pass, so a layer is

    latent attention   as in `latent_mixer`, with a window
    lightning          GEMM (q, k, v, gate), block_epilogue (silu), decay_scan, gated_norm, GEMM
    dense              GEMM (gate, up), clamped_glu, GEMM
    experts            GEMM (router), expert_route, expert_gather, expert_gemm (up, squared relu), expert_gemm (down); their
                       weighted sum is part of the next stream_mix

with one `stream_mix` in front of each sublayer.  The cache row of a token is [latent | rotated key part], shared by all heads.
Layers of the loop keep pages and state per pass: both are numbered by layer run.  In bf16 the streams, norms, angles, scores,
softmax, router and recurrent state are fp32; in float32 everything is.
"""

from __future__ import annotations

from dataclasses import dataclass
from functools import partial

import torch
import torch.nn.functional as F

from .attention import B200PagedAttention
from .experts import expert_gather, expert_gemm, expert_route
from .latent_mixer import LatentAttention, LatentAttentionConfig
from .layers import block_epilogue, clamped_glu, stream_mix
from .model_parts import check_positive, check_shapes, full_accumulation, product32, stack_blocks, take_keys
from .recurrent import decay_scan, decay_table, gated_norm
from .sequence_cache import CacheSpec, StateSpec


# ---- configuration -----------------------------------------------------------------------------
@dataclass(frozen=True)
class LightningConfig:
    heads: int
    dim: int
    vdim: int
    decay: tuple

    @classmethod
    def from_json(cls, entry: dict, what: str) -> "LightningConfig":
        m = take_keys(entry, what, ("heads", "dim", "vdim", "decay"))
        check_positive(what, heads=m["heads"], dim=m["dim"], vdim=m["vdim"])
        decay = tuple(float(d) for d in m["decay"])
        if len(decay) != m["heads"] or not all(0.0 <= d <= 1.0 for d in decay):
            raise ValueError(f"{what}: decay needs one number between 0 and 1 per head")
        return cls(m["heads"], m["dim"], m["vdim"], decay)


MIXERS = {"latent_attention": partial(LatentAttentionConfig.from_json, windowed=True), "lightning": LightningConfig.from_json}


@dataclass(frozen=True)
class DenseConfig:
    ff: int
    limit: float

    @classmethod
    def from_json(cls, entry: dict, what: str) -> "DenseConfig":
        m = take_keys(entry, what, ("kind", "ff", "limit"))
        check_positive(what, ff=m["ff"])
        return cls(m["ff"], float(m["limit"]))


@dataclass(frozen=True)
class ExpertsConfig:
    experts: int
    top: int
    ff: int

    @classmethod
    def from_json(cls, entry: dict, what: str) -> "ExpertsConfig":
        m = take_keys(entry, what, ("kind", "expert", "router"))
        expert, router = take_keys(m["expert"], what + " expert", ("ff",)), take_keys(m["router"], what + " router", ("experts", "top"))
        check_positive(what, ff=expert["ff"], **router)
        if router["top"] > router["experts"]:
            raise ValueError(f"{what}: top exceeds the number of experts")
        return cls(router["experts"], router["top"], expert["ff"])


FEED_FORWARDS = {"dense": DenseConfig, "moe": ExpertsConfig}


@dataclass(frozen=True)
class StreamLayerConfig:
    mixer: LatentAttentionConfig | LightningConfig
    ff: DenseConfig | ExpertsConfig | None = None


@dataclass(frozen=True)
class BigramConfig:
    buckets: int
    mul_prev: int
    mul_cur: int


@dataclass(frozen=True)
class StreamLMConfig:
    vocab: int
    width: int
    eps: float
    streams: int
    layers: tuple
    bigram: BigramConfig | None = None
    loop: tuple = (0, 0, 1)           # start, stop, times

    @classmethod
    def from_json(cls, config: dict) -> "StreamLMConfig":
        check_positive("config", vocab=config.get("vocab"), width=config.get("width"), streams=config.get("streams"))
        layers = []
        for i, entry in enumerate(config["layers"]):
            what = f"layer {i}"
            entry = take_keys(entry, what, ("type", "mixer"), ("mlp",))
            if entry["type"] not in MIXERS:
                raise ValueError(f"{what}: unknown mixer type {entry['type']!r}; known: {', '.join(MIXERS)}")
            mixer, ff = MIXERS[entry["type"]](entry["mixer"], what), None
            if entry["mlp"]:
                kind = entry["mlp"].get("kind")
                if kind not in FEED_FORWARDS:
                    raise ValueError(f"{what}: unknown feed-forward kind {kind!r}; known: {', '.join(FEED_FORWARDS)}")
                ff = FEED_FORWARDS[kind].from_json(entry["mlp"], what + " mlp")
            layers.append(StreamLayerConfig(mixer, ff))
        bigram = None
        embedding = take_keys(config.get("embedding") or {}, "embedding", (), ("bigram",))
        if embedding["bigram"]:
            b = take_keys(embedding["bigram"], "embedding.bigram", ("buckets", "mul_prev", "mul_cur"))
            check_positive("embedding.bigram", buckets=b["buckets"])
            bigram = BigramConfig(b["buckets"], int(b["mul_prev"]), int(b["mul_cur"]))
            if bigram.mul_prev < 0 or bigram.mul_cur < 0 or config["vocab"] * (bigram.mul_prev + bigram.mul_cur) >= 2 ** 63:
                raise ValueError("embedding.bigram: multipliers must be non-negative and their products fit 64 bits")
        loop = (0, 0, 1)
        if config.get("loop"):
            entry = take_keys(config["loop"], "loop", ("start", "stop", "times"))
            loop = (entry["start"], entry["stop"], entry["times"])
            check_positive("loop", times=loop[2])
            if not 0 <= loop[0] <= loop[1] <= len(layers):
                raise ValueError("loop: start .. stop must lie within the layers")
        return cls(config["vocab"], config["width"], float(config["norm"]["eps"]), config["streams"], tuple(layers), bigram, loop)

    @property
    def runs(self) -> list[int]:
        """The layer of every run, in order: the looped range as often as the loop says."""
        start, stop, times = self.loop
        everything = list(range(len(self.layers)))
        return everything[:start] + everything[start:stop] * times + everything[stop:]


def parameter_shapes(config: StreamLMConfig) -> dict[str, tuple]:
    w, s = config.width, config.streams
    shapes = {"embed": (config.vocab, w), "embed.norm": (w,), "final.norm": (w,), "head": (config.vocab, w)}
    if config.bigram:
        shapes["bigram"] = (config.bigram.buckets + 1, w)
    for i, layer in enumerate(config.layers):
        p, m, f = f"l{i}.", layer.mixer, layer.ff
        for q in (1, 2) if f else (1,):
            shapes.update({f"{p}norm{q}": (w,), f"{p}hc{q}.in": (s,), f"{p}hc{q}.out": (s,), f"{p}hc{q}.mix": (s, s)})
        if isinstance(m, LatentAttentionConfig):
            shapes.update(m.parameter_shapes(p + "mix.", w))
        else:
            inner = m.heads * m.vdim
            shapes.update({p + "mix.q": (m.heads * m.dim, w), p + "mix.k": (m.heads * m.dim, w), p + "mix.v": (inner, w),
                           p + "mix.g": (inner, w), p + "mix.norm": (inner,), p + "mix.o": (w, inner)})
        if isinstance(f, DenseConfig):
            shapes.update({p + "mlp.gate": (f.ff, w), p + "mlp.up": (f.ff, w), p + "mlp.down": (w, f.ff)})
        elif f:
            shapes.update({p + "mlp.router": (f.experts, w), p + "mlp.correction": (f.experts,)})
            for e in range(f.experts):
                shapes[f"{p}mlp.e{e}.up"], shapes[f"{p}mlp.e{e}.down"] = (f.ff, w), (w, f.ff)
    return shapes


# ---- the model ---------------------------------------------------------------------------------
@dataclass
class _Sublayer:
    """A sublayer's place between the streams: the norm in front of it, what it reads, what its output does."""

    norm: torch.Tensor
    reads: torch.Tensor       # [S]
    writes: tuple             # (out [S], mix [S, S])


@dataclass
class _Pending:
    """A sublayer's output that has not been added to the streams yet."""

    writes: tuple
    delta: torch.Tensor
    parts: tuple | None = None


class _Layer:
    """Stacked weights of one layer and where their columns lie."""

    def __init__(self, model: "StreamLM", index: int, take):
        config = model.config.layers[index]
        self.mixer, self.ff = config.mixer, config.ff
        m, f, p = self.mixer, self.ff, f"l{index}."
        fp32 = lambda name: take(p + name, torch.float32)
        self.sublayers = [_Sublayer(fp32(f"norm{q}"), fp32(f"hc{q}.in"), (fp32(f"hc{q}.out"), fp32(f"hc{q}.mix")))
                          for q in ((1, 2) if f else (1,))]
        if isinstance(m, LatentAttentionConfig):
            self.latent = LatentAttention(m, p + "mix.", take, model.attention, model.config.eps, model.device)
        else:
            self.w_o = take(p + "mix.o")
            self.w_in, (self.q_at, self.k_at, self.v_at, self.g_at), _ = stack_blocks([take(p + "mix." + n) for n in "qkvg"], 0)
            self.out_norm = fp32("mix.norm")
            self.decay = decay_table(m.decay, model.device)
        if isinstance(f, DenseConfig):
            self.w_gate_up, (_, self.up_col), _ = stack_blocks([take(p + "mlp.gate"), take(p + "mlp.up")], 0)
            self.w_ff_down = take(p + "mlp.down")
        elif f:
            self.router, self.correction = take(p + "mlp.router"), fp32("mlp.correction")
            self.e_up = torch.stack([take(f"{p}mlp.e{e}.up") for e in range(f.experts)])
            self.e_down = torch.stack([take(f"{p}mlp.e{e}.down") for e in range(f.experts)])


class StreamLM:
    """Inference-only model over hyper-connected streams; see the module docstring."""

    glu_slope = 1.702

    def __init__(self, config: StreamLMConfig, state_dict: dict, device="cuda", dtype: torch.dtype = torch.bfloat16,
                 attention: B200PagedAttention | None = None):
        if dtype not in (torch.float32, torch.bfloat16):
            raise ValueError("StreamLM runs in float32 or bfloat16")
        self.config, self.device, self.dtype = config, torch.device(device), dtype
        check_shapes(parameter_shapes(config), state_dict)

        def take(name, as_type=None):
            return state_dict[name].to(device=self.device, dtype=as_type or dtype).contiguous()

        self.attention = attention or B200PagedAttention()
        self.embed, self.head = take("embed"), take("head")
        self.embed_norm, self.final_norm = take("embed.norm", torch.float32), take("final.norm", torch.float32)
        b = config.bigram
        self.bigram = (take("bigram"), b.mul_prev, b.mul_cur) if b else None
        self.layers = [_Layer(self, i, take) for i in range(len(config.layers))]

    @property
    def vocab_size(self) -> int:
        return self.config.vocab

    def cache_spec(self) -> CacheSpec:
        layers, states = {}, {}
        for run, i in enumerate(self.config.runs):
            m = self.config.layers[i].mixer
            if isinstance(m, LatentAttentionConfig):
                layers[run] = m.cache
            else:
                states[f"r{run}.state"] = StateSpec((m.heads, m.dim, m.vdim), torch.float32)
        return CacheSpec(layers=layers, states=states, block=64)      # a page is a stage of the attention over cache rows

    # ---- one step ------------------------------------------------------------------------------
    def _mix(self, streams, pending, norm, reads, **kw):
        return stream_mix(streams, norm, self.config.eps, self.dtype, delta=pending.delta if pending else None,
                          parts=pending.parts if pending else None, ran=pending.writes if pending else None, follows=reads, **kw)

    def forward_step(self, batch, cache, after_layer=None):
        """All rows of an engine step through every layer run.  Returns (streams, last sublayer's output): `step_logits` adds
        the two for the rows that need logits.  `after_layer(run, residual)` is called with the complete sum of the streams
        after every run (tests and debugging: it costs a pass over the streams)."""
        c = self.config
        streams = torch.empty(batch.rows, c.streams, c.width, dtype=torch.float32, device=self.device)
        pending = None
        routed = [r for r, i in enumerate(c.runs) if isinstance(c.layers[i].ff, ExpertsConfig)]
        counts = torch.zeros(len(routed), max((c.layers[c.runs[r]].ff.experts for r in routed), default=0), dtype=torch.int32, device=self.device)
        queues = dict(zip(routed, counts))
        with full_accumulation(), self.attention.shared_plan():
            for run, index in enumerate(c.runs):
                layer = self.layers[index]
                for q, sub in enumerate(layer.sublayers):
                    start = {} if pending else dict(tokens=batch.tokens, previous=batch.previous, embed=self.embed, bigram=self.bigram,
                                                    embed_weight=self.embed_norm)
                    h = self._mix(streams, pending, sub.norm, sub.reads, **start)
                    parts = None
                    if q == 0:
                        latent = isinstance(layer.mixer, LatentAttentionConfig)
                        delta = layer.latent(h, cache.key[run], batch) if latent else self._lightning(run, layer, h, batch, cache)
                    elif isinstance(layer.ff, DenseConfig):
                        act = clamped_glu(F.linear(h, layer.w_gate_up), layer.up_col, layer.ff.ff, layer.ff.limit, self.glu_slope)
                        delta = F.linear(act, layer.w_ff_down)
                    else:
                        delta, parts = self._experts(layer, h, queues[run][:layer.ff.experts])
                    pending = _Pending(sub.writes, delta, parts)
                if after_layer is not None:
                    total = streams.clone()
                    self._mix(total, pending, self.final_norm, None)
                    after_layer(run, total.sum(1))
        return streams, pending

    def _lightning(self, run, layer, h, batch, cache):
        m, rows = layer.mixer, h.shape[0]
        proj = F.linear(h, layer.w_in)
        qkv = torch.empty(rows, layer.g_at, dtype=self.dtype, device=self.device)
        block_epilogue(proj, batch, act=(0, layer.g_at, "silu", qkv, 0))
        inner, keys = m.heads * m.vdim, m.heads * m.dim
        q, k, v = (qkv[:, at:at + n] for at, n in ((layer.q_at, keys), (layer.k_at, keys), (layer.v_at, inner)))
        y = torch.empty(rows, inner, dtype=self.dtype, device=self.device)
        for group in batch.groups:
            decay_scan(q, k, v, layer.decay, cache.state[f"r{run}.state"], y, group)
        gated = torch.empty_like(y)
        gated_norm(y, proj[:, layer.g_at:layer.g_at + inner], layer.out_norm, gated, 1, self.config.eps, gate_behind=True)
        return F.linear(gated, layer.w_o)

    def _experts(self, layer, h, queue):
        routing = expert_route(product32(h, layer.router), layer.correction, layer.ff.top, counts=queue)
        x = expert_gather(h, routing)
        y = expert_gemm(expert_gemm(x, layer.e_up, routing.counts, "squared_relu"), layer.e_down, routing.counts)
        return y, (routing.places, routing.weights)

    def step_logits(self, hidden, rows=None):
        """fp32 logits of the given rows (int64 indices; None: all)."""
        streams, pending = hidden
        with full_accumulation():
            return product32(self._mix(streams, pending, self.final_norm, None, row_index=rows, store=False), self.head)
