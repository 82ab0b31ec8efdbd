"""Sobipel: a decoder of parallel blocks whose mixers are attention or Mamba-2 layers, in any order.

A layer reads one norm of the 32-bit residual stream and adds mixer and feed-forward to it together:

    h = rmsnorm(x) * (1 + w);    x <- x + mixer(h) + ff(h)

Both sublayers share their input and their output, so a layer is two GEMMs: the mixer's input projections
and the feed-forward's up projection stacked by rows, and the mixer's output projection and the down projection
side by side, over one operand into which the kernels in between write:

    attention   GEMM, block_epilogue (K and V to their pages, gelu), attention (+ merge), GEMM, residual_norm
    mamba2      GEMM, causal_conv (and gelu), ssd_scan, gated_norm, GEMM, residual_norm

Attention knows positions through a distance bias and a query temperature only (`ScoreTerms`); a layer may
attend to the keys and values another layer's cache holds (`kv_from`).  In bf16 the residual, norms, scores,
softmax, recurrent state and everything that drives it are fp32; in float32 everything is.
"""

from __future__ import annotations

from dataclasses import dataclass

import torch
import torch.nn.functional as F

from .attention import B200PagedAttention, ScoreTerms
from .layers import block_epilogue, residual_norm
from .model_parts import check_positive, check_shapes, full_accumulation, product32, stack_blocks, take_keys
from .recurrent import causal_conv, gated_norm, ssd_scan
from .sequence_cache import CacheSpec, KVSpec, StateSpec


# ---- configuration -----------------------------------------------------------------------------
@dataclass(frozen=True)
class AttentionConfig:
    heads: int
    kv_heads: int
    dim: int
    vdim: int
    scale: float
    temp_coef: float = 0.0
    temp_every: int = 1
    kv_from: int | None = None

    @classmethod
    def from_json(cls, entry: dict, what: str) -> "AttentionConfig":
        m = take_keys(entry, what, ("heads", "kv_heads", "dim", "vdim", "scale"), ("q_temp", "kv_from"))
        check_positive(what, heads=m["heads"], kv_heads=m["kv_heads"], dim=m["dim"], vdim=m["vdim"])
        if m["heads"] % m["kv_heads"]:
            raise ValueError(f"{what}: heads must be a multiple of kv_heads")
        temp = take_keys(m["q_temp"], what + " q_temp", ("coef", "every")) if m["q_temp"] else {"coef": 0.0, "every": 1}
        if int(temp["every"]) != temp["every"] or temp["every"] < 1:
            raise ValueError(f"{what}: q_temp.every must be a positive integer")
        return cls(m["heads"], m["kv_heads"], m["dim"], m["vdim"], float(m["scale"]), float(temp["coef"]), int(temp["every"]),
                   m["kv_from"])

    @property
    def terms(self) -> ScoreTerms:
        return ScoreTerms(self.scale, self.temp_coef, self.temp_every, distance_bias=True)


@dataclass(frozen=True)
class Mamba2Config:
    heads: int
    vdim: int
    state: int
    groups: int
    conv: int
    norm_groups: int

    @classmethod
    def from_json(cls, entry: dict, what: str) -> "Mamba2Config":
        m = take_keys(entry, what, ("heads", "vdim", "state", "groups", "conv", "norm_groups"))
        check_positive(what, **m)
        if m["heads"] % m["groups"] or m["heads"] * m["vdim"] % m["norm_groups"]:
            raise ValueError(f"{what}: heads must be a multiple of groups, and heads * vdim of norm_groups")
        return cls(**m)

    @property
    def inner(self) -> int:
        return self.heads * self.vdim

    @property
    def channels(self) -> int:        # what passes the convolution: x, B and C
        return self.inner + 2 * self.groups * self.state


MIXERS = {"attention": AttentionConfig, "mamba2": Mamba2Config}


@dataclass(frozen=True)
class HybridLayerConfig:
    mixer: AttentionConfig | Mamba2Config
    ff: int = 0                       # feed-forward width, 0 without one


@dataclass(frozen=True)
class HybridLMConfig:
    vocab: int
    width: int
    eps: float
    layers: tuple

    @classmethod
    def from_json(cls, config: dict) -> "HybridLMConfig":
        check_positive("config", vocab=config.get("vocab"), width=config.get("width"))
        layers = []
        for i, entry in enumerate(config["layers"]):
            what = f"layer {i}"
            entry = take_keys(entry, what, ("type", "mixer"), ("mlp",))
            if entry["type"] not in MIXERS:
                raise ValueError(f"{what}: unknown mixer type {entry['type']!r}; known: {', '.join(MIXERS)}")
            mixer = MIXERS[entry["type"]].from_json(entry["mixer"], what)
            ff = 0
            if entry["mlp"]:
                mlp = take_keys(entry["mlp"], what + " mlp", ("ff",), ("kind",))
                if mlp["kind"] not in (None, "dense"):
                    raise ValueError(f"{what}: unknown feed-forward kind {mlp['kind']!r}")
                check_positive(what + " mlp", ff=mlp["ff"])
                ff = mlp["ff"]
            layers.append(HybridLayerConfig(mixer, ff))
        built = cls(config["vocab"], config["width"], float(config["norm"]["eps"]), tuple(layers))
        built.check()
        return built

    def check(self) -> None:
        for i, layer in enumerate(self.layers):
            source = getattr(layer.mixer, "kv_from", None)
            if source is None:
                continue
            other = self.layers[source].mixer if isinstance(source, int) and 0 <= source < i else None
            if not isinstance(other, AttentionConfig) or other.kv_from is not None:
                raise ValueError(f"layer {i}: kv_from must name an earlier attention layer with projections of its own")
            if (other.kv_heads, other.dim, other.vdim) != (layer.mixer.kv_heads, layer.mixer.dim, layer.mixer.vdim):
                raise ValueError(f"layer {i}: kv_from layer {source} has other key/value sizes")


def parameter_shapes(config: HybridLMConfig) -> dict[str, tuple]:
    w = config.width
    shapes = {"embed": (config.vocab, w), "final.norm": (w,), "head": (config.vocab, w)}
    for i, layer in enumerate(config.layers):
        p, m = f"l{i}.", layer.mixer
        shapes[p + "norm1"] = (w,)
        if isinstance(m, AttentionConfig):
            shapes[p + "mix.q"] = (m.heads * m.dim, w)
            if m.kv_from is None:
                shapes[p + "mix.k"], shapes[p + "mix.v"] = (m.kv_heads * m.dim, w), (m.kv_heads * m.vdim, w)
            shapes[p + "mix.o"] = (w, m.heads * m.vdim)
        else:
            shapes.update({p + "mix.in": (m.inner + m.channels + m.heads, w), p + "mix.conv": (m.channels, m.conv),
                           p + "mix.conv.b": (m.channels,), p + "mix.dt_bias": (m.heads,), p + "mix.A_log": (m.heads,),
                           p + "mix.D": (m.heads,), p + "mix.norm": (m.inner,), p + "mix.o": (w, m.inner)})
        if layer.ff:
            shapes[p + "mlp.up"], shapes[p + "mlp.down"] = (layer.ff, w), (w, layer.ff)
    return shapes


# ---- the model ---------------------------------------------------------------------------------
class _Layer:
    """Stacked weights of one layer and where their columns lie."""

    def __init__(self, model: "HybridLM", index: int, take):
        config = model.config.layers[index]
        self.mixer, self.ff = config.mixer, config.ff
        p = f"l{index}."
        self.norm = take(p + "norm1", torch.float32)
        up = [take(p + "mlp.up")] if self.ff else []
        down = [take(p + "mlp.down")] if self.ff else []
        m = self.mixer
        if isinstance(m, AttentionConfig):
            self.source = index if m.kv_from is None else m.kv_from
            own = m.kv_from is None
            blocks = [take(p + "mix.q")] + ([take(p + "mix.k"), take(p + "mix.v")] if own else [])
            self.inner = m.heads * m.vdim
            self.w_in, offsets, _ = stack_blocks(blocks + up, 0)
            self.k_col, self.v_col = (offsets[1], offsets[2]) if own else (0, 0)
            self.terms = m.terms
        else:
            self.inner = m.inner
            self.w_in, offsets, _ = stack_blocks([take(p + "mix.in")] + up, 0)
            self.conv, self.conv_bias = take(p + "mix.conv", torch.float32), take(p + "mix.conv.b", torch.float32)
            self.dt_bias, self.a_log, self.d = (take(p + "mix." + n, torch.float32) for n in ("dt_bias", "A_log", "D"))
            self.gate_norm = take(p + "mix.norm", torch.float32)
        self.up_col = offsets[-1] if self.ff else 0
        self.w_out, offsets, self.operand_width = stack_blocks([take(p + "mix.o")] + down, 1)
        self.act_col = offsets[-1] if self.ff else 0
        self.padded = self.operand_width != self.inner + self.ff


class HybridLM:
    """Inference-only model of stacked parallel blocks; see the module docstring."""

    activation = "gelu"
    norm_offset = 1.0                 # norm weights are stored around zero

    def __init__(self, config: HybridLMConfig, state_dict: dict, device="cuda", dtype: torch.dtype = torch.bfloat16,
                 attention: B200PagedAttention | None = None):
        if dtype not in (torch.float32, torch.bfloat16):
            raise ValueError("HybridLM runs in float32 or bfloat16")
        self.config, self.device, self.dtype = config, torch.device(device), dtype
        check_shapes(parameter_shapes(config), state_dict)

        def take(name, as_type=None):
            return state_dict[name].to(device=self.device, dtype=as_type or dtype).contiguous()

        self.attention = attention or B200PagedAttention()
        self.embed, self.head = take("embed"), take("head")
        self.final_norm = take("final.norm", torch.float32)
        self.layers = [_Layer(self, i, take) for i in range(len(config.layers))]

    @property
    def vocab_size(self) -> int:
        return self.config.vocab

    def cache_spec(self) -> CacheSpec:
        layers, states = {}, {}
        for i, layer in enumerate(self.config.layers):
            m = layer.mixer
            if isinstance(m, Mamba2Config):
                states[f"l{i}.conv"] = StateSpec((m.conv - 1, m.channels))
                states[f"l{i}.ssm"] = StateSpec((m.heads, m.state, m.vdim), torch.float32)
            elif m.kv_from is None:
                layers[i] = KVSpec(m.kv_heads, m.dim, m.vdim)
        return CacheSpec(layers=layers, states=states)

    # ---- one step ------------------------------------------------------------------------------
    def forward_step(self, batch, cache, after_layer=None):
        """All rows of an engine step through every layer.  Returns (residual, last layer's contribution): the two are
        added, and normed, by `step_logits` for the rows that need logits.  `after_layer(i, residual)` is called with
        the complete 32-bit residual after every layer (tests and debugging: it costs an addition per layer)."""
        residual = torch.empty(batch.rows, self.config.width, dtype=torch.float32, device=self.device)
        eps, delta = self.config.eps, None
        with full_accumulation(), self.attention.shared_plan():
            for i, layer in enumerate(self.layers):
                first = i == 0
                h = residual_norm(residual, layer.norm, eps, self.dtype, delta=delta, tokens=batch.tokens if first else None,
                                  embed=self.embed if first else None, weight_offset=self.norm_offset)
                proj = F.linear(h, layer.w_in)
                operand = (torch.zeros if layer.padded else torch.empty)(batch.rows, layer.operand_width, dtype=self.dtype,
                                                                         device=self.device)
                if isinstance(layer.mixer, AttentionConfig):
                    self._attention(i, layer, proj, operand, batch, cache)
                else:
                    self._mamba2(i, layer, proj, operand, batch, cache)
                delta = F.linear(operand, layer.w_out)
                if after_layer is not None:
                    after_layer(i, residual + delta.float())
        return residual, delta

    def _attention(self, index, layer, proj, operand, batch, cache):
        m, rows = layer.mixer, batch.rows
        key, value = cache.key[layer.source], cache.value[layer.source]
        kv = (layer.k_col, layer.v_col, key, value) if m.kv_from is None else None
        act = (layer.up_col, layer.ff, self.activation, operand, layer.act_col) if layer.ff else None
        block_epilogue(proj, batch, kv=kv, act=act)
        q = proj[:, :m.heads * m.dim].view(rows, m.heads, m.dim)
        out = operand[:, :layer.inner].view(rows, m.heads, m.vdim)
        for group in batch.groups:
            self.attention.scored(q[group.rows], out[group.rows], key, value, group.tables, group.lengths, group.local_cu,
                                  group.max_new, layer.terms)

    def _mamba2(self, index, layer, proj, operand, batch, cache):
        m, rows = layer.mixer, batch.rows
        gate, xbc = proj[:, :m.inner], proj[:, m.inner:m.inner + m.channels]
        dt = proj[:, m.inner + m.channels:m.inner + m.channels + m.heads]
        mixed = torch.empty(rows, m.channels, dtype=self.dtype, device=self.device)
        y = torch.empty(rows, m.inner, dtype=self.dtype, device=self.device)
        act = (proj[:, layer.up_col:layer.up_col + layer.ff], self.activation,
               operand[:, layer.act_col:layer.act_col + layer.ff]) if layer.ff else None
        x, b, c = mixed.split((m.inner, m.groups * m.state, m.groups * m.state), dim=1)
        for group in batch.groups:
            causal_conv(xbc, layer.conv, layer.conv_bias, cache.state[f"l{index}.conv"], mixed, group, act=act)
            ssd_scan(x, b, c, dt, layer.dt_bias, layer.a_log, layer.d, cache.state[f"l{index}.ssm"], y, group)
        gated_norm(y, gate, layer.gate_norm, operand[:, :layer.inner], m.norm_groups, self.config.eps)

    def step_logits(self, hidden, rows=None):
        """fp32 logits of the given rows (int64 indices; None: all)."""
        residual, delta = hidden
        with full_accumulation():
            h = residual_norm(residual, self.final_norm, self.config.eps, self.dtype, delta=delta, row_index=rows,
                              weight_offset=self.norm_offset, store=False)
            return product32(h, self.head)
