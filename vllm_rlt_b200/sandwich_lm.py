"""Kezuvik: a decoder with a layer norm on both sides of every sublayer, whose mixers are latent attention of two kinds or windowed
attention behind a short convolution, in any order, each followed by a gated feed-forward or none.

    x <- x + m * norm_b(mixer(norm(x)));    x <- x + m * norm_b(ff(norm(x)))

The residual x is one 32-bit row.  The norm behind a sublayer, its addition and the norm in front of the next one are a single pass
(`residual_norm`), so a layer is two of those, the mixer (`latent_mixer`, `windowed_mixer`), and

    feed-forward    GEMM (gate, up), gated_unit (tanh gelu), GEMM

The embedding table is also the head; logits are bounded softly.  In bf16 the residual, norms, angles, scores and softmax are fp32; in
float32 everything is.
"""

from __future__ import annotations

from dataclasses import dataclass
from functools import partial

import torch
import torch.nn.functional as F

from .attention import B200PagedAttention
from .latent_mixer import LatentAttention, LatentAttentionConfig
from .layers import gated_unit, residual_norm, soft_cap
from .model_parts import check_positive, check_shapes, full_accumulation, product32, stack_blocks, take_keys
from .sequence_cache import CacheSpec
from .windowed_mixer import WindowedAttention, WindowedAttentionConfig


# ---- configuration -----------------------------------------------------------------------------
MIXERS = {
    "latent_attention": partial(LatentAttentionConfig.from_json, halves=True, gate="element"),
    "latent_attention_2": partial(LatentAttentionConfig.from_json, halves=True, scaled=True, sink=True, gate="head"),
    "attention": WindowedAttentionConfig.from_json,
}


@dataclass(frozen=True)
class SandwichLayerConfig:
    mixer: LatentAttentionConfig | WindowedAttentionConfig
    ff: int = 0           # 0: no feed-forward


@dataclass(frozen=True)
class SandwichLMConfig:
    vocab: int
    width: int
    eps: float
    residual_mult: float
    logit_softcap: float
    layers: tuple

    @classmethod
    def from_json(cls, config: dict) -> "SandwichLMConfig":
        check_positive("config", vocab=config.get("vocab"), width=config.get("width"))
        top = take_keys({k: v for k, v in config.items() if k in ("residual_mult", "logit_softcap", "norm", "layers")}, "config",
                        ("residual_mult", "logit_softcap", "norm", "layers"))
        if not top["logit_softcap"] > 0:
            raise ValueError("config: logit_softcap must be positive")
        layers = []
        for i, entry in enumerate(top["layers"]):
            what = f"layer {i}"
            entry = take_keys(entry, what, ("type", "mixer"), ("mlp",))
            if entry["type"] not in MIXERS:
                raise ValueError(f"{what}: unknown mixer type {entry['type']!r}; known: {', '.join(MIXERS)}")
            mixer, ff = MIXERS[entry["type"]](entry["mixer"], what), 0
            if entry["mlp"]:
                mlp = take_keys(entry["mlp"], what + " mlp", ("ff", "kind"))
                if mlp["kind"] != "dense":
                    raise ValueError(f"{what}: unknown feed-forward kind {mlp['kind']!r}")
                check_positive(what + " mlp", ff=mlp["ff"])
                ff = mlp["ff"]
            layers.append(SandwichLayerConfig(mixer, ff))
        if not layers:
            raise ValueError("config: a model needs layers")
        return cls(config["vocab"], config["width"], float(take_keys(top["norm"], "norm", ("eps",))["eps"]), float(top["residual_mult"]),
                   float(top["logit_softcap"]), tuple(layers))


def parameter_shapes(config: SandwichLMConfig) -> dict[str, tuple]:
    w = config.width
    shapes = {"embed": (config.vocab, w), "final.norm": (w,)}
    for i, layer in enumerate(config.layers):
        p = f"l{i}."
        for q in (1, 2) if layer.ff else (1,):
            shapes.update({f"{p}norm{q}": (w,), f"{p}norm{q}b": (w,)})
        shapes.update(layer.mixer.parameter_shapes(p + "mix.", w))
        if layer.ff:
            shapes.update({p + "mlp.gate": (layer.ff, w), p + "mlp.up": (layer.ff, w), p + "mlp.down": (w, layer.ff)})
    return shapes


# ---- the model ---------------------------------------------------------------------------------
class _Layer:
    """One layer's weights: the norms in front of and behind its sublayers, its mixer, its stacked feed-forward."""

    def __init__(self, model: "SandwichLM", index: int, take):
        config, p = model.config.layers[index], f"l{index}."
        self.ff = config.ff
        count = 2 if self.ff else 1
        self.before = [take(f"{p}norm{q + 1}", torch.float32) for q in range(count)]
        self.behind = [take(f"{p}norm{q + 1}b", torch.float32) for q in range(count)]
        eps = model.config.eps
        if isinstance(config.mixer, LatentAttentionConfig):
            self.mixer = LatentAttention(config.mixer, p + "mix.", take, model.attention, eps, model.device)
        else:
            self.mixer = WindowedAttention(config.mixer, p + "mix.", take, model.attention, eps)
        if self.ff:
            self.w_gate_up, (_, self.up_col), _ = stack_blocks([take(p + "mlp.gate"), take(p + "mlp.up")], 0)
            self.w_down = take(p + "mlp.down")


class SandwichLM:
    """Inference-only model with norms on both sides of its sublayers; see the module docstring."""

    activation = "gelu_tanh"

    def __init__(self, config: SandwichLMConfig, state_dict: dict, device="cuda", dtype: torch.dtype = torch.bfloat16,
                 attention: B200PagedAttention | None = None):
        if dtype not in (torch.float32, torch.bfloat16):
            raise ValueError("SandwichLM runs in float32 or bfloat16")
        self.config, self.device, self.dtype = config, torch.device(device), dtype
        check_shapes(parameter_shapes(config), state_dict)

        def take(name, as_type=None):
            return state_dict[name].to(device=self.device, dtype=as_type or dtype).contiguous()

        self.attention = attention or B200PagedAttention()
        self.embed, self.final_norm = take("embed"), take("final.norm", torch.float32)
        self.layers = [_Layer(self, i, take) for i in range(len(config.layers))]

    @property
    def vocab_size(self) -> int:
        return self.config.vocab

    def cache_spec(self) -> CacheSpec:
        mixers = {i: layer.mixer for i, layer in enumerate(self.config.layers)}
        return CacheSpec(layers={i: m.cache for i, m in mixers.items()},
                         states={f"l{i}.conv": m.state for i, m in mixers.items() if isinstance(m, WindowedAttentionConfig)},
                         block=64)       # a page is a stage of the attention over cache rows

    # ---- one step ------------------------------------------------------------------------------
    def _norm(self, residual, weight, pending, **kw):
        """The norm in front of a sublayer, after the output of the one before (pending: its output and the norm behind it) was added."""
        delta, behind = pending if pending else (None, None)
        return residual_norm(residual, weight, self.config.eps, self.dtype, delta=delta, centred=True,
                             behind=None if pending is None else (behind, self.config.residual_mult), **kw)

    def forward_step(self, batch, cache, after_layer=None):
        """All rows of an engine step through every layer.  Returns (residual, last sublayer's output and norm): `step_logits` adds
        the two for the rows that need logits.  `after_layer(i, residual)` is called with the complete residual after every layer
        (tests and debugging: it costs a pass over the residual)."""
        residual = torch.empty(batch.rows, self.config.width, dtype=torch.float32, device=self.device)
        pending = None
        with full_accumulation(), self.attention.shared_plan():
            for i, layer in enumerate(self.layers):
                start = {} if pending else dict(tokens=batch.tokens, embed=self.embed)
                h = self._norm(residual, layer.before[0], pending, **start)
                if isinstance(layer.mixer, LatentAttention):
                    delta = layer.mixer(h, cache.key[i], batch)
                else:
                    delta = layer.mixer(h, cache.key[i], cache.value[i], cache.state[f"l{i}.conv"], batch)
                pending = delta, layer.behind[0]
                if layer.ff:
                    h = self._norm(residual, layer.before[1], pending)
                    act = gated_unit(F.linear(h, layer.w_gate_up), layer.up_col, layer.ff, self.activation)
                    pending = F.linear(act, layer.w_down), layer.behind[1]
                if after_layer is not None:
                    total = residual.clone()
                    self._norm(total, self.final_norm, pending)
                    after_layer(i, total)
        return residual, pending

    def step_logits(self, hidden, rows=None):
        """fp32 logits of the given rows (int64 indices; None: all)."""
        residual, pending = hidden
        with full_accumulation():
            h = self._norm(residual, self.final_norm, pending, row_index=rows, store=False)
            return soft_cap(product32(h, self.embed), self.config.logit_softcap)
