"""Degavik: a decoder that norms its sublayers' outputs only, whose mixers are the gated delta rule with a decay per channel, retention, or
windowed attention with bounded scores and talking heads, in any order, each followed by a dense or mixture-of-experts feed-forward or none.

    x <- x + norm(mixer(x));    x <- x + norm(ff(x))

The residual x is one 32-bit row, and sublayers read it as it is.  The norm behind a sublayer, its addition (and the weighted sum over a
token's experts in front of it) and the operand of the next sublayer are a single pass (`residual_norm`), so a layer is two of those, the
mixer (`delta_mixer`, `retention_mixer`, `talking_mixer`) and the feed-forward (`gated_feed_forward`).  A layer may use another one's
weights, with pages and state of its own.  In bf16 the residual, norms, angles, scores, softmax, router, recurrent state and what drives it
are fp32; in float32 everything is.
"""

from __future__ import annotations

from dataclasses import dataclass

import torch

from .attention import B200PagedAttention
from .delta_mixer import ChannelDelta, ChannelDeltaConfig
from .gated_feed_forward import GatedExperts, GatedExpertsConfig, GatedUnit, GatedUnitConfig, feed_forward_config
from .layers import residual_norm
from .model_parts import check_positive, check_shapes, full_accumulation, product32, take_keys
from .retention_mixer import Retention, RetentionConfig
from .sequence_cache import CacheSpec
from .talking_mixer import TalkingAttention, TalkingAttentionConfig


# ---- configuration -----------------------------------------------------------------------------
MIXERS = {"channel_delta": ChannelDeltaConfig, "attention": TalkingAttentionConfig, "retention": RetentionConfig}


@dataclass(frozen=True)
class PostNormLayerConfig:
    mixer: ChannelDeltaConfig | TalkingAttentionConfig | RetentionConfig
    ff: GatedUnitConfig | GatedExpertsConfig | None
    weights: int              # the layer whose weights it uses, mostly itself


@dataclass(frozen=True)
class PostNormLMConfig:
    vocab: int
    width: int
    eps: float
    layers: tuple

    @classmethod
    def from_json(cls, config: dict) -> "PostNormLMConfig":
        check_positive("config", vocab=config.get("vocab"), width=config.get("width"))
        top = take_keys({k: v for k, v in config.items() if k in ("norm", "layers")}, "config", ("norm", "layers"))
        layers = []
        for i, entry in enumerate(top["layers"]):
            what = f"layer {i}"
            entry = take_keys(entry, what, ("type", "mixer"), ("mlp", "weights_of"))
            if entry["type"] not in MIXERS:
                raise ValueError(f"{what}: unknown mixer type {entry['type']!r}; known: {', '.join(MIXERS)}")
            source = i if entry["weights_of"] is None else entry["weights_of"]
            if isinstance(source, bool) or not isinstance(source, int) or not 0 <= source < len(top["layers"]):
                raise ValueError(f"{what}: weights_of must be the number of a layer")
            layers.append(PostNormLayerConfig(MIXERS[entry["type"]].from_json(entry["mixer"], what), feed_forward_config(entry["mlp"], what + " mlp"), source))
        if not layers:
            raise ValueError("config: a model needs layers")
        for i, layer in enumerate(layers):
            source = i
            for _ in layers:                       # a layer may use the weights of one that uses another's
                source = layers[source].weights
            if layers[source].weights != source:
                raise ValueError(f"layer {i}: weights_of leads in a circle")
            if (layers[source].mixer, layers[source].ff) != (layer.mixer, layer.ff):
                raise ValueError(f"layer {i}: uses the weights of layer {source}, whose entry differs")
            layers[i] = PostNormLayerConfig(layer.mixer, layer.ff, source)
        return cls(config["vocab"], config["width"], float(take_keys(top["norm"], "norm", ("eps",))["eps"]), tuple(layers))

    @property
    def own(self) -> list[int]:
        """The layers with weights of their own."""
        return [i for i, layer in enumerate(self.layers) if layer.weights == i]


def parameter_shapes(config: PostNormLMConfig, rank_of) -> dict[str, tuple]:
    """rank_of(name): the rank of the low-rank projection whose first tensor has this name."""
    w = config.width
    shapes = {"embed": (config.vocab, w), "final.norm": (w,), "head": (config.vocab, w)}
    for i in config.own:
        p, layer = f"l{i}.", config.layers[i]
        shapes[p + "norm1"] = (w,)
        shapes.update(layer.mixer.parameter_shapes(p + "mix.", w, rank_of))
        if layer.ff:
            shapes[p + "norm2"] = (w,)
            shapes.update(layer.ff.parameter_shapes(p + "mlp.", w))
    return shapes


# ---- the model ---------------------------------------------------------------------------------
class _Layer:
    """One layer's weights: its mixer, its feed-forward and the norms behind them."""

    def __init__(self, model: "PostNormLM", index: int, take):
        config, p, eps = model.config.layers[index], f"l{index}.", model.config.eps
        if isinstance(config.mixer, ChannelDeltaConfig):
            self.mixer = ChannelDelta(config.mixer, p + "mix.", take, eps)
        elif isinstance(config.mixer, RetentionConfig):
            self.mixer = Retention(config.mixer, p + "mix.", take, eps)
        else:
            self.mixer = TalkingAttention(config.mixer, p + "mix.", take, model.attention, eps)
        self.mixer_norm = take(p + "norm1", torch.float32)
        self.ff = None
        if config.ff:
            self.ff_norm = take(p + "norm2", torch.float32)
            kind = GatedUnit if isinstance(config.ff, GatedUnitConfig) else GatedExperts
            self.ff = kind(config.ff, p + "mlp.", take, model.activation)


class PostNormLM:
    """Inference-only model with norms behind its sublayers; see the module docstring."""

    activation = "silu"

    def __init__(self, config: PostNormLMConfig, state_dict: dict, device="cuda", dtype: torch.dtype = torch.bfloat16,
                 attention: B200PagedAttention | None = None):
        if dtype not in (torch.float32, torch.bfloat16):
            raise ValueError("PostNormLM runs in float32 or bfloat16")
        self.config, self.device, self.dtype = config, torch.device(device), dtype
        check_shapes(parameter_shapes(config, lambda name: state_dict[name].shape[0] if name in state_dict else 1), state_dict)

        def take(name, as_type=None):
            return state_dict[name].to(device=self.device, dtype=as_type or dtype).contiguous()

        self.attention = attention or B200PagedAttention()
        self.embed, self.head, self.final_norm = take("embed"), take("head"), take("final.norm", torch.float32)
        own = {i: _Layer(self, i, take) for i in config.own}
        self.layers = [own[layer.weights] for layer in config.layers]

    @property
    def vocab_size(self) -> int:
        return self.config.vocab

    def cache_spec(self) -> CacheSpec:
        layers, states = {}, {}
        for i, layer in enumerate(self.config.layers):
            if isinstance(layer.mixer, TalkingAttentionConfig):
                layers[i] = layer.mixer.cache
            else:
                states.update({f"l{i}.{name}": spec for name, spec in layer.mixer.states.items()})
        return CacheSpec(layers=layers, states=states, block=64)      # a page is a stage of the attention over pages

    # ---- one step ------------------------------------------------------------------------------
    def _add(self, residual, pending, weight=None, **kw):
        """The residual after the pending sublayer's output was added: the next sublayer's operand, or with a weight its norm."""
        delta, parts, behind = pending if pending else (None, None, None)
        return residual_norm(residual, weight, self.config.eps, self.dtype, delta=delta, parts=parts, behind=None if behind is None else (behind, 1.0), **kw)

    def forward_step(self, batch, cache, after_layer=None):
        """All rows of an engine step through every layer.  Returns (residual, last sublayer's output and norm): `step_logits` adds
        the two for the rows that need logits.  `after_layer(i, residual)` is called with the complete residual after every layer
        (tests and debugging: it costs a pass over the residual)."""
        c = self.config
        residual = torch.empty(batch.rows, c.width, dtype=torch.float32, device=self.device)
        routed = [i for i, layer in enumerate(c.layers) if isinstance(layer.ff, GatedExpertsConfig)]
        counts = torch.zeros(len(routed), max((c.layers[i].ff.experts for i in routed), default=0), dtype=torch.int32, device=self.device)
        queues = dict(zip(routed, counts))
        pending = None
        with full_accumulation(), self.attention.shared_plan():
            for i, layer in enumerate(self.layers):
                h = self._add(residual, pending, **({} if pending else dict(tokens=batch.tokens, embed=self.embed)))
                if isinstance(layer.mixer, TalkingAttention):
                    delta = layer.mixer(h, cache.key[i], cache.value[i], batch)
                else:
                    delta = layer.mixer(h, lambda name: cache.state[f"l{i}.{name}"], batch)
                pending = delta, None, layer.mixer_norm
                if layer.ff is not None:
                    h = self._add(residual, pending)
                    delta, parts = layer.ff(h, queues[i][:c.layers[i].ff.experts]) if i in queues else (layer.ff(h), None)
                    pending = delta, parts, layer.ff_norm
                if after_layer is not None:
                    total = residual.clone()
                    self._add(total, pending)
                    after_layer(i, total)
        return residual, pending

    def step_logits(self, hidden, rows=None):
        """fp32 logits of the given rows (int64 indices; None: all)."""
        residual, pending = hidden
        with full_accumulation():
            return product32(self._add(residual, pending, self.final_norm, row_index=rows, store=False), self.head)
