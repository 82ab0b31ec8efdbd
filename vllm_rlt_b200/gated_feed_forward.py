"""Gated feed-forwards of the model classes: a dense unit, W_down (act(W_gate h) * (W_up h)), and a mixture of such units with an optional
one that every token uses.

    dense      GEMM (gate, up), gated_unit, GEMM
    experts    GEMM (router), expert_route, expert_gather, expert_gemm (gate and up in pairs, the activation on the way out), expert_gemm (down);
               the weighted sum over a token's experts is part of the norm that follows, and the shared unit's output joins it there
"""

from __future__ import annotations

from dataclasses import dataclass

import torch
import torch.nn.functional as F

from .experts import expert_gather, expert_gemm, expert_route, paired_rows
from .layers import gated_unit
from .model_parts import check_positive, product32, stack_blocks, take_keys


@dataclass(frozen=True)
class GatedUnitConfig:
    ff: int

    @classmethod
    def from_json(cls, entry: dict, what: str, *, kind: bool = True) -> "GatedUnitConfig":
        ff = take_keys(entry, what, ("kind", "ff") if kind else ("ff",))["ff"]
        check_positive(what, ff=ff)
        return cls(ff)

    def parameter_shapes(self, prefix: str, width: int) -> dict[str, tuple]:
        return {prefix + "gate": (self.ff, width), prefix + "up": (self.ff, width), prefix + "down": (width, self.ff)}


@dataclass(frozen=True)
class GatedExpertsConfig:
    experts: int
    top: int
    expert: GatedUnitConfig
    shared: GatedUnitConfig | None = None

    @classmethod
    def from_json(cls, entry: dict, what: str) -> "GatedExpertsConfig":
        m = take_keys(entry, what, ("kind", "expert", "router"), ("shared",))
        router = take_keys(m["router"], what + " router", ("experts", "top"))
        check_positive(what + " router", **router)
        if router["top"] > router["experts"]:
            raise ValueError(f"{what}: top exceeds the number of experts")
        unit = lambda name: GatedUnitConfig.from_json(m[name], f"{what} {name}", kind=False)
        return cls(router["experts"], router["top"], unit("expert"), unit("shared") if m["shared"] else None)

    def parameter_shapes(self, prefix: str, width: int) -> dict[str, tuple]:
        shapes = {prefix + "router": (self.experts, width), prefix + "router.b": (self.experts,)}
        for e in range(self.experts):
            shapes.update(self.expert.parameter_shapes(f"{prefix}e{e}.", width))
        if self.shared:
            shapes.update(self.shared.parameter_shapes(prefix + "shared.", width))
        return shapes


FEED_FORWARDS = {"dense": GatedUnitConfig, "moe": GatedExpertsConfig}


def feed_forward_config(entry: dict | None, what: str):
    """The configuration an `mlp` entry describes, None for none."""
    if not entry:
        return None
    if entry.get("kind") not in FEED_FORWARDS:
        raise ValueError(f"{what}: unknown feed-forward kind {entry.get('kind')!r}; known: {', '.join(FEED_FORWARDS)}")
    return FEED_FORWARDS[entry["kind"]].from_json(entry, what)


class GatedUnit:
    """A dense unit's stacked weights, and its step."""

    def __init__(self, config: GatedUnitConfig, prefix: str, take, activation: str):
        self.ff, self.activation = config.ff, activation
        self.w_gate_up, (_, self.up_col), _ = stack_blocks([take(prefix + "gate"), take(prefix + "up")], 0)
        self.w_down = take(prefix + "down")

    def __call__(self, h):
        return F.linear(gated_unit(F.linear(h, self.w_gate_up), self.up_col, self.ff, self.activation), self.w_down)


class GatedExperts:
    """The experts' stacked weights, and their step."""

    def __init__(self, config: GatedExpertsConfig, prefix: str, take, activation: str):
        self.config, self.activation = config, activation
        self.router, self.bias = take(prefix + "router"), take(prefix + "router.b", torch.float32)
        names = [f"{prefix}e{e}." for e in range(config.experts)]
        self.w_gate_up = torch.stack([paired_rows(take(n + "gate"), take(n + "up")) for n in names])
        self.w_down = torch.stack([take(n + "down") for n in names])
        self.shared = GatedUnit(config.shared, prefix + "shared.", take, activation) if config.shared else None

    def __call__(self, h, queue):
        """(the shared unit's output or None, (experts' outputs, their rows, their weights)).  queue: int32 [experts] of zeros."""
        routing = expert_route(product32(h, self.router), None, self.config.top, bias=self.bias, counts=queue, floor_sum=0.0)
        act = expert_gemm(expert_gather(h, routing), self.w_gate_up, routing.counts, self.activation, paired=True)
        y = expert_gemm(act, self.w_down, routing.counts)
        return self.shared(h) if self.shared else None, (y, routing.places, routing.weights)
