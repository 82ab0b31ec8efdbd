"""Small random models and configurations for the tests of the decoder that norms its sublayers' outputs only."""

from __future__ import annotations

import torch


def delta_layer(heads, kv_heads, dim, vdim, taps, *, mlp=None):
    return {"type": "channel_delta", "mlp": mlp, "mixer": {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "conv": taps}}


def attention_layer(heads, kv_heads, dim, vdim, window, keep, *, dims=None, base=300.0, scale=None, cap=15.0, mlp=None):
    return {"type": "attention", "mlp": mlp,
            "mixer": {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "scale": scale or 2.0 * dim ** -0.5, "softcap": cap,
                      "mask": {"size": window, "keep_first": keep}, "rot": {"base": base, "dims": dim // 2 * 2 if dims is None else dims}}}


def retention_layer(heads, dim, vdim, *, dims=None, base=1e4, decay=None, mlp=None):
    return {"type": "retention", "mlp": mlp,
            "mixer": {"heads": heads, "dim": dim, "vdim": vdim, "rot": {"base": base, "dims": dim // 2 * 2 if dims is None else dims},
                      "decay": decay or [1 - 2.0 ** (-1 - 1.3 * h) for h in range(heads)]}}


def dense(ff):
    return {"kind": "dense", "ff": ff}


def moe(experts, top, ff, shared=None):
    entry = {"kind": "moe", "router": {"experts": experts, "top": top}, "expert": {"ff": ff}}
    return entry | {"shared": {"ff": shared}} if shared else entry


def again(layers, j):
    """The entry of a layer that uses layer j's weights."""
    return layers[j] | {"weights_of": j}


def make_config(layers, *, vocab, width, eps=1e-4):
    return {"architecture": "Degavik", "vocab": vocab, "width": width, "norm": {"eps": eps}, "layers": layers}


# Sizes that differ from layer to layer, values that are 1, rows and columns that are no multiple of anything.
_MIXED = [attention_layer(4, 2, 24, 40, 21, 3, dims=16, mlp=moe(6, 2, 40, 56)),
          delta_layer(6, 3, 24, 40, 4, mlp=dense(72)),
          retention_layer(3, 40, 24, dims=24, mlp=moe(5, 5, 24)),
          delta_layer(4, 4, 64, 64, 3),
          attention_layer(6, 6, 64, 32, 70, 9, cap=30.0)]
_ODD = [delta_layer(3, 1, 9, 7, 6, mlp=dense(33)),
        attention_layer(3, 1, 10, 7, 1, 1, dims=2, mlp=moe(3, 1, 11, 7)),
        attention_layer(2, 2, 5, 3, 35, 0, cap=2.0),
        retention_layer(1, 7, 13, dims=2, decay=[0.8], mlp=dense(9)),
        delta_layer(1, 1, 5, 14, 1, mlp=moe(4, 3, 5)),
        retention_layer(2, 6, 15, decay=[1.0, 0.6])]
_WIDE = [delta_layer(4, 2, 128, 128, 4, mlp=moe(8, 3, 72, 40)),
         attention_layer(8, 2, 128, 128, 130, 70, dims=64, cap=50.0, mlp=dense(104)),
         retention_layer(2, 128, 128, mlp=dense(64)),
         attention_layer(12, 4, 72, 136, 64, 5, cap=90.0),
         delta_layer(2, 2, 80, 72, 2)]
CONFIGS = {
    "mixed": make_config([*_MIXED, again(_MIXED, 1), again(_MIXED, 0)], vocab=131, width=96),
    "odd": make_config([*_ODD, again(_ODD, 0)], vocab=83, width=52, eps=1e-3),
    "wide": make_config([*_WIDE, again(_WIDE, 2)], vocab=211, width=128),
}
RANKS = {"mixed": (12, 20), "odd": (3, 1), "wide": (64, 24)}


def rank_of(name):
    """Ranks of the two low-rank projections of a named configuration."""
    return lambda tensor: RANKS[name][tensor.endswith("g1")]


def random_weights(parameter_shapes, seed, dtype=torch.bfloat16, steady=True):
    """Weights at a scale that keeps every mechanism visible: attention scores spread over several units, norm weights away from their
    neutral value, mixing matrices and temperatures away from the identity, decays from a few tokens to hundreds.

    `steady`: routing without close calls, for models whose activations are rounded.  The first coordinates of every embedding
    row hold a ladder of well separated values in an order of the token's own, no sublayer writes to them, and the routers
    read nothing else."""
    g = torch.Generator().manual_seed(seed)
    out = {}
    for name, shape in parameter_shapes.items():
        r = torch.randn(shape, generator=g)
        last = name.rsplit(".", 1)[-1]
        if "norm" in last:
            r = 1 + 0.2 * r
        elif last == "conv":
            r = 0.3 * r
            r[:, -1] += 0.6
        elif last == "A_log":
            r = torch.linspace(-2.0, 1.0, shape[0]) + 0.1 * r
        elif last == "dt_bias":
            r = -3.0 + 1.5 * r
        elif last == "temp":
            r = 1 + 0.3 * r
        elif last == "talk":
            r = torch.eye(shape[0]) + 0.4 * r
        elif name == "embed":
            pass
        elif last == "router":
            r = 2.0 * r / shape[1] ** 0.5
        elif name.endswith("router.b"):
            r = 0.5 * r
        else:
            r = r / shape[-1] ** 0.5
        out[name] = r
    if steady:
        codes = max([shape[0] for name, shape in parameter_shapes.items() if name.endswith("router")], default=0)
        ladder = torch.linspace(-2.5, 2.5, max(codes, 1))
        for row in out["embed"]:
            row[:codes] = ladder[torch.randperm(codes, generator=g)]
        for name in out:
            if name.endswith((".o", ".down")):
                out[name][:codes] = 0
            elif name.endswith("router"):
                experts = out[name].shape[0]
                out[name].zero_()
                out[name][torch.arange(experts), torch.randperm(codes, generator=g)[:experts]] = 3.0
            elif name.endswith("router.b"):
                out[name].zero_()
                out[name][1 % len(out[name])] = 20.0         # chosen by every token
    return {name: r.to(dtype) for name, r in out.items()}
