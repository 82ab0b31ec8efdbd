"""Small random models and configurations for the tests of the decoder with norms on both sides of its sublayers."""

from __future__ import annotations

import torch


def latent_layer(heads, dim, rot_dim, vdim, q_rank, kv_rank, *, base=500.0, scale=None, scaling=None, second=False, ff=0):
    """`second`: the kind with a sink, a gate per head and, with scaling = (factor, original, fast, slow), scaled frequencies."""
    rot = {"base": base, "dims": rot_dim}
    if scaling:
        rot["scaling"] = dict(zip(("factor", "original", "fast", "slow"), scaling))
    return {"type": "latent_attention_2" if second else "latent_attention", "mlp": dense(ff),
            "mixer": {"heads": heads, "dim": dim, "rot_dim": rot_dim, "vdim": vdim, "q_rank": q_rank, "kv_rank": kv_rank,
                      "scale": scale or (dim + rot_dim) ** -0.5, "rot": rot}}


def windowed_layer(heads, kv_heads, dim, vdim, taps, window, *, scale=None, ff=0):
    return {"type": "attention", "mlp": dense(ff),
            "mixer": {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "conv": taps, "mask": {"size": window},
                      "scale": scale or 2.0 * dim ** -0.5}}


def dense(ff):
    return {"kind": "dense", "ff": ff} if ff else None


def make_config(layers, *, vocab, width, mult=0.6, cap=8.0, eps=1e-4):
    return {"architecture": "Kezuvik", "vocab": vocab, "width": width, "residual_mult": mult, "logit_softcap": cap, "norm": {"eps": eps},
            "layers": layers}


# Sizes that differ from layer to layer, values that are 1, rows and columns that are no multiple of anything.
CONFIGS = {
    "mixed": make_config([windowed_layer(4, 2, 24, 40, 4, 21, ff=88),
                          latent_layer(6, 24, 16, 40, 56, 48, second=True, base=1e4, scaling=(8.0, 512, 16.0, 0.5), ff=72),
                          latent_layer(3, 32, 8, 16, 24, 36, ff=40),                    # sizes the prompt kernel takes over a row it does not
                          windowed_layer(6, 3, 64, 32, 2, 70),
                          latent_layer(5, 40, 32, 24, 40, 64, base=1e4)],
                         vocab=131, width=96),
    "odd": make_config([latent_layer(5, 9, 6, 7, 13, 11, ff=33),
                        windowed_layer(3, 1, 10, 7, 1, 1, ff=17),
                        windowed_layer(1, 1, 5, 3, 6, 35),
                        latent_layer(1, 5, 2, 3, 6, 4, second=True, base=10.0, scaling=(2.0, 64, 4.0, 1.0), ff=9),
                        latent_layer(2, 7, 4, 1, 5, 9, second=True, base=300.0)],
                       vocab=83, width=52, mult=1.0, cap=3.0, eps=1e-3),
    "wide": make_config([latent_layer(4, 128, 64, 128, 96, 512, second=True, base=1e5, scaling=(40.0, 256, 32.0, 1.0), ff=200),
                         windowed_layer(8, 2, 128, 128, 3, 130, ff=104),
                         latent_layer(20, 64, 16, 80, 64, 72, base=1e4, ff=64),
                         windowed_layer(4, 4, 72, 136, 4, 64)],
                        vocab=211, width=128, mult=0.9, cap=20.0),
}


def random_weights(parameter_shapes, seed, dtype=torch.bfloat16):
    """Weights at a scale that keeps every mechanism visible: attention scores spread over several units, norm weights away from their
    neutral value, sinks among the larger scores, biases as large as what they are added to."""
    g = torch.Generator().manual_seed(seed)
    out = {}
    for name, shape in parameter_shapes.items():
        r = torch.randn(shape, generator=g)
        if "norm" in name.rsplit(".", 1)[-1]:
            r = 1 + 0.2 * r
        elif name.endswith("sink"):
            r = 2.0 + r
        elif name.endswith(".conv"):
            r = 0.3 * r
            r[:, -1] += 0.6
        elif name.endswith(".b"):
            r = 0.7 * r
        elif name == "embed":
            r = 0.5 * r
        elif name.endswith(("mix.uq", "mix.uk")):
            r = 1.5 * r / shape[1] ** 0.5
        else:
            r = r / shape[-1] ** 0.5
        out[name] = r.to(dtype)
    return out
