"""Small random models and configurations for the tests of the decoder over hyper-connected streams."""

from __future__ import annotations

import torch


def latent_layer(heads, dim, rot_dim, vdim, q_rank, kv_rank, window, *, base=500.0, scale=None, mlp=None):
    return {"type": "latent_attention", "mlp": mlp,
            "mixer": {"heads": heads, "dim": dim, "rot_dim": rot_dim, "vdim": vdim, "q_rank": q_rank, "kv_rank": kv_rank,
                      "scale": scale or (dim + rot_dim) ** -0.5, "rot": {"base": base, "dims": rot_dim},
                      **({"mask": {"size": window}} if window else {})}}


def lightning_layer(decay, dim, vdim, *, mlp=None):
    return {"type": "lightning", "mlp": mlp, "mixer": {"heads": len(decay), "dim": dim, "vdim": vdim, "decay": list(decay)}}


def dense(ff, limit):
    return {"kind": "dense", "ff": ff, "limit": limit}


def moe(experts, top, ff):
    return {"kind": "moe", "router": {"experts": experts, "top": top}, "expert": {"ff": ff}}


def make_config(layers, *, streams, vocab, width, loop=None, bigram=(61, 31, 7), eps=1e-5):
    config = {"architecture": "Sugosun", "vocab": vocab, "width": width, "streams": streams, "norm": {"eps": eps}, "layers": layers}
    if bigram:
        config["embedding"] = {"bigram": dict(zip(("buckets", "mul_prev", "mul_cur"), bigram))}
    if loop:
        config["loop"] = dict(zip(("start", "stop", "times"), loop))
    return config


# Sizes that differ from layer to layer, values that are 1, rows and columns that are no multiple of anything.
CONFIGS = {
    "mixed": make_config([latent_layer(6, 24, 16, 40, 56, 48, 21, mlp=moe(9, 3, 40)),
                          lightning_layer([0.3, 0.7, 0.9, 0.97, 1.0], 24, 40, mlp=dense(88, 1.5)),
                          latent_layer(3, 32, 8, 16, 24, 36, 0, base=1e4),       # sizes the prompt kernel takes over a row it does not
                          lightning_layer([0.95, 0.5], 8, 16, mlp=moe(5, 1, 24))],
                         streams=3, vocab=131, width=96, loop=(1, 3, 2)),
    "odd": make_config([latent_layer(5, 9, 6, 7, 13, 11, 1, mlp=dense(33, 0.8)),
                        lightning_layer([0.8, 0.99, 0.0], 10, 7, mlp=moe(3, 3, 17)),
                        latent_layer(1, 5, 2, 3, 6, 4, 35, base=10.0, mlp=moe(7, 2, 9))],
                       streams=1, vocab=83, width=52, loop=(0, 3, 2), bigram=(5, 1, 3), eps=1e-3),
    "wide": make_config([latent_layer(4, 128, 64, 128, 96, 512, 70, base=1e4, mlp=moe(16, 2, 64)),
                         lightning_layer([0.9, 0.995], 128, 128, mlp=dense(200, 2.0)),
                         latent_layer(20, 64, 24, 80, 64, 72, 130, mlp=moe(40, 4, 72))],
                        streams=4, vocab=211, width=128, loop=(0, 2, 2)),
}


def random_weights(parameter_shapes, seed, dtype=torch.bfloat16, steady=False):
    """Weights at a scale that keeps every mechanism visible: attention scores spread over several units, norm weights away from
    their neutral value, mixing matrices away from the identity.

    `steady`: routing without close calls, for models whose activations are rounded.  The first coordinates of every embedding
    row hold a ladder of well separated values in an order of the token's own, no sublayer writes to them, and the routers
    read nothing else."""
    g = torch.Generator().manual_seed(seed)
    out = {}
    for name, shape in parameter_shapes.items():
        r = torch.randn(shape, generator=g)
        if name.endswith(("norm", "norm1", "norm2")):
            r = 1 + 0.2 * r
        elif name.endswith((".in", ".out")):
            r = 0.7 + 0.3 * r.abs()
        elif name.endswith(".mix"):
            r = 0.6 * torch.eye(shape[0]) + 0.15 * r.abs() + 0.05
        elif name.endswith("correction"):
            r = 0.05 * r
        elif name in ("embed", "bigram"):
            r = (1.0 if name == "embed" else 0.6) * r
        elif name.endswith(("mix.uq", "mix.uk")):
            r = 1.5 * r / shape[1] ** 0.5
        elif name.endswith("router"):
            r = 2.0 * r / shape[1] ** 0.5
        else:
            r = r / shape[-1] ** 0.5
        out[name] = r
    if steady:
        codes = max([shape[0] for name, shape in parameter_shapes.items() if name.endswith("router")], default=0)
        ladder = torch.linspace(-2.5, 2.5, max(codes, 1))
        for row in out["embed"]:
            row[:codes] = ladder[torch.randperm(codes, generator=g)]
        if "bigram" in out:
            out["bigram"][:, :codes] = 0
        for name in out:
            if name.endswith(("mix.o", ".down")):
                out[name][:codes] = 0
            elif name.endswith(("norm1", "norm2", "embed.norm")):
                out[name][:codes] = 1
            elif name.endswith("router"):
                experts = out[name].shape[0]
                out[name].zero_()
                out[name][torch.arange(experts), torch.randperm(codes, generator=g)[:experts]] = 3.0
            elif name.endswith("correction"):
                out[name].zero_()
                out[name][1 % len(out[name])] = 2.0          # always chosen, weighted without it
    return {name: r.to(dtype) for name, r in out.items()}
