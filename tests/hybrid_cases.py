"""Small random models and configurations for the hybrid decoder's tests."""

from __future__ import annotations

import json
import struct

import torch

NAMES = {torch.bfloat16: "BF16", torch.float32: "F32", torch.int32: "I32"}


def attention_layer(heads, kv_heads, dim, vdim, *, scale=None, temp=(0.4, 24), kv_from=None, ff=72):
    mixer = {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "scale": scale or dim ** -0.5}
    if temp is not None:
        mixer["q_temp"] = {"coef": temp[0], "every": temp[1]}
    if kv_from is not None:
        mixer["kv_from"] = kv_from
    return {"type": "attention", "mixer": mixer, "mlp": {"kind": "dense", "ff": ff} if ff else None}


def mamba_layer(heads, vdim, state, groups, *, conv=4, norm_groups=1, ff=72):
    return {"type": "mamba2", "mixer": {"heads": heads, "vdim": vdim, "state": state, "groups": groups, "conv": conv,
                                        "norm_groups": norm_groups},
            "mlp": {"kind": "dense", "ff": ff} if ff else None}


def make_config(layers, *, vocab=157, width=96, eps=1e-5):
    return {"architecture": "Sobipel", "vocab": vocab, "width": width, "norm": {"eps": eps}, "layers": layers}


# Sizes that differ from layer to layer, values that are 1, rows and columns that are no multiple of anything.
CONFIGS = {
    "mixed": make_config([attention_layer(6, 2, 24, 40, temp=(0.5, 16)),
                          mamba_layer(6, 16, 20, 3, norm_groups=2, ff=None),
                          attention_layer(6, 2, 24, 40, temp=None, kv_from=0, ff=56),
                          mamba_layer(4, 24, 32, 1, conv=3, norm_groups=4),
                          attention_layer(3, 1, 16, 8, scale=0.4, ff=None)]),
    "odd": make_config([mamba_layer(3, 10, 12, 3, conv=2, norm_groups=3, ff=50),
                        attention_layer(5, 5, 20, 12, temp=(0.7, 5), ff=33),
                        mamba_layer(2, 7, 9, 2, conv=1, norm_groups=1),
                        attention_layer(5, 5, 20, 12, kv_from=1)], vocab=83, width=52),
    "wide": make_config([attention_layer(4, 2, 128, 128, temp=(0.3, 64)),
                         mamba_layer(4, 64, 128, 2, norm_groups=2),
                         attention_layer(6, 3, 64, 64, temp=(0.2, 40), ff=None),
                         attention_layer(4, 2, 128, 128, kv_from=0, temp=(0.2, 33)),
                         mamba_layer(2, 80, 144, 1, conv=5)], vocab=211, width=128),
}


def random_weights(parameter_shapes, seed, dtype=torch.bfloat16):
    """Weights at a scale that keeps every mechanism visible: attention scores spread over several units, decays from
    nearly 0 to nearly 1, norm weights away from their neutral value."""
    g = torch.Generator().manual_seed(seed)
    out = {}
    for name, shape in parameter_shapes.items():
        r = torch.randn(shape, generator=g)
        if name.endswith(("norm1", "final.norm")):
            r = 0.2 * r
        elif name.endswith("mix.norm"):
            r = 1 + 0.2 * r
        elif name.endswith("A_log"):
            r = torch.linspace(-3.0, 1.5, shape[0]) + 0.1 * r
        elif name.endswith("dt_bias"):
            r = -1.0 + r
        elif name.endswith("mix.D"):
            r = 0.5 + 0.5 * r
        elif name.endswith("mix.conv"):
            r = 0.6 * r
        elif name.endswith("conv.b"):
            r = 0.2 * r
        elif name == "embed":
            pass
        elif name.endswith(("mix.q", "mix.k")):
            r = 1.5 * r / shape[1] ** 0.5
        else:
            r = r / shape[-1] ** 0.5
        out[name] = r.to(dtype)
    return out


def write_safetensors(path, tensors):
    header, at, data = {}, 0, []
    for name, t in tensors.items():
        raw = t.contiguous().view(torch.uint8).numpy().tobytes()
        header[name] = {"dtype": NAMES[t.dtype], "shape": list(t.shape), "data_offsets": [at, at + len(raw)]}
        data.append(raw)
        at += len(raw)
    text = json.dumps(header).encode()
    path.write_bytes(struct.pack("<Q", len(text)) + text + b"".join(data))


def write_model(folder, config, tensors):
    folder.mkdir(parents=True, exist_ok=True)
    (folder / "config.json").write_text(json.dumps(config))
    write_safetensors(folder / "model.safetensors", tensors)


def prompt(seed, length, vocab):
    return torch.randint(0, vocab, (length,), generator=torch.Generator().manual_seed(seed)).tolist()
