"""Small random Tometar models for the tests: configurations, weights that are exact in bfloat16, model folders."""
import json
import os
import struct

import numpy as np

from nfai_b200 import _lib


def latent(heads, dim, rot, vdim, rank, window, scale=None, base=10000.0):
    return {"heads": heads, "dim": dim, "rot_dim": rot, "vdim": vdim, "kv_rank": rank, "mask": {"size": window},
            "rot": {"base": base, "dims": rot}, "scale": scale if scale is not None else float((dim + rot) ** -0.5)}


def ssm(heads, vdim, state, groups, taps, norm_groups):
    return {"heads": heads, "vdim": vdim, "state": state, "groups": groups, "conv": taps, "norm_groups": norm_groups}


def layer(mixer, ff=None):
    return {"type": "latent_attention" if "kv_rank" in mixer else "mamba2", "mixer": mixer,
            "mlp": {"kind": "dense", "ff": ff} if ff else None}


def config(layers, width, vocab, streams, eps=1e-5):
    return {"architecture": "Tometar", "layers": layers, "norm": {"eps": eps}, "streams": streams, "vocab": vocab, "width": width}


# name -> configuration; none of the sizes is meant to be convenient
CONFIGS = {
    # every size a multiple of the vector width: tensor-core products, vector copies
    "even": config([layer(latent(4, 32, 16, 48, 64, 40), 144), layer(ssm(6, 16, 32, 2, 4, 3)), layer(ssm(4, 40, 24, 1, 3, 1), 96),
                    layer(latent(2, 48, 32, 32, 96, 17))], 112, 200, 3),
    # nothing is: the any-size kernels
    "odd": config([layer(ssm(5, 11, 19, 5, 2, 5), 37), layer(latent(3, 21, 6, 13, 35, 29), 41), layer(latent(1, 9, 2, 7, 11, 90, base=500.0)),
                   layer(ssm(3, 21, 50, 1, 4, 7))], 51, 77, 2, eps=1e-6),
    # values that are one: one stream, one tap, one head, a window of the token itself
    "ones": config([layer(latent(1, 16, 8, 24, 24, 1), 40), layer(ssm(1, 24, 8, 1, 1, 1), 24), layer(latent(2, 24, 8, 16, 40, 2))],
                   40, 64, 1),
    # wider heads and states
    "wide": config([layer(latent(3, 72, 56, 104, 160, 70), 264), layer(ssm(4, 72, 136, 2, 5, 4)), layer(ssm(2, 128, 64, 2, 4, 2))],
                   192, 320, 6),
}


def bf16_bits(a):
    """Round to nearest even bfloat16, as uint16 bits."""
    b = np.ascontiguousarray(a, np.float32).view(np.uint32)
    return ((b + 0x7FFF + ((b >> 16) & 1)) >> 16).astype(np.uint16)


def bf16_round(a):
    return (bf16_bits(a).astype(np.uint32) << 16).view(np.float32)


def weights(cfg, seed=0):
    """name -> float32 array holding bfloat16 values."""
    from nfai_b200 import config_tensors
    rng = np.random.default_rng(seed)
    W = {}
    for name, shape in config_tensors(cfg).items():
        n = rng.standard_normal(shape)
        last = name.split(".")[-1]
        if last in ("norm", "norm1", "norm2"):
            a = 1.0 + 0.2 * n
        elif last == "b" or last == "dt_bias":
            a = 0.3 * n
        elif last == "A_log":
            a = rng.uniform(-2.5, 1.0, shape)
        elif last == "D":
            a = 1.0 + 0.3 * n
        elif last == "conv":
            a = n / np.sqrt(shape[1])
        elif ".hc" in name and last == "in":
            a = 1.0 / shape[0] + 0.2 * n
        elif ".hc" in name and last == "out":
            a = 0.8 + 0.3 * n
        elif ".hc" in name and last == "mix":
            a = 0.9 * np.eye(shape[0]) + 0.1 * n
        elif name == "embed":
            a = n
        else:
            a = n / np.sqrt(shape[-1])
        W[name] = bf16_round(a.astype(np.float32)).reshape(shape)
    return W


def tensors(W):
    """(name, bfloat16 bits, code) triples for PlannedModel.from_tensors."""
    return [(n, bf16_bits(a), _lib.BF16) for n, a in W.items()]


def write_folder(path, cfg, W):
    os.makedirs(path, exist_ok=True)
    with open(os.path.join(path, "config.json"), "w") as f:
        json.dump(cfg, f)
    head, data = {}, b""
    for name, a in W.items():
        raw = bf16_bits(a).astype("<u2").tobytes()
        head[name] = {"dtype": "BF16", "shape": list(a.shape), "data_offsets": [len(data), len(data) + len(raw)]}
        data += raw
    h = json.dumps(head).encode()
    with open(os.path.join(path, "model.safetensors"), "wb") as f:
        f.write(struct.pack("<Q", len(h)) + h + data)
    return str(path)


def error(got, want):
    """Root mean square of the difference with its mean taken off, over that of the wanted rows; the worst row."""
    got, want = np.atleast_2d(np.asarray(got, np.float64)), np.atleast_2d(np.asarray(want, np.float64))
    d = got - want
    d = d - d.mean(axis=1, keepdims=True)
    w = want - want.mean(axis=1, keepdims=True)
    return float(np.sqrt((d * d).mean(axis=1)).max() / np.sqrt((w * w).mean()))
