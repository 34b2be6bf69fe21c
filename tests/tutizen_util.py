"""Small random Tutizen models for the tests: configurations, weights that are exact in bfloat16, token sequences."""
import numpy as np

from . import plain_tutizen as P
from .tometar_util import bf16_bits, bf16_round, error, tensors, write_folder  # noqa: F401


def attn(heads, kv_heads, dim, vdim, kv_from=None, scale=None):
    m = {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "scale": float(dim ** -0.5) if scale is None else scale}
    return m if kv_from is None else dict(m, kv_from=kv_from)


def dense(ff, limit=1.5):
    return {"kind": "dense", "ff": ff, "limit": limit}


def moe(experts, top, ff, shared, groups=1, keep=1, scale=1.7, limit=0.9, shared_limit=1.3):
    return {"kind": "moe", "expert": {"ff": ff, "limit": limit}, "shared": {"ff": shared, "limit": shared_limit},
            "router": {"experts": experts, "top": top, "scale": scale, "groups": {"count": groups, "keep": keep}}}


def layer(mixer, mlp=None):
    return {"type": "attention", "mixer": mixer, "mlp": mlp}


def config(layers, width, vocab, mult=0.6, eps=1e-5):
    return {"architecture": "Tutizen", "layers": layers, "norm": {"eps": eps}, "residual_mult": mult, "vocab": vocab, "width": width}


# name -> configuration; none of the sizes is meant to be convenient
CONFIGS = {
    # every size a multiple of the vector width; keys borrowed from a neighbour and from far below; unequal head sizes
    "even": config([layer(attn(6, 2, 32, 48), dense(136)), layer(attn(6, 2, 32, 48, kv_from=0), moe(12, 3, 40, 56, 3, 2)),
                    layer(attn(4, 4, 64, 32, scale=0.05)), layer(attn(6, 2, 32, 48, kv_from=0, scale=0.4), moe(8, 2, 64, 32))], 112, 200),
    # nothing is: the any-size kernels
    "odd": config([layer(attn(3, 1, 21, 13), dense(37)), layer(attn(5, 5, 9, 30), moe(6, 2, 11, 9, 2, 1)),
                   layer(attn(3, 1, 21, 13, kv_from=0), moe(9, 4, 7, 23, 3, 3))], 51, 77, mult=1.0, eps=1e-6),
    # values that are one: one head, one expert, groups of one expert, one kept group
    "ones": config([layer(attn(1, 1, 16, 24), moe(1, 1, 24, 8)), layer(attn(1, 1, 16, 24, kv_from=0), moe(4, 2, 16, 8, 4, 2)),
                    layer(attn(2, 1, 8, 8), dense(40, 0.7))], 40, 64, mult=0.25),
    # wider heads and many experts
    "wide": config([layer(attn(8, 2, 128, 128), moe(64, 6, 24, 40, 8, 3)), layer(attn(4, 1, 72, 104), dense(264)),
                    layer(attn(4, 1, 72, 104, kv_from=1), moe(48, 8, 16, 16, 6, 2, scale=0.8))], 160, 320),
}


def weights(cfg, seed=0, steady=True):
    """name -> float32 array holding bfloat16 values. steady: the routers read a quarter of the coordinates that no sublayer
    writes, so that which experts a token gets follows from the token and its position alone (see tokens())."""
    from nfai_b200 import config_tensors
    rng = np.random.default_rng(seed)
    W = {}
    own = cfg["width"] // 4
    for name, shape in config_tensors(cfg).items():
        n = rng.standard_normal(shape)
        last = name.split(".")[-1]
        if last in ("norm", "norm1", "norm2"):
            a = 1.0 + 0.2 * n
        elif last == "b":
            a = 0.3 * n
        elif last == "correction":
            a = 0.2 * n
        elif name == "embed":
            a = n
        elif last == "router":
            a = n * 1.5 / np.sqrt(own if steady else shape[1])
            if steady:
                a[:, own:] = 0
        else:
            a = n / np.sqrt(shape[-1])
        if steady and (last in ("o", "down") or name.endswith("o.b")):
            a[:own] = 0
        W[name] = bf16_round(np.asarray(a, np.float32)).reshape(shape)
    return W


def margin(z, correction, router):
    """How far the nearest other choice of experts or groups is, in choice score."""
    c = P.sigmoid(z) + correction
    n, keep, top = router["groups"]["count"], router["groups"]["keep"], router["top"]
    two = np.sort(c.reshape(n, -1), axis=1)[:, -2:].sum(1)
    order = np.argsort(-two)
    best = np.inf if keep == n else two[order[keep - 1]] - two[order[keep]]
    allowed = np.sort(c.reshape(n, -1)[order[:keep]].ravel())[::-1]
    return min(best, np.inf if top == len(allowed) else allowed[top - 1] - allowed[top])


def tokens(cfg, W, n, seed=0, least=0.02):
    """n random tokens whose experts are no close call in any layer, so that 16-bit rounding does not change them."""
    rng = np.random.default_rng(seed)
    E = W["embed"].astype(np.float64)
    routed = [(f"l{i}.mlp.", L["mlp"]["router"]) for i, L in enumerate(cfg["layers"]) if L["mlp"] and L["mlp"]["kind"] == "moe"]
    out = []
    for p in range(n):
        x = P.position_vector(p, cfg["width"])
        for t in rng.permutation(cfg["vocab"]):
            if all(margin(W[k + "router"].astype(np.float64) @ (E[t] + x), W[k + "correction"].astype(np.float64), r) > least for k, r in routed):
                out.append(int(t))
                break
        else:
            raise ValueError("no token with a clear choice of experts")
    return out
