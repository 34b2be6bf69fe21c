"""A plain, slow float64 statement of the Tutizen decoder, one function per mechanism.

Used only by the tests; shares no code with the library. A sequence is evaluated token by token with everything that
earlier tokens left behind kept in a `State`, so prompts, portions and decoding are the same computation here.
Weights are a dict name -> float array (linear weights [out, in]).

`act` and `cache` (identity by default) are applied where a 16-bit model rounds: `act` to the operands of matrix products,
`cache` to the rows an attention layer keeps.
"""
import numpy as np


def same(v):
    return v


# ---- mechanisms ---------------------------------------------------------------------------------------------------
def unit_rms(x, eps):
    """x over its root mean square along the last axis."""
    return x / np.sqrt(np.mean(x * x, axis=-1, keepdims=True) + eps)


def sigmoid(z):
    return 1.0 / (1.0 + np.exp(-z))


def position_vector(p, width):
    i = np.arange(width)
    a = p * 10000.0 ** (-2.0 * (i // 2) / width)
    return np.where(i % 2 == 0, np.sin(a), np.cos(a))


def slopes(heads):
    return 2.0 ** (-8.0 * (np.arange(heads) + 1) / heads)


def softmax(s):
    e = np.exp(s - s.max())
    return e / e.sum()


def attend(q, K, V, scale, slope, pos):
    """One head: query at `pos` over the keys and values of positions 0 .. pos."""
    return softmax(K @ q * scale - slope * (pos - np.arange(len(K)))) @ V


def attention(h, W, pre, spec, eps, pos, past, act=same, cache=same):
    """`past` holds the (key, value) heads of every earlier position. A layer with keys of its own appends this position's
    pair; one that borrows finds it there already."""
    H, G, d, dv = spec["heads"], spec["kv_heads"], spec["dim"], spec["vdim"]
    q = act(unit_rms((W[pre + "q"] @ h + W[pre + "q.b"]).reshape(H, d), eps))
    if spec.get("kv_from") is None:
        k = unit_rms((W[pre + "k"] @ h + W[pre + "k.b"]).reshape(G, d), eps)
        v = unit_rms((W[pre + "v"] @ h + W[pre + "v.b"]).reshape(G, dv), eps)
        past.append((cache(k), cache(v)))
    K, V = np.stack([k for k, _ in past]), np.stack([v for _, v in past])
    m = slopes(H)
    o = np.stack([attend(q[i], K[:, i // (H // G)], V[:, i // (H // G)], spec["scale"], m[i], pos) for i in range(H)])
    o = o * sigmoid(W[pre + "g"] @ h)[:, None]
    return W[pre + "o"] @ act(o.reshape(-1)) + W[pre + "o.b"]


def clamped_glu(gate, up, limit):
    g, u = np.minimum(gate, limit), np.clip(up, -limit, limit)
    return g * sigmoid(1.702 * g) * (u + 1.0)


def feed_forward(h, W, pre, limit, act=same):
    return W[pre + "down"] @ act(clamped_glu(W[pre + "gate"] @ h, W[pre + "up"] @ h, limit))


def route(z, correction, router):
    """Router logits -> (chosen experts, their weights)."""
    s = sigmoid(z)
    c = s + correction
    n, keep = router["groups"]["count"], router["groups"]["keep"]
    size = len(c) // n
    groups = [sorted(range(g * size, (g + 1) * size), key=lambda e: -c[e]) for g in range(n)]
    best = sorted(range(n), key=lambda g: -sum(c[e] for e in groups[g][:2]))[:keep]
    allowed = [e for e in range(len(c)) if e // size in best]
    chosen = sorted(allowed, key=lambda e: -c[e])[:router["top"]]
    w = s[chosen]
    return chosen, w / (w.sum() + 1e-20) * router["scale"]


def experts(h, W, pre, spec, act=same):
    chosen, w = route(W[pre + "router"] @ h, W[pre + "correction"], spec["router"])
    y = sum(wi * feed_forward(h, W, f"{pre}e{e}.", spec["expert"]["limit"], act) for e, wi in zip(chosen, w))
    shared = feed_forward(h, W, pre + "shared.", spec["shared"]["limit"], act)
    return y + sigmoid(W[pre + "shared.sg"] @ h) * shared


# ---- the model ----------------------------------------------------------------------------------------------------
class State:
    def __init__(self, cfg):
        self.pos = 0
        self.past = [[] for _ in cfg["layers"]]


def step(cfg, W, st, token, taps=None, act=same, cache=same):
    """Logits of one token; `taps` (a list) receives the residual after every layer."""
    eps, m = cfg["norm"]["eps"], cfg["residual_mult"]
    x = W["embed"][int(token)].astype(np.float64) + position_vector(st.pos, cfg["width"])
    for i, L in enumerate(cfg["layers"]):
        p = f"l{i}."
        src = L["mixer"].get("kv_from")
        y = attention(act(x), W, p + "mix.", L["mixer"], eps, st.pos, st.past[i if src is None else src], act, cache)
        x = x + m * unit_rms(y, eps) * W[p + "norm1"]
        if L["mlp"] is not None:
            h = act(x)
            y = feed_forward(h, W, p + "mlp.", L["mlp"]["limit"], act) if L["mlp"]["kind"] == "dense" else \
                experts(h, W, p + "mlp.", L["mlp"], act)
            x = x + m * unit_rms(y, eps) * W[p + "norm2"]
        if taps is not None:
            taps.append(x)
    st.pos += 1
    return W["head"] @ act(unit_rms(x, eps) * W["final.norm"])


def forward(cfg, W, tokens, st=None, taps=None, act=same, cache=same):
    """[len(tokens), vocab] logits; `taps` receives one list of layer outputs per token."""
    st = st or State(cfg)
    out = []
    for t in tokens:
        tp = [] if taps is not None else None
        out.append(step(cfg, W, st, t, tp, act, cache))
        if taps is not None:
            taps.append(tp)
    return np.array(out)
