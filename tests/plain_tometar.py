"""A plain, slow float64 statement of the Tometar decoder, one function per mechanism.

Used only by the tests; shares no code with the library. A sequence is evaluated token by token with everything that
earlier tokens left behind kept in a `State`, so prompts, portions and decoding are the same computation here.
Weights are a dict name -> float array (linear weights [out, in]).

`act` and `cache` (identity by default) are applied where a 16-bit model rounds: `act` to the operands of matrix products and
to what a convolution hands on, `cache` to the rows an attention layer keeps.
"""
import json
import os
import struct

import numpy as np


def same(v):
    return v


# ---- mechanisms ---------------------------------------------------------------------------------------------------
def rms_norm(x, w, eps):
    return x / np.sqrt(np.mean(x * x) + eps) * w


def silu(z):
    return z / (1.0 + np.exp(-z))


def sigmoid(z):
    return 1.0 / (1.0 + np.exp(-z))


def softplus(z):
    return np.logaddexp(0.0, z)


def rotate_half(v, pos, base, dims):
    """Rotate the first `dims` entries of the last axis: entry i with entry i + dims/2 by pos * base^(-2 i / dims)."""
    half = dims // 2
    a = pos * float(base) ** (-2.0 * np.arange(half) / dims)
    c, s = np.cos(a), np.sin(a)
    out = v.copy()
    lo, hi = v[..., :half], v[..., half:dims]
    out[..., :half] = lo * c - hi * s
    out[..., half:dims] = hi * c + lo * s
    return out


def softmax(s):
    e = np.exp(s - s.max())
    return e / e.sum()


def hyper_read(streams, w_in):
    return w_in @ streams


def hyper_write(streams, y, w_mix, w_out):
    """new[t] = sum_s mix[s, t] old[s] + out[t] y"""
    return w_mix.T @ streams + np.outer(w_out, y)


def latent_attention(h, W, pre, spec, eps, pos, past, act=same, cache=same):
    """`past` holds (latent, rotated key) of every earlier position; this position's pair is appended."""
    H, d, r, dv, R = spec["heads"], spec["dim"], spec["rot_dim"], spec["vdim"], spec["kv_rank"]
    base, dims = spec["rot"]["base"], spec["rot"]["dims"]
    q = (W[pre + "q"] @ h).reshape(H, d + r)
    qu, qr = act(q[:, :d]), act(rotate_half(q[:, d:], pos, base, dims))
    kv = W[pre + "dkv"] @ h
    past.append((cache(rms_norm(kv[:R], W[pre + "dkv.norm"], eps)), cache(rotate_half(kv[R:], pos, base, dims))))
    lo = max(0, pos - spec["mask"]["size"] + 1)
    C = np.stack([c for c, _ in past[lo:]])
    Kr = np.stack([k for _, k in past[lo:]])
    Ku = act(C @ W[pre + "uk"].T).reshape(-1, H, d)
    V = act(C @ W[pre + "uv"].T).reshape(-1, H, dv)
    out = np.empty((H, dv))
    for i in range(H):
        s = (Ku[:, i] @ qu[i] + Kr @ qr[i]) * spec["scale"]
        out[i] = softmax(s) @ V[:, i]
    o = out.reshape(-1) * sigmoid(W[pre + "g"] @ h)
    return W[pre + "o"] @ act(o)


def short_conv(history, w, b):
    """Causal convolution per channel over `history` (oldest first, the current input last) and silu."""
    taps = w.shape[1]
    acc = b.copy()
    for j in range(taps):
        back = taps - 1 - j
        if back < len(history):
            acc = acc + w[:, j] * history[len(history) - 1 - back]
    return silu(acc)


def ssm_step(S, x, B, C, dt, A_log, D, groups):
    """S [heads, N, V], x [heads, V], B and C [groups, N], dt [heads] -> (new S, y [heads, V])"""
    heads = x.shape[0]
    y = np.empty_like(x)
    S = S.copy()
    for h in range(heads):
        g = h // (heads // groups)
        S[h] = np.exp(-np.exp(A_log[h]) * dt[h]) * S[h] + dt[h] * np.outer(B[g], x[h])
        y[h] = C[g] @ S[h] + D[h] * x[h]
    return S, y


def grouped_norm(y, w, parts, eps):
    g = y.reshape(parts, -1)
    g = g / np.sqrt(np.mean(g * g, axis=1, keepdims=True) + eps)
    return g.reshape(-1) * w


def mamba2(h, W, pre, spec, eps, st, act=same):
    heads, V, N, G = spec["heads"], spec["vdim"], spec["state"], spec["groups"]
    inner = heads * V
    u = W[pre + "in"] @ h
    z, xbc, dt = u[:inner], u[inner:2 * inner + 2 * G * N], u[2 * inner + 2 * G * N:]
    st["conv"].append(xbc)
    c = act(short_conv(st["conv"], W[pre + "conv"], W[pre + "conv.b"]))
    st["conv"] = st["conv"][-W[pre + "conv"].shape[1]:]
    x, B, C = c[:inner].reshape(heads, V), c[inner:inner + G * N].reshape(G, N), c[inner + G * N:].reshape(G, N)
    dt = softplus(dt + W[pre + "dt_bias"])
    st["S"], y = ssm_step(st["S"], x, B, C, dt, W[pre + "A_log"], W[pre + "D"], G)
    y = grouped_norm(y.reshape(-1) * silu(z), W[pre + "norm"], spec["norm_groups"], eps)
    return W[pre + "o"] @ act(y)


def feed_forward(h, W, pre, act=same):
    gate = W[pre + "gate"] @ h + W[pre + "gate.b"]
    up = W[pre + "up"] @ h + W[pre + "up.b"]
    return W[pre + "down"] @ act(np.maximum(gate, 0.0) * up) + W[pre + "down.b"]


# ---- the model ----------------------------------------------------------------------------------------------------
class State:
    def __init__(self, cfg):
        self.pos = 0
        self.layers = []
        for L in cfg["layers"]:
            m = L["mixer"]
            if L["type"] == "latent_attention":
                self.layers.append([])
            else:
                self.layers.append({"S": np.zeros((m["heads"], m["state"], m["vdim"])), "conv": []})


def step(cfg, W, st, token, taps=None, act=same, cache=same):
    """Logits of one token; `taps` (a list) receives the sum of the streams after every layer."""
    eps, n = cfg["norm"]["eps"], cfg["streams"]
    X = np.tile(W["embed"][int(token)].astype(np.float64), (n, 1))
    for i, L in enumerate(cfg["layers"]):
        p = f"l{i}."
        h = act(rms_norm(hyper_read(X, W[p + "hc1.in"]), W[p + "norm1"], eps))
        if L["type"] == "latent_attention":
            y = latent_attention(h, W, p + "mix.", L["mixer"], eps, st.pos, st.layers[i], act, cache)
        else:
            y = mamba2(h, W, p + "mix.", L["mixer"], eps, st.layers[i], act)
        X = hyper_write(X, y, W[p + "hc1.mix"], W[p + "hc1.out"])
        if L["mlp"] is not None:
            h = act(rms_norm(hyper_read(X, W[p + "hc2.in"]), W[p + "norm2"], eps))
            X = hyper_write(X, feed_forward(h, W, p + "mlp.", act), W[p + "hc2.mix"], W[p + "hc2.out"])
        if taps is not None:
            taps.append(X.sum(0))
    st.pos += 1
    return W["head"] @ act(rms_norm(X.sum(0), W["final.norm"], eps))


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


# ---- model folders (config.json + model.safetensors) -----------------------------------------------------------------
def read_folder(path):
    with open(os.path.join(path, "config.json")) as f:
        cfg = json.load(f)
    with open(os.path.join(path, "model.safetensors"), "rb") as f:
        raw = f.read()
    n = struct.unpack("<Q", raw[:8])[0]
    W = {}
    for name, t in json.loads(raw[8:8 + n]).items():
        if name == "__metadata__":
            continue
        a, b = t["data_offsets"]
        buf = raw[8 + n + a:8 + n + b]
        if t["dtype"] == "BF16":
            v = (np.frombuffer(buf, "<u2").astype(np.uint32) << 16).view(np.float32)
        elif t["dtype"] == "F32":
            v = np.frombuffer(buf, "<f4")
        else:
            v = np.frombuffer(buf, {"I32": "<i4", "F16": "<f2"}[t["dtype"]])
        W[name] = v.reshape(t["shape"]).astype(np.float64)
    return cfg, W
