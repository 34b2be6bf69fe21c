"""Tutizen models on a GPU against the plain float64 statement (tests/plain_tutizen.py): every mechanism, prompts, portions,
decoding, reuse, far keys, generation. float32 models are held to float32 accuracy, bfloat16 models to what rounding
activations to bfloat16 costs."""
import json
import os
import subprocess
import sys

import numpy as np
import pytest

from nfai_b200 import ModelOptions, NfaiError, PlannedModel, _lib, trace, try_create

from . import plain_tutizen as P
from . import tutizen_util as U

pytestmark = pytest.mark.gpu
torch = pytest.importorskip("torch")

TOL = {"f32": 2e-5, "bf16": 4e-2}
CTX = 320
_cache = {}


def bf16(v):
    return U.bf16_round(np.asarray(v, np.float32)).astype(np.float64)


def to64(W):
    return {k: v.astype(np.float64) for k, v in W.items()}


def plain(name, n=260, seed=0):
    """(config, weights, tokens, logits [n][V], layer outputs [n][L][H]) of a named configuration, computed once."""
    key = (name, n, seed)
    if key not in _cache:
        cfg = U.CONFIGS[name]
        W = U.weights(cfg, seed)
        toks = U.tokens(cfg, W, n, seed + 100)
        taps = []
        logits = P.forward(cfg, to64(W), toks, taps=taps)
        _cache[key] = (cfg, W, toks, logits, np.array(taps))
    return _cache[key]


def build(ctx, cfg, W, dtype, size=CTX):
    return PlannedModel.from_tensors(ctx, cfg, U.tensors(W), size, dtype)


@pytest.fixture(params=[(n, d) for n in U.CONFIGS for d in ("f32", "bf16")], ids=lambda p: f"{p[0]}-{p[1]}")
def case(request, cuda_ctx):
    name, dtype = request.param
    m = build(cuda_ctx, U.CONFIGS[name], plain(name)[1], dtype)
    yield (m, dtype) + plain(name)
    m.Dispose()


def test_whole_prompt(case):
    m, dtype, cfg, W, toks, want, taps = case
    places = sorted(set(range(0, len(toks), 3)) | {len(toks) - 1})
    assert U.error(m.forward(toks, places), want[places]) < TOL[dtype]
    for l in range(m.L):
        assert U.error(m.read_hidden(l), taps[-1, l]) < TOL[dtype]
    assert m.position == len(toks)


def test_token_by_token(case):
    m, dtype, cfg, W, toks, want, taps = case
    n = 110
    got = [m.decode(t)[0] for t in toks[:n]]
    assert U.error(got, want[:n]) < TOL[dtype]
    for l in range(m.L):
        assert U.error(m.read_hidden(l), taps[n - 1, l]) < TOL[dtype]


def test_portions(case):
    """Cut anywhere: portions below the batched path's minimum, around the kernels' tiles, and single tokens in between."""
    m, dtype, cfg, W, toks, want, _ = case
    for sizes in ([2, 3, 1, 8, 9, 7, 16, 31, 1, 33, 2, 64, 15], [129, 2, 1], [37, 37, 2, 5], [2]):
        m.reset()
        got, at, i = [], 0, 0
        end = 60 if sizes == [2] else len(toks)
        while at < end:
            n = min(sizes[i % len(sizes)], end - at)
            got += list(m.forward(toks[at:at + n], range(n)))
            at, i = at + n, i + 1
        assert U.error(got, want[:end]) < TOL[dtype], sizes


def test_prompt_then_decoding(case):
    m, dtype, cfg, W, toks, want, _ = case
    for cut in (1, 2, 33, 200):
        m.reset()
        logits, am = m.prefill(toks[:cut])
        assert U.error(logits, want[cut - 1]) < TOL[dtype] and am == int(np.argmax(logits))
        got = [m.decode(t)[0] for t in toks[cut:cut + 45]]
        assert U.error(got, want[cut:cut + 45]) < TOL[dtype]


def test_reuse_leaves_no_trace(case):
    """A sequence gives the same bits whatever ran before it: from a reset, from a snapshot, from an earlier position."""
    m, dtype, cfg, W, toks, want, _ = case
    run = lambda: np.vstack([m.forward(toks[:50], range(0, 50, 7)), [m.decode(t)[0] for t in toks[50:60]]])  # noqa: E731
    first = run()
    other = [(t * 7 + 3) % cfg["vocab"] for t in toks]
    m.reset()
    m.forward(other[:170])
    m.reset()
    assert np.array_equal(run(), first)
    snap = m.snapshot()
    a = np.array([m.decode(t)[0] for t in toks[60:70]])
    m.set_position(60)
    assert np.array_equal(np.array([m.decode(t)[0] for t in toks[60:70]]), a)
    m.reset()
    m.forward(other[:90])
    snap.restore()
    assert m.position == 60
    assert np.array_equal(np.array([m.decode(t)[0] for t in toks[60:70]]), a)
    snap.close()


def test_several_passes(cuda_ctx, monkeypatch):
    """A prompt longer than one pass of the batched path."""
    monkeypatch.setenv("NFAI_PREFILL_CHUNK", "48")
    for name in ("even", "odd"):
        cfg, W, toks, want, taps = plain(name)
        for dtype in ("f32", "bf16"):
            m = build(cuda_ctx, cfg, W, dtype)
            assert U.error(m.forward(toks, range(len(toks))), want) < TOL[dtype]
            assert U.error(m.read_hidden(m.L - 1), taps[-1, -1]) < TOL[dtype]
            m.Dispose()


def test_any_size_attention_on_bfloat16(tmp_path):
    """The any-size attention kernel on a bfloat16 model (the switch is read once per process)."""
    cfg, W, toks, want, _ = plain("wide")
    U.write_folder(tmp_path / "m", cfg, W)
    code = ("import sys, numpy as np; sys.path.insert(0, sys.argv[1]); from nfai_b200 import *; "
            "m = try_create(CudaContext(0), ModelOptions(ModelPath=sys.argv[2], KVCacheSize=320)); "
            "np.save(sys.argv[3], m.forward(eval(sys.argv[4]), range(0, 260, 5)))")
    root = os.path.dirname(os.path.dirname(os.path.abspath(__file__)))
    out = str(tmp_path / "o.npy")
    subprocess.run([sys.executable, "-c", code, root, str(tmp_path / "m"), out, str(toks)], check=True, timeout=120,
                   env=dict(os.environ, NFAI_PREFILL_ATTN="0"))
    assert U.error(np.load(out), want[::5]) < TOL["bf16"]


# ---- mechanisms alone -----------------------------------------------------------------------------------------------------
def alone(cuda_ctx, cfg, W, toks, dtype, size=None):
    """A prompt and token-by-token decoding. bfloat16 models are compared with the plain statement rounded where they round
    (prompts: operands and cache rows; decoding: cache rows only), so that the bounds stay close."""
    W64 = to64(W)
    m = build(cuda_ctx, cfg, W, dtype, size or len(toks))
    ref = P.forward(cfg, W64, toks, **(dict(act=bf16, cache=bf16) if dtype == "bf16" else {}))
    assert U.error(m.forward(toks, range(len(toks))), ref) < {"f32": 3e-5, "bf16": 2e-2}[dtype]
    m.reset()
    ref = P.forward(cfg, W64, toks, **(dict(cache=bf16) if dtype == "bf16" else {}))
    assert U.error([m.decode(t)[0] for t in toks], ref) < {"f32": 3e-5, "bf16": 2e-3}[dtype]
    m.Dispose()


@pytest.mark.parametrize("dtype", ["f32", "bf16"])
@pytest.mark.parametrize("mixer", [
    U.attn(5, 1, 24, 40), U.attn(12, 3, 64, 64), U.attn(2, 2, 130, 7), U.attn(8, 8, 128, 128, scale=0.3), U.attn(3, 3, 200, 256),
    U.attn(2, 1, 257, 33), U.attn(1, 1, 300, 512), U.attn(20, 4, 8, 64, scale=-0.2), U.attn(7, 7, 6, 3),
], ids=str)
def test_attention_alone(cuda_ctx, mixer, dtype):
    """Attention and the residual, with a layer on top that borrows the keys and values."""
    cfg = U.config([U.layer(mixer), U.layer(dict(mixer, kv_from=0, scale=0.7 * mixer["scale"]))], 64, 96)
    toks = np.random.default_rng(5).integers(0, 96, 150).tolist()
    alone(cuda_ctx, cfg, U.weights(cfg, 11), toks, dtype)


@pytest.mark.parametrize("dtype", ["f32", "bf16"])
def test_feed_forward_alone(cuda_ctx, dtype):
    """The attention's output matrix is zero (its bias stays): what is left are clamped feed-forwards and the residual. Values
    are large enough for all three clamps to act."""
    cfg = U.config([U.layer(U.attn(1, 1, 4, 8), U.dense(200, 0.8)), U.layer(U.attn(1, 1, 4, 8), U.dense(24, 3.0))], 72, 50, mult=1.3)
    W = U.weights(cfg, 2)
    for i in (0, 1):
        W[f"l{i}.mix.o"][:] = 0
        for part in ("gate", "up"):
            W[f"l{i}.mlp.{part}"] = U.bf16_round(W[f"l{i}.mlp.{part}"] * 2)
    alone(cuda_ctx, cfg, W, list(range(50)), dtype)


@pytest.mark.parametrize("dtype", ["f32", "bf16"])
@pytest.mark.parametrize("mlp", [
    U.moe(16, 4, 32, 64, 4, 2), U.moe(5, 5, 48, 16), U.moe(130, 3, 8, 8, 10, 1), U.moe(300, 32, 8, 24, 60, 20), U.moe(33, 7, 9, 5, 11, 4),
    U.moe(1024, 2, 8, 8, 64, 3), U.moe(2, 1, 136, 264), U.moe(40, 6, 72, 8, 40, 9),
], ids=str)
def test_experts_alone(cuda_ctx, mlp, dtype):
    """The attention's output matrix is zero. Corrections pull some choice scores below zero and some groups up."""
    cfg = U.config([U.layer(U.attn(1, 1, 4, 8), mlp)], 48, 120, mult=0.9)
    W = U.weights(cfg, 7)
    W["l0.mix.o"][:] = 0
    W["l0.mlp.correction"] = U.bf16_round(W["l0.mlp.correction"] * 3 - 0.4)
    alone(cuda_ctx, cfg, W, U.tokens(cfg, W, 140, 3, least=1e-3), dtype)


def test_experts_read_what_attention_writes(cuda_ctx):
    """Routers that read every coordinate (float32 only: their choices may be close)."""
    for name in ("even", "odd"):
        cfg = U.CONFIGS[name]
        W = U.weights(cfg, 21, steady=False)
        alone(cuda_ctx, cfg, W, np.random.default_rng(8).integers(0, cfg["vocab"], 90).tolist(), "f32")


@pytest.mark.parametrize("dtype", ["f32", "bf16"])
def test_all_tokens_to_the_same_experts(cuda_ctx, dtype):
    """Corrections that decide alone: a few experts get every token (several row tiles each), the others none."""
    cfg = U.config([U.layer(U.attn(1, 1, 8, 8), U.moe(24, 3, 40, 16, 4, 2))], 64, 60)
    W = U.weights(cfg, 3)
    W["l0.mlp.correction"][:] = 0
    W["l0.mlp.correction"][[0, 9, 10]] = 4
    alone(cuda_ctx, cfg, W, np.random.default_rng(1).integers(0, 60, 300).tolist(), dtype)


def test_positions_far_out(cuda_ctx):
    """The position vector at large positions: a token far out against the same token close by, keys left out."""
    cfg = U.config([U.layer(U.attn(1, 1, 4, 4))], 50, 30)
    W = U.weights(cfg, 1)
    W["l0.mix.o"][:] = 0
    W64 = to64(W)
    m = build(cuda_ctx, cfg, W, "f32", 20000)
    at = 0
    for p in (1, 777, 4096, 19990):
        m.forward([3] * (p - at))
        got, _ = m.decode(5)
        at = p + 1
        x = W64["embed"][5] + P.position_vector(p, 50)
        x = x + cfg["residual_mult"] * P.unit_rms(W64["l0.mix.o.b"], 1e-5) * W64["l0.norm1"]
        assert U.error(got, W64["head"] @ (P.unit_rms(x, 1e-5) * W64["final.norm"])) < 2e-5
    m.Dispose()


def test_cached_rows(cuda_ctx):
    """The cache holds normed keys and values, whichever path wrote them; a borrowing layer shows its source's."""
    cfg, W, toks, _, _ = plain("even")
    st = P.State(cfg)
    P.forward(cfg, to64(W), toks[:40], st)
    m = build(cuda_ctx, cfg, W, "f32")
    m.forward(toks[:30])
    for t in toks[30:40]:
        m.decode(t)
    for i, src in ((0, 0), (1, 0), (2, 2), (3, 0)):
        for pos in (0, 1, 29, 30, 39):
            k, v = m.read_kv(i, pos)
            assert np.abs(k - st.past[src][pos][0]).max() < 1e-4 and np.abs(v - st.past[src][pos][1]).max() < 1e-4
    m.Dispose()


# ---- far keys -------------------------------------------------------------------------------------------------------------
def needle_model(scale, heads=4, kv_heads=2, dim=16, vdim=24, seed=0):
    """One layer whose queries all point the same way and whose keys point there (the needle) or the other way (all other
    tokens), so that the needle outscores the rest by 2 * dim * scale wherever it lies; the distance bias decides how far it is
    seen by which head."""
    width, vocab = 64, 24
    cfg = U.config([U.layer(U.attn(heads, kv_heads, dim, vdim, scale=scale))], width, vocab, mult=2.0)
    W = U.weights(cfg, seed)
    rng = np.random.default_rng(seed + 1)
    u = rng.choice([-1.0, 1.0], dim)
    W["embed"] = U.bf16_round(W["embed"])
    W["embed"][:, -1] = -20.0
    W["embed"][0, -1] = 20.0  # token 0 is the needle (the position vector adds at most 1)
    W["l0.mix.q"][:] = 0
    W["l0.mix.q.b"] = U.bf16_round(np.tile(u, heads).astype(np.float32))
    W["l0.mix.k"][:] = 0
    W["l0.mix.k"][:, -1] = U.bf16_round(np.tile(u, kv_heads).astype(np.float32))
    W["l0.mix.k.b"][:] = 0
    W["l0.mix.v"][:, -1] = 0
    return cfg, W


@pytest.mark.parametrize("dtype", ["f32", "bf16"])
@pytest.mark.parametrize("ctx", [700, 4200], ids=["head-per-block", "heads-share"])
def test_far_keys(cuda_ctx, dtype, ctx):
    """The needle just behind the query, at the borders of tiles and splits, and as far back as there are tokens."""
    cfg, W = needle_model(1.0)
    W64 = to64(W)
    m = build(cuda_ctx, cfg, W, dtype, ctx)
    rng = np.random.default_rng(4)
    for pos in (40, 129, 511, 640):
        filler = rng.integers(1, 24, pos + 1).tolist()
        for back in (1, 31, 32, 33, 63, 64, 65, 127, 128, 129, 510, 511, 512, 513, 640):
            if back > pos:
                continue
            toks = list(filler)
            toks[pos - back] = 0
            st = P.State(cfg)
            h = [W64["embed"][t] + P.position_vector(p, 64) for p, t in enumerate(toks)]  # (one layer: every row is direct)
            for x in h[:-1]:
                st.past[0].append((P.unit_rms((W64["l0.mix.k"] @ x).reshape(2, 16), 1e-5),
                                   P.unit_rms((W64["l0.mix.v"] @ x + W64["l0.mix.v.b"]).reshape(2, 24), 1e-5)))
            st.pos = pos
            without = P.State(cfg)
            without.pos, without.past = pos, [list(st.past[0])]
            without.past[0][pos - back] = without.past[0][0 if back != pos else 1]
            ref = P.step(cfg, W64, st, toks[-1])
            seen = U.error(P.step(cfg, W64, without, toks[-1]), ref)
            assert seen > 0.05  # the test sees what it is about
            m.reset()
            assert U.error(m.forward(toks, [pos]), ref) < TOL[dtype], (pos, back, "prompt")
            for cut in (pos, max(1, pos - 1), max(1, pos - back), max(1, pos - back + 1)):
                m.reset()
                m.forward(toks[:cut])
                assert U.error(m.forward(toks[cut:], [pos - cut]), ref) < TOL[dtype], (pos, back, cut)
    m.Dispose()


@pytest.mark.parametrize("dtype", ["f32", "bf16"])
def test_keys_put_out_of_reach(cuda_ctx, dtype):
    """Small scores under steep biases: what the kernels may leave out must not show, what they may not must. Long enough for
    splits in decoding, and for the steepest heads to reach only a small part of the sequence."""
    cfg = U.config([U.layer(U.attn(8, 2, 16, 32, scale=0.02)), U.layer(U.attn(8, 2, 16, 32, scale=1.5, kv_from=0))], 48, 64)
    W = U.weights(cfg, 6)
    toks = np.random.default_rng(2).integers(0, 64, 900).tolist()
    W64, kw = to64(W), dict(cache=bf16) if dtype == "bf16" else {}
    st = P.State(cfg)
    ref = P.forward(cfg, W64, toks, st, **kw)
    for ctx in (1000, 5000):
        m = build(cuda_ctx, cfg, W, dtype, ctx)
        assert U.error(m.forward(toks[:880], range(3, 880, 40)), ref[3:880:40]) < TOL[dtype]
        assert U.error([m.decode(t)[0] for t in toks[880:]], ref[880:]) < TOL[dtype]
        m.Dispose()


# ---- generation ----------------------------------------------------------------------------------------------------------------
def test_greedy_generation(cuda_ctx, tmp_path):
    cfg, W, toks, _, _ = plain("even")
    W64 = to64(W)
    m = try_create(cuda_ctx, ModelOptions(ModelPath=U.write_folder(tmp_path / "m", cfg, W), KVCacheSize=300, WeightDType="f32"))
    st = P.State(cfg)
    lg = P.forward(cfg, W64, toks[:20], st)[-1]
    want = [int(np.argmax(lg))]
    while len(want) < 200:
        want.append(int(np.argmax(P.step(cfg, W64, st, want[-1]))))
    assert m.run_tokens(toks[:20], 60) == want[:60]
    m.reset()
    _, tk = m.prefill(toks[:20])
    got, ms = m.decode_greedy(tk, 199)  # long decoding, fed back on the device
    assert [tk] + got.tolist() == want and ms > 0
    m.Dispose()


def test_sampled_generation(cuda_ctx):
    cfg, W, toks, _, _ = plain("even")
    m = build(cuda_ctx, cfg, W, "bf16", 300)
    us = np.random.default_rng(3).random(12, dtype=np.float32)
    _, tk = m.prefill(toks[:20])
    got, _ = m.decode_sampled(tk, us, temperature=1.3)
    m.reset()
    m.prefill(toks[:20])
    x, stepped = tk, []
    for u in us:
        m.decode(x)
        x = m.sample_top_p(temperature=1.3, u=float(u))
        stepped.append(x)
    assert got.tolist() == stepped and len(set(stepped)) > 1
    m.Dispose()


# ---- replay, errors, timers -------------------------------------------------------------------------------------------------------
def test_replay_of_two_sequences(cuda_ctx, tmp_path):
    """Two interleaved sequences replayed against each alone."""
    cfg, W, toks, want, _ = plain("odd")
    m = try_create(cuda_ctx, ModelOptions(ModelPath=U.write_folder(tmp_path / "model", cfg, W), KVCacheSize=CTX, WeightDType="f32"))
    other = U.tokens(cfg, W, 70, 9)
    ref_other = P.forward(cfg, to64(W), other)
    steps = [{"step": 0, "entries": [{"id": "x", "tokens": toks[:33], "want": [0, 32]}], "end": []},
             {"step": 1, "entries": [{"id": "y", "tokens": other[:9], "want": [8]}], "end": []},
             {"step": 2, "entries": [{"id": "x", "tokens": toks[33:35], "want": [0, 1]}, {"id": "y", "tokens": other[9:70], "want": [60]}], "end": ["y"]},
             {"step": 3, "entries": [{"id": "x", "tokens": toks[35:200], "want": [164]}], "end": ["x"]}]
    trace.replay(m, [json.dumps(s) for s in steps], str(tmp_path), lambda s: None)
    read = lambda n: np.fromfile(tmp_path / f"{n}.f32", "<f4").reshape(-1, cfg["vocab"])  # noqa: E731
    assert U.error(read(0), want[[0, 32]]) < TOL["f32"] and U.error(read(1), ref_other[8]) < TOL["f32"]
    assert U.error(read(2), np.vstack([want[[33, 34]], ref_other[[69]]])) < TOL["f32"]
    assert U.error(read(3), want[199]) < TOL["f32"]
    m.Dispose()


def test_trace_program(tmp_path):
    cfg, W, toks, want, _ = plain("ones")
    U.write_folder(tmp_path / "model", cfg, W)
    root = os.path.dirname(os.path.dirname(os.path.abspath(__file__)))
    steps = [{"step": 0, "entries": [{"id": "x", "tokens": toks[:40], "want": [39]}], "end": []},
             {"step": 1, "entries": [{"id": "x", "tokens": toks[40:41], "want": [0]}], "end": ["x"]}]
    r = subprocess.run([os.path.join(root, "bin", "trace_run"), "--model", str(tmp_path / "model"), "--dtype", "float32", "--out",
                        str(tmp_path), "--max-tokens", "41"], input="".join(json.dumps(s) + "\n" for s in steps), text=True,
                       capture_output=True, timeout=600)
    assert r.returncode == 0, r.stderr
    assert r.stdout.splitlines()[-2:] == ["done 0", "done 1"]
    got = np.vstack([np.fromfile(tmp_path / f"{n}.f32", "<f4").reshape(1, -1) for n in (0, 1)])
    assert U.error(got, want[39:41]) < TOL["f32"]


def test_misuse_is_an_error(cuda_ctx):
    cfg, W, toks, _, _ = plain("ones")
    t = U.tensors(W)
    for bad in (t[:-1], [x for x in t if x[0] != "l0.mlp.correction"], [x for x in t if x[0] != "l1.norm2"]):
        with pytest.raises(NfaiError) as e:
            PlannedModel.from_tensors(cuda_ctx, cfg, bad, 32, "bf16")
        assert e.value.code == _lib.ERR_STATE
    for name, shape in (("l0.norm1", (40,)), ("l1.mix.k", (16, 40)), ("l1.mlp.e4.gate", (16, 40)), ("l2.mix.q.b", (8,))):
        with pytest.raises(NfaiError) as e:
            PlannedModel.from_tensors(cuda_ctx, cfg, [(name, np.zeros(shape, np.float32), _lib.F32)], 32, "bf16")
        assert e.value.code == _lib.ERR_ARG
    deep = U.config([U.layer(U.attn(1, 1, 520, 8))], 40, 64)
    with pytest.raises(NfaiError) as e:
        build(cuda_ctx, deep, U.weights(deep), "bf16")
    assert e.value.code == _lib.ERR_ARG
    m = build(cuda_ctx, cfg, W, "bf16", 32)
    m.forward(toks[:20])
    with pytest.raises(NfaiError) as e:
        m.forward(toks[:13], [0, 12])
    assert e.value.code == _lib.ERR_CONTEXT_FULL
    m.Dispose()


def test_profiled_kernels(cuda_ctx):
    cfg, W, toks, want, _ = plain("even")
    m = build(cuda_ctx, cfg, W, "bf16")
    m.forward(toks[:100])
    assert {"ffn_gate_up", "expert_gate_up", "shared_gate_up_router", "expert_down", "attention", "lm_head"} <= set(m.KERNELS)
    for name in m.KERNELS:
        ms, nbytes = m.profile_kernel(name, 4)
        assert ms > 0 and nbytes > 0
    assert U.error(m.decode(toks[100])[0], want[100]) < TOL["bf16"]  # timing leaves the sequence as it was
    m.Dispose()
